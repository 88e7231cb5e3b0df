"""Furesun in the engine against its plain float64 statement (``plain_furesun``): its kernels and each mechanism alone,
every way of cutting the work, batches, pages and state slots used again, keys far away and at the edges of windows, pages
and key tiles, keys of another layer, the first tokens, long decoding, generation."""
import copy
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import furesun_configs as fc
import plain_furesun as pf
import statement_tools
import trace_tools

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# max |logit difference| relative to the largest |logit|
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
# bfloat16: one row in fifty may reach ``STRAY_FACTOR`` times what is allowed (two draws of noise do not meet every jump)
STRAY = {"float32": 0.0, "bfloat16": 0.02}
STRAY_FACTOR = 4.0
LENGTHS = {"A": [1, 2, 15, 16, 17, 33, 63, 64, 65, 150], "B": [3, 31, 32, 48, 97, 129, 210]}


def expected(cfg, w, seqs):
    return statement_tools.expected(pf.forward, cfg, w, seqs)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(name, dtype) -> folder, config, weights, sequences, expected logits.  The bfloat16 runs get the same weights with
    routers that no rounding can flip (``furesun_configs.steady_routing``)."""
    out = {}
    for i, (name, cfg) in enumerate(fc.CONFIGS.items()):
        rng = random.Random(400 + i)
        seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in LENGTHS[name]]
        for dtype, edit in (("float32", fc.steady), ("bfloat16", fc.steady_routing)):
            folder = fc.make_folder(cfg, str(tmp_path_factory.mktemp(f"u{name}{dtype}")), seed=61 + i, edit=edit)
            cfg_read, w = fc.read_folder(folder)
            out[name, dtype] = (folder, cfg_read, w, seqs, expected(cfg_read, w, seqs))
    return out


def make_runner(folder, dtype, max_tokens, page_size=16, max_requests=4, **kw):
    from qwen_decoder_b200.engine import ModelRunner
    pages = (max_tokens + page_size - 1) // page_size
    return ModelRunner.from_folder(folder, dtype=dtype, device=DEV, num_pages=pages, page_size=page_size,
                                   max_requests=max_requests, max_positions=pages * page_size, **kw)


def held(seqs):
    return max((len(s) + 63) // 64 * 64 for s in seqs)


def all_free(runner):
    runner.cache.check()
    assert runner.cache.free_pages() == [runner.cache.num_pages] * len(runner.cache.pools)


def run(runner, tr, want, dtype, out_dir):
    got = trace_tools.run_inprocess(runner, tr, str(out_dir))
    trace_tools.compare(tr, got, want, TOL[dtype], stray=STRAY[dtype], stray_factor=STRAY_FACTOR, allow=want.allow[dtype])
    return got


def run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=128, tail=20, sizes=(7, 2, 24, 3, 2, 16, 5, 2, 31, 2), **kw):
    runner = make_runner(folder, dtype, max_tokens, **kw)
    for k, tr in enumerate((trace_tools.whole(seqs), trace_tools.portions(seqs, sizes=sizes),
                            trace_tools.decode_tail(seqs, tail=tail))):
        run(runner, tr, want, dtype, tmp_path / f"o{k}")
    all_free(runner)


# ---------------------------------------------------------------------------------------------------- the kernels alone
@pytest.mark.parametrize("D", [64, 96, 128, 100, 66, 2048, 4096, 12288])
def test_the_sum_itself_and_the_norm_of_a_branch(D, guard_regions):
    """x += n(delta), and the rounded sum (or chosen rows of it) as the next branch reads it."""
    from qwen_decoder_b200 import kernels
    gen = torch.Generator().manual_seed(D)
    rnd = lambda *s: torch.randn(s, generator=gen)
    x, w, parts = rnd(5, D), rnd(D), rnd(3, 5, D) * 30
    want = x.double() + pf.rms_div(parts.double().sum(0), 0.3) * w.double()
    for dt, tol in ((torch.bfloat16, 1e-2), (torch.float32, 1e-5)):
        xd, out = x.to(DEV), torch.empty((5, D), dtype=dt, device=DEV)
        kernels.group_add_norm(xd, parts.to(DEV), (w.to(DEV), 0.3, 1), out=out)
        assert torch.allclose(xd.cpu().double(), want, rtol=1e-5, atol=1e-4)
        assert torch.equal(out, xd.to(dt))
        rows = torch.tensor([4, 1], dtype=torch.int32, device=DEV)
        two = torch.empty((2, D), dtype=dt, device=DEV)
        kernels.group_add_norm(xd, None, out=two, rows=rows)
        assert torch.equal(two, xd[[4, 1]].to(dt))


def test_soft_cap(guard_regions):
    from qwen_decoder_b200 import kernels
    for n in (1, 3, 4, 1021, 4096):
        z = torch.randn(n, generator=torch.Generator().manual_seed(n)) * 40
        zd = torch.empty((n,), dtype=torch.float32, device=DEV).copy_(z)
        kernels.soft_cap(zd, 15.0)
        assert torch.allclose(zd.cpu().double(), pf.soft_cap(z.double(), 15.0), rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("T", [1, 5, 8])
def test_gelu_gates_in_every_form_of_the_feed_forward(T, guard_regions):
    """The one-launch feed-forward, the few-token kernels with their partial sums, library products, and float32."""
    from qwen_decoder_b200.parts.mlp import SwiGLU
    from qwen_decoder_b200.weights.loader import TensorSource
    for D, F, n in ((256, 1536, T), (2304, 512, T), (128, 264, 16), (512, 640, 12), (512, 640, 40), (256, 512, 100), (96, 40, 70)):
        gen = torch.Generator().manual_seed(D + F + n)
        part = SwiGLU(D, F, prefix="", names=("gate", "up", "down"), weight_suffix="", activation="gelu_tanh")
        w = {s.name: (torch.randn(s.shape, generator=gen) * D ** -0.5).bfloat16() for s in part.tensor_specs()}
        x = torch.randn((n, D), generator=gen).bfloat16()
        want = pf.gated(x.double(), {k: v.double() for k, v in w.items()}, "", pf.gelu_tanh)
        other = pf.gated(x.double(), {k: v.double() for k, v in w.items()}, "", pf.silu)
        assert float((other - want).abs().max()) > 0.08 * float(want.abs().max())
        for dt, tol in ((torch.bfloat16, 2e-2), (torch.float32, 1e-5)):
            part.bind(TensorSource.from_dict(w), dt, torch.device(DEV))
            assert float((part.forward(x.to(DEV, dt), None).double().reshape(-1, n, D).sum(0).cpu() - want).abs().max()) <= tol * float(want.abs().max())


def test_gelu_gates_element_by_element(guard_regions):
    """Large, small and negative gates through the elementwise kernels."""
    from qwen_decoder_b200 import kernels
    g = torch.cat([torch.linspace(-30, 30, 241), torch.tensor([-1e4, -300.0, 300.0, 1e4, 0.0, 1e-3, -1e-3])])
    g = torch.cat([g, torch.zeros(256 - g.numel())]).repeat(3, 1)
    u = torch.randn(3, 256, generator=torch.Generator().manual_seed(1))
    gu = torch.cat([g, u], dim=1)
    want = pf.gelu_tanh(g.double()) * u.double()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        x = gu.to(dt)
        ref = pf.gelu_tanh(x[:, :256].double()) * x[:, 256:].double()
        out = torch.empty((3, 256), dtype=dt, device=DEV)
        kernels.swiglu(x.to(DEV), out, kernels.ACT_GATED_GELU)
        assert torch.allclose(out.cpu().double(), ref, rtol=tol, atol=1e-5)
        kernels.gated_act(gu.to(DEV), out, kernels.ACT_GATED_GELU)
        assert torch.allclose(out.cpu().double(), want, rtol=tol, atol=1e-5)
    out = torch.empty((3, 256), dtype=torch.bfloat16, device=DEV)
    kernels.swiglu_partial(torch.stack([gu * 0.25, gu * 0.75]).to(DEV), out, act=kernels.ACT_GATED_GELU)
    assert torch.allclose(out.cpu().double(), want, rtol=2e-2, atol=1e-5)


@pytest.mark.parametrize("E", [3, 40, 256, 300])
def test_normalised_sigmoid_routing(E, guard_regions):
    """The largest sigmoids over their sum times a constant, by both choice kernels; very small scores too."""
    from qwen_decoder_b200 import kernels
    gen = torch.Generator().manual_seed(E)
    for top in (1, 2, 3):
        z = torch.randn((9, E), generator=gen) * 3
        z[4] -= 40.0
        idx = torch.empty((9, top), dtype=torch.int32, device=DEV)
        wt = torch.empty((9, top), dtype=torch.float32, device=DEV)
        kernels.moe_choose(z.to(DEV), top, idx, wt, kernels.MOE_ROUTE_TOP_SIGMOID_NORM, scale=2.5)
        best = torch.topk(z.double(), top)
        s = torch.sigmoid(best.values)
        assert torch.equal(idx.cpu().long(), best.indices)
        assert torch.allclose(wt.cpu().double(), 2.5 * s / (s.sum(-1, keepdim=True) + 1e-20), rtol=1e-5)


def _step(lens, slots):
    """What the recurrence's kernels read of a step's context."""
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device=DEV)
    req = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(lens)).to(torch.int32).to(DEV)
    return SimpleNamespace(num_requests=len(lens), token_request=req, cu_tokens=cu, positions=torch.zeros_like(req),
                           state_slots=torch.tensor(slots, dtype=torch.int32, device=DEV))


@pytest.mark.parametrize("H,d,dv", [(2, 16, 8), (4, 64, 64), (3, 20, 100), (2, 128, 130), (1, 7, 5), (6, 96, 48), (3, 33, 12),
                                     (2, 256, 31), (1, 48, 300)])
def test_exponential_gates_and_the_normaliser(H, d, dv, guard_regions):
    """``LinearAttention.inner`` with exponential gates against the recurrence in float64: portions of unequal length (one longer
    than a turn of the gates' scan), single tokens, states and maxima that are not zero, slots that must stay as they are, a
    portion cut in four.  eps is large enough for the denominator to show."""
    from qwen_decoder_b200.cache import FixedState  # noqa: F401
    from qwen_decoder_b200.parts.base import StateCacheView
    from qwen_decoder_b200.parts.linear_attention import LinearAttention
    gen = torch.Generator().manual_seed(H * 1000 + d + dv)
    rnd = lambda *s: torch.randn(s, generator=gen)
    eps, cap = 0.4, 6.0
    part = LinearAttention(8, H, d, dv, eps=eps, q_scale=d ** -0.5, gate_cap=cap, norm_weight="all", output_gate="sigmoid", prefix="")
    part.norm, part.i_bias, part.f_bias = rnd(H * dv).to(DEV), rnd(H).to(DEV), (rnd(H) + 2).to(DEV)
    n, width = part.state_size(), 2 * H * d + 2 * H * dv + 2 * H
    state0 = rnd(5, n) * 0.2
    for lens, slots in (([1, 37, 16, 2], [3, 0, 4, 1]), ([1, 1, 1], [2, 4, 0]), ([300], [1]), ([2], [2])):
        T = sum(lens)
        u = rnd(T, width + (-width) % 8)
        u[:, part.i_off:part.i_off + 2 * H] *= 4.0                           # gates that open, close and meet the cap
        S = state0[:, :H * (dv + 1) * d].double().reshape(5, H, dv + 1, d).clone()
        m = state0[:, H * (dv + 1) * d:H * (dv + 1) * d + H].double().clone()
        want = torch.zeros((T, H * dv), dtype=torch.float64)
        capped = lambda z: cap * torch.tanh(z / cap)
        i = capped(u[:, part.i_off:part.i_off + H].double() + part.i_bias.cpu().double())
        f = pf.log_sigmoid(capped(u[:, part.f_off:part.f_off + H].double() + part.f_bias.cpu().double()))
        t, floors = 0, 0
        for ln, sl in zip(lens, slots):
            for _ in range(ln):
                for h in range(H):
                    q, k = u[t, h * d:(h + 1) * d].double() * d ** -0.5, u[t, H * d + h * d:H * d + (h + 1) * d].double()
                    v = torch.cat([u[t, 2 * H * d + h * dv:2 * H * d + (h + 1) * dv].double(), torch.ones(1, dtype=torch.float64)])
                    new = max(float(f[t, h] + m[sl, h]), float(i[t, h]))
                    S[sl, h] = np.exp(float(f[t, h] + m[sl, h]) - new) * S[sl, h] + np.exp(float(i[t, h]) - new) * v[:, None] * k[None, :]
                    m[sl, h] = new
                    o = S[sl, h] @ q
                    floors += abs(float(o[dv])) < np.exp(-new)
                    y = o[:dv] / (max(abs(float(o[dv])), np.exp(-new)) + 1e-6)
                    gate = torch.sigmoid(u[t, 2 * H * d + H * dv + h * dv:2 * H * d + H * dv + (h + 1) * dv].double())
                    want[t, h * dv:(h + 1) * dv] = pf.rms_div(y, eps) * part.norm.cpu().double()[h * dv:(h + 1) * dv] * gate
                t += 1
        if T > 20:
            assert 0 < floors < T * H                                        # both sides of the maximum in the denominator
        full = state0.double().clone()
        full[:, :H * (dv + 1) * d] = S.reshape(5, -1)
        full[:, H * (dv + 1) * d:H * (dv + 1) * d + H] = m
        x = torch.zeros((T, 8), dtype=torch.float32, device=DEV)
        state, out = state0.to(DEV), torch.zeros((T, H * dv + 4), device=DEV)
        part.inner(x, _step(lens, slots), StateCacheView(state, True), out[:, :H * dv], u=u.to(DEV))
        assert float((out[:, :H * dv].cpu().double() - want).abs().max()) <= 1e-4 * float(want.abs().max())
        assert not out[:, H * dv:].any()
        assert float((state.cpu().double() - full).abs().max()) <= 2e-5 * float(full.abs().max())
        for sl in set(range(5)) - set(slots):
            assert torch.equal(state[sl].cpu(), state0[sl])
        assert torch.equal(state[:, H * (dv + 1) * d + H:].cpu(), state0[:, H * (dv + 1) * d + H:])
        if lens == [300]:                                                    # cut into 1 + 20 + 270 + 9: the same
            st2, out2 = state0.to(DEV), torch.zeros_like(out)
            for a, b in ((0, 1), (1, 21), (21, 291), (291, 300)):
                part.inner(x[a:b], _step([b - a], slots), StateCacheView(st2, True), out2[a:b, :H * dv], u=u[a:b].to(DEV))
            assert float((st2 - state).abs().max()) <= 1e-5 * float(full.abs().max())
            assert float((out2 - out).abs().max()) <= 1e-4 * float(want.abs().max())
            for a, b in ((0, 300), (0, 1)):                                  # runs that do not write
                part.inner(x[a:b], _step([b - a], slots), StateCacheView(st2, False), out2[a:b, :H * dv], u=u[a:b].to(DEV))
            assert float((st2 - state).abs().max()) <= 1e-5 * float(full.abs().max())


# ------------------------------------------------------------------------------------------------- each mechanism alone
SMALL = fc.attn(2, 1, 8, 8, 30)
ONE_LAYER = {
    # name: (mixer, feed-forward, width, eps); a large eps lets the size of a recurrent head's output show
    "window_of_five": (fc.attn(4, 2, 16, 24, 5, softcap=1.5, scale=0.9), None, 64, 1e-5),
    "window_of_a_page_part_rotated": (fc.attn(2, 2, 24, 8, 16, rot_dims=12, base=50.0, softcap=50.0), None, 64, 1e-5),
    "window_of_sixty_four_wide_heads": (fc.attn(2, 1, 128, 64, 64, scale=0.06), None, 64, 1e-5),
    "window_of_one": (fc.attn(3, 3, 10, 6, 1), None, 66, 1e-5),
    "window_past_the_prompt_many_heads": (fc.attn(40, 2, 8, 16, 1000, rot_dims=4, softcap=0.7, scale=1.1), None, 48, 1e-5),
    "window_odd_head_no_rotation_no_cap": ({"type": "attention", "mixer": {**fc.attn(2, 1, 9, 7, 40)["mixer"], "rot": None, "softcap": None}}, None, 40, 1e-5),
    "window_heads_of_176": (fc.attn(4, 2, 176, 88, 33, rot_dims=64), None, 64, 1e-5),
    "latent": (fc.latent(4, 16, 8, 24, 32, 20), None, 64, 1e-5),
    "latent_one_key_no_stretch": (fc.latent(2, 8, 8, 8, 16, 1, scaling=None), None, 64, 1e-5),
    "latent_wide_heads_stretched": (fc.latent(2, 128, 64, 128, 96, 70, scaling=(8.0, 32, 32.0, 1.0)), None, 64, 1e-5),
    "latent_rows_of_no_whole_pieces": (fc.latent(3, 12, 6, 10, 21, 64, base=30.0), None, 60, 1e-5),
    "latent_window_past_the_prompt": (fc.latent(9, 24, 16, 40, 56, 500, scale=0.5), None, 64, 1e-5),
    "latent_part_rotated": ({"type": "latent_attention", "mixer": {**fc.latent(2, 16, 24, 16, 40, 30)["mixer"], "rot": {"base": 90.0, "dims": 8}}}, None, 64, 1e-5),
    "memory_one_head": (fc.mlstm(1, 64, 64), None, 64, 0.5),
    "memory_values_larger": (fc.mlstm(3, 24, 40, cap=4.0), None, 64, 0.2),
    "memory_values_smaller_low_cap": (fc.mlstm(4, 32, 12, cap=0.5), None, 64, 1e-3),
    "memory_odd_sizes": (fc.mlstm(3, 21, 13), None, 60, 0.3),
    "memory_heads_of_200": (fc.mlstm(2, 200, 24), None, 64, 0.1),
    "memory_wide": (fc.mlstm(2, 128, 96), fc.dense(32), 64, 1e-2),
    "dense": (SMALL, fc.dense(88), 64, 1e-5),
    "dense_odd": (fc.mlstm(2, 8, 8), fc.dense(50), 100, 1e-2),
    "experts": (SMALL, fc.moe(7, 3, 24), 64, 1e-5),
    "experts_one_of_many_and_shared": (SMALL, fc.moe(9, 1, 40, scale=2.5, shared=56), 64, 1e-5),
    "experts_all_chosen": (SMALL, fc.moe(3, 3, 16, scale=0.5, shared=8), 64, 1e-5),
    "a_width_of_no_whole_16_byte_rows": (fc.latent(2, 10, 4, 12, 20, 30), fc.moe(4, 2, 22, shared=14), 100, 1e-4),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_each_mechanism_alone(name, dtype, tmp_path):
    """One layer: a prompt at once, in portions, and its tail token by token."""
    mix, mlp, width, eps = ONE_LAYER[name]
    cfg = fc.one_layer(mix, mlp, width=width, eps=eps)
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=sum(map(ord, name)), std=0.15,
                            edit=fc.steady_routing if dtype == "bfloat16" else fc.steady)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(len(name))
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1, 2, 37, 90)]
    run_all_ways(folder, dtype, seqs, expected(cfg, w, seqs), tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_whole_and_decode_tail(models, name, dtype, tmp_path):
    folder, cfg, w, seqs, want = models[name, dtype]
    runner = make_runner(folder, dtype, held(seqs), page_size=32 if name == "B" else 16)
    for k, tr in enumerate((trace_tools.whole(seqs), trace_tools.decode_tail(seqs, tail=40))):
        run(runner, tr, want, dtype, tmp_path / f"o{k}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_down_to_two_tokens(models, name, dtype, tmp_path):
    folder, cfg, w, seqs, want = models[name, dtype]
    runner = make_runner(folder, dtype, held(seqs), page_size=16 if name == "B" else 24)     # 24: no divisor of a key tile
    for k, sizes in enumerate(((7, 2, 24, 3, 2, 16, 5, 2, 31, 2), (2,), (64, 1, 3), (1, 1, 2, 1), (40, 33, 2))):
        run(runner, trace_tools.portions(seqs, sizes=sizes), want, dtype, tmp_path / f"o{k}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype, tmp_path):
    """Unequal requests side by side, portions beside single tokens, in a pool of about two of the longest with three
    state slots: every page and every slot serves several requests in turn.  A key read from a page's former owner, or a
    state or maximum left over from a slot's former owner, shows against the statement."""
    folder, cfg, w, seqs, want = models[name, dtype]
    max_tokens = 2 * held(seqs)
    runner = make_runner(folder, dtype, max_tokens, max_requests=3)
    for seed, sizes in ((11, (2, 3, 5, 8, 13, 24)), (12, (2, 35, 50))):
        tr = trace_tools.mixed(seqs + seqs[::-1], max_tokens, seed=seed, max_live=3, portion_sizes=sizes)
        assert sum(len(s["entries"]) > 1 for s in tr.steps) > 5
        run(runner, tr, want + want[::-1], dtype, tmp_path / f"o{seed}")
    all_free(runner)


def test_a_request_alone_and_in_a_batch_agree(models, tmp_path):
    """float32: the same rows from a batch of unequal requests and from each request alone differ by rounding
    of sums at most (far less than from the plain statement)."""
    folder, cfg, w, seqs, want = models["A", "float32"]
    runner = make_runner(folder, "float32", 4 * held(seqs))
    a = trace_tools.whole(seqs)
    ga = trace_tools.run_inprocess(runner, a, str(tmp_path / "a"))
    b = trace_tools.mixed(seqs, 4 * held(seqs), seed=3, max_live=4)
    gb = trace_tools.run_inprocess(runner, b, str(tmp_path / "b"))
    rows_a = {rp: ga[s][i] for s, rows in a.expect.items() for i, rp in enumerate(rows)}
    rows_b = {rp: gb[s][i] for s, rows in b.expect.items() for i, rp in enumerate(rows)}
    scale = max(float(np.abs(x).max()) for x in want)
    assert max(float(np.abs(rows_a[k] - rows_b[k]).max()) for k in rows_b) <= 1e-5 * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_and_first_tokens(models, name, dtype, tmp_path):
    """Two tokens of prompt, then 300 tokens one by one across many pages, windows and key tiles: the states are carried
    300 times; the first positions are compared one by one."""
    folder, cfg, w, _, _ = models[name, dtype]
    rng = random.Random(77)
    seq = [rng.randrange(cfg["vocab"]) for _ in range(302)]
    runner = make_runner(folder, dtype, 320)
    run(runner, trace_tools.decode_tail([seq], tail=300), expected(cfg, w, [seq]), dtype, tmp_path)
    all_free(runner)


# ------------------------------------------------------------------------------- faults that random weights would hide
def moved(cfg, w, seq, want, change_cfg=None, change_w=None):
    """The share of positions at which the statement itself moves, by far more than the tolerance, under a change."""
    c, ww = copy.deepcopy(cfg), dict(w)
    if change_cfg:
        change_cfg(c)
    if change_w:
        change_w(ww)
    d = np.abs(pf.forward(c, ww, seq).numpy() - want).max(axis=-1)
    return d > 3 * TOL["float32"] * np.abs(want).max()


EDGES = {
    "attention": fc.attn(4, 2, 16, 40, 96, base=200.0, softcap=30.0, scale=1.0),
    "attention_low_cap": fc.attn(4, 2, 16, 40, 96, base=200.0, softcap=4.0, scale=1.0),
    "latent": fc.latent(4, 16, 8, 40, 32, 96, base=200.0, scale=1.0),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", sorted(EDGES))
def test_single_keys_at_the_edges_of_windows(kind, dtype, tmp_path, monkeypatch):
    """Scores sharpened so that single keys (or the one in the denominator) take most of the weight: prompts that end just
    before, at and just after page, key-tile and window borders, their tails decoded token by token.  The statement is
    shown to depend on the edge on both sides, on the one, and on the cap."""
    f = 1.0 if dtype == "float32" else 0.45
    cfg = fc.one_layer(EDGES[kind], None, vocab=400, width=48)

    def sharpen(t):
        if "l0.mix.q.norm" in t:
            t["l0.mix.q.norm"] = (t["l0.mix.q.norm"].float() * 1.1 * f).to(torch.bfloat16)
        else:
            t["l0.mix.q"] = (t["l0.mix.q"].float() * 8.0 * f).to(torch.bfloat16)
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=5, std=0.2, edit=sharpen)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(8)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (95, 96, 97, 193, 400)]
    want = expected(cfg, w, seqs)
    for size in (95, 97):
        other = lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", size)
        assert moved(cfg, w, seqs[-1], want[-1], change_cfg=other).mean() > 0.1
    if kind != "latent":
        with monkeypatch.context() as m:
            m.setattr(pf, "softmax_plus_one", pf.softmax)
            assert moved(cfg, w, seqs[-1], want[-1]).mean() > 0.1
        assert moved(cfg, w, seqs[-1], want[-1], change_cfg=lambda c: c["layers"][0]["mixer"].__setitem__("softcap", None)).mean() > 0.1
    else:
        assert moved(cfg, w, seqs[-1], want[-1], change_cfg=lambda c: c["layers"][0]["mixer"]["rot"].pop("scaling")).mean() > 0.1
    runner = make_runner(folder, dtype, 512)
    for i, tr in enumerate((trace_tools.whole(seqs), trace_tools.decode_tail(seqs, tail=36), trace_tools.portions(seqs, sizes=(100, 2, 3, 64)),
                            trace_tools.portions(seqs, sizes=(31, 33, 2)))):
        run(runner, tr, want, dtype, tmp_path / f"o{i}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("own,reader", [(8, 120), (120, 8)])
def test_keys_of_another_layer_through_another_window(own, reader, dtype, tmp_path):
    """A layer that reads an earlier layer's keys through a wider (and a narrower) window than that layer's own, its queries
    sharpened: a wide reader still finds the keys that the owner's window has passed, in prompts and while decoding.  The
    statement depends on the reader's window and on whose keys they are."""
    f = 1.0 if dtype == "float32" else 0.5
    a, b = fc.attn(2, 2, 16, 24, own, softcap=30.0, scale=0.5), fc.attn(4, 2, 16, 24, reader, softcap=20.0, scale=0.9, kv_from=0)
    cfg = fc.config(300, 48, 1e-5, [(a, None), (b, fc.dense(32))])

    def sharpen(t):
        t["l1.mix.q.norm"] = (t["l1.mix.q.norm"].float() * 2.5 * f).to(torch.bfloat16)
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=15, std=0.2, edit=sharpen)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(4)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (300, 129, 121)]
    want = expected(cfg, w, seqs)
    for change in (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", reader - 1),
                   lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", own + 1)):
        assert moved(cfg, w, seqs[0], want[0], change_cfg=change).mean() > 0.1
    runner = make_runner(folder, dtype, 320)
    assert runner.layout.groups[0].need.window == 120 and len(runner.layout.groups) == 1
    for i, tr in enumerate((trace_tools.whole(seqs), trace_tools.decode_tail(seqs, tail=60), trace_tools.portions(seqs, sizes=(50, 2, 3, 64)))):
        run(runner, tr, want, dtype, tmp_path / f"o{i}")
    all_free(runner)
    runner = make_runner(folder, dtype, 640, max_requests=2)
    tr = trace_tools.mixed(seqs + seqs[::-1], 640, seed=2, max_live=2, portion_sizes=(2, 9, 40))
    run(runner, tr, want + want[::-1], dtype, tmp_path / "mixed")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_token_far_back_in_the_memory(dtype, tmp_path):
    """One token hundreds of positions back whose write stays readable: open forget gates, and a key, value and input gate that
    stand out.  The statement's logits at the end depend on that token and on the normaliser it went into; a state or a maximum
    lost, reset or left over on the way shows."""
    cfg = fc.one_layer(fc.mlstm(2, 16, 24, cap=9.0), None, vocab=300, width=48, eps=0.5)

    def edit(t):
        t["l0.mix.f.b"].fill_(6.0)
        t["l0.mix.i.b"].fill_(-1.0)
        t["l0.mix.k"][:] = (0.9 * t["l0.mix.q"].float() + 0.2 * t["l0.mix.k"].float()).to(torch.bfloat16)
        for tok in range(300):                      # one channel belongs to token 7 alone; values and input gates read it strongly
            t["embed"][tok][0] = 30.0 if tok == 7 else 0.0
        t["l0.mix.k"][:, 0] *= 0.1
        t["l0.mix.v"][:, 0] *= 4.0
        t["l0.mix.v"][:, 1:] *= 0.5
        t["l0.mix.i"][:, 0] = 0.12
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=9, std=0.2, edit=edit)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(6)
    seq = [rng.choice([x for x in range(300) if x != 7]) for _ in range(420)]
    seq[33] = 7
    seqs = [seq, seq[:330]]
    want = expected(cfg, w, seqs)
    other = list(seq)
    other[33] = 8
    d = np.abs(pf.forward(cfg, w, other).numpy()[300:] - want[0][300:]).max(axis=-1)
    assert (d > 2 * np.maximum(TOL[dtype] * np.abs(want[0]).max(), want.allow[dtype][0][300:])).mean() > 0.3
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=448, tail=60, sizes=(100, 2, 3, 64, 1))
    runner = make_runner(folder, dtype, 2 * 448, max_requests=2)
    tr = trace_tools.mixed(seqs + seqs[::-1], 2 * 448, seed=2, max_live=2, portion_sizes=(2, 9, 40))
    run(runner, tr, want + want[::-1], dtype, tmp_path / "mixed")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_decoding_over_a_long_window(kind, dtype, tmp_path):
    """A thousand keys in the window of each decoded token: its keys are shared among many CTAs whose partial results are
    added up (with the one in the denominator); alone and side by side."""
    mix = fc.attn(4, 2, 32, 40, 1000, base=5000.0, softcap=25.0, scale=0.9) if kind == "attention" else \
        fc.latent(4, 24, 8, 40, 48, 1000, base=5000.0, scale=0.5)
    cfg = fc.one_layer(mix, None, vocab=150)
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=12, std=0.15)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(2)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1030, 1093)]
    want = expected(cfg, w, seqs)
    runner = make_runner(folder, dtype, 2304, page_size=32)
    run(runner, trace_tools.decode_tail(seqs, tail=70, keep=lambda r, p: p >= 940), want, dtype, tmp_path / "o")
    tr = trace_tools.Trace()
    n0 = 1000
    tr.add([(r, 0, s[:n0], []) for r, s in enumerate(seqs)])
    for p in range(n0, 1030):
        tr.add([(r, p, s[p:p + 1], [0]) for r, s in enumerate(seqs)], end=[0, 1] if p == 1029 else [])
    run(runner, tr, want, dtype, tmp_path / "p")
    all_free(runner)


def test_expanded_and_absorbed_latent_attention_agree(tmp_path, monkeypatch):
    """bfloat16: long portions expand keys and values of the rows in the window, short ones carry the queries into the
    latent; both forms over the same steps, and with portions that start deep inside the sequence beside single tokens."""
    from qwen_decoder_b200 import kernels
    from qwen_decoder_b200.parts import latent_attention as la
    cfg = fc.config(200, 64, 1e-5, [(fc.latent(4, 24, 16, 32, 48, 50, scale=0.4), None), (fc.latent(2, 72, 64, 24, 64, 130), None)])
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=3, std=0.15)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(1)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (300, 150, 64)]
    want = expected(cfg, w, seqs)
    calls = []
    real = kernels.latent_queries
    monkeypatch.setattr(kernels, "latent_queries", lambda *a, **k: (calls.append(1), real(*a, **k)))
    for least, expands in ((2, True), (10000, False)):
        monkeypatch.setattr(la, "EXPAND_TOKENS", least)
        calls.clear()
        runner = make_runner(folder, "bfloat16", 768)
        for i, tr in enumerate((trace_tools.whole(seqs), trace_tools.portions(seqs, sizes=(60, 2, 41)),
                                trace_tools.mixed(seqs, 768, seed=4, portion_sizes=(2, 40, 64)))):
            run(runner, tr, want, "bfloat16", tmp_path / f"o{least}_{i}")
        all_free(runner)
        assert bool(calls) == expands


# -------------------------------------------------------------------------------------------------- the engine around it
def test_greedy_generation_through_the_engine(models):
    """``Engine.generate`` (scheduler, portions of prompts, batched decoding as replayed graphs, the sampler's
    argmax) against greedy decoding with the plain statement, for prompts of unequal length at once."""
    from qwen_decoder_b200.engine import Engine, SamplingParams
    folder, cfg, w, seqs, _ = models["A", "float32"]
    prompts = [seqs[2], seqs[5][:20], seqs[4], seqs[1], seqs[9][:50]]
    new = 12
    engine = Engine(folder, dtype="float32", max_batch=3, max_prefill_tokens_per_step=24, max_total_tokens=64,
                    num_pages=40, page_size=16, max_positions=256)
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    for prompt, out in zip(prompts, outs):
        seq = list(prompt)
        for _ in range(new):
            logits = pf.forward(cfg, w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            assert float(top2[0] - top2[1]) > 1e-4, "a close call: choose another seed for this test"
            seq.append(int(torch.argmax(logits)))
        assert out == seq[len(prompt):]
    all_free(engine.runner)
    # bfloat16 with replayed graphs: every token the engine chose is, for the statement, the best one or within the
    # rounding of it (a near-tie may go either way, after which the statement follows the engine's sequence)
    folder, cfg, w, _, _ = models["A", "bfloat16"]
    e16 = Engine(folder, dtype="bfloat16", max_batch=4, max_prefill_tokens_per_step=32, max_total_tokens=64,
                 num_pages=40, page_size=16, max_positions=256)
    for prompt, out in zip(prompts, e16.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))):
        seq = list(prompt)
        assert len(out) == new
        for tok in out:
            logits = pf.forward(cfg, w, seq)[-1]
            assert float(logits.max() - logits[tok]) <= 2 * TOL["bfloat16"] * float(logits.abs().max())
            seq.append(tok)
    all_free(e16.runner)


def test_the_programs_take_the_folder(models, tmp_path):
    """``bin/decoder_main`` and ``bin/trace_run`` as separate processes on a Furesun folder: the command line's greedy
    tokens are the statement's, and a replayed trace with four live requests in a small pool gives its logits."""
    import os
    import subprocess
    import sys
    root = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..")
    folder, cfg, w, seqs, want = models["A", "float32"]
    prompts = [seqs[2], seqs[3]]
    stdin = "".join(" ".join(map(str, p)) + "\n" for p in prompts) + "\n"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "decoder_main"), folder, "8", "4096", "16", "64", "0",
                        "--dtype", "float32", "--max-new-tokens", "5", "--num-pages", "16", "--ignore-eos"],
                       input=stdin, capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr
    lines = [l for l in r.stdout.splitlines() if l.startswith("[")]
    assert len(lines) == 2
    for p, line in zip(prompts, lines):
        got = [int(t) for t in line.split(")", 1)[1].split()]
        seq = list(p)
        for tok in got:
            logits = pf.forward(cfg, w, seq)[-1]
            assert float(logits.max() - logits[tok]) <= 1e-4 * float(logits.abs().max())
            seq.append(tok)
        assert len(got) == 5
    tr = trace_tools.mixed(seqs, max_tokens=2 * held(seqs), seed=9)
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", str(2 * held(seqs))], input=tr.lines(), capture_output=True,
                       text=True, timeout=900)
    assert r.returncode == 0, r.stderr
    assert r.stdout.splitlines() == [f"done {s['step']}" for s in tr.steps]
    trace_tools.compare(tr, trace_tools.read_outputs(tr, str(out), cfg["vocab"]), want, TOL["float32"],
                        allow=want.allow["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(1, 13)))
def test_models_drawn_at_random(seed, dtype, tmp_path):
    """Layers of any kind in any order with sizes, windows, shared keys, constants and feed-forwards drawn anew for every
    layer: whole, in portions, with decoded tails, and as mixed batches in a small pool with three state slots."""
    cfg = fc.drawn(seed)
    folder = fc.make_folder(cfg, str(tmp_path / "m"), seed=100 + seed, std=0.13, edit=fc.steady if dtype == "float32" else fc.steady_routing)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(seed)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1, 2, 19, 64, 65, 141)]
    want = expected(cfg, w, seqs)
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=192, tail=30, page_size=16 if seed % 2 else 32)
    max_tokens = 2 * held(seqs)
    runner = make_runner(folder, dtype, max_tokens, max_requests=3)
    tr = trace_tools.mixed(seqs + seqs[::-1], max_tokens, seed=seed, max_live=3, portion_sizes=(2, 3, 5, 13, 24, 40))
    run(runner, tr, want + want[::-1], dtype, tmp_path / "mixed")
    all_free(runner)


LARGER = fc.config(420, 192, 1e-5, [
    (fc.attn(6, 2, 128, 96, 256, rot_dims=64, base=2e5), fc.moe(6, 2, 64, shared=96)),
    (fc.mlstm(4, 64, 96), fc.dense(320)),
    (fc.attn(4, 2, 128, 96, 100, rot_dims=64, base=2e5, kv_from=0), fc.moe(5, 3, 72, scale=2.0)),
    (fc.latent(4, 128, 64, 128, 128, 200, scaling=(4.0, 128, 16.0, 1.0)), None),
    (fc.mlstm(2, 128, 64, cap=8.0), fc.moe(4, 1, 64, shared=64)),
])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_larger_model_with_long_prompts(dtype, tmp_path):
    """Heads of 128 and 192 with values of 96 and 128, prompts of up to 700 tokens over windows of 256, 100 and 200: several
    key tiles per query tile, single tokens whose keys are shared among CTAs, more than one turn of the gates' scan, every way
    of cutting, and a mixed batch in a small pool."""
    folder = fc.make_folder(LARGER, str(tmp_path / "m"), seed=31, std=0.1, edit=fc.steady if dtype == "float32" else fc.steady_routing)
    cfg, w = fc.read_folder(folder)
    rng = random.Random(14)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (700, 257, 384, 129, 513)]
    want = expected(cfg, w, seqs)
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=704, tail=40, sizes=(100, 2, 3, 64, 200, 7))
    runner = make_runner(folder, dtype, 1408, max_requests=3, page_size=32)
    tr = trace_tools.mixed(seqs, 1408, seed=5, max_live=3, prompt_frac=0.8, portion_sizes=(2, 9, 33, 64, 130))
    run(runner, tr, want, dtype, tmp_path / "mixed")
    all_free(runner)
