"""Gopevik in the engine against its plain float64 statement (``plain_gopevik``): its kernels and each mechanism alone,
every way of cutting the work, batches, pages and state slots used again, keys far away and at the edges of blocks, pages
and key tiles, the first tokens, long decoding, generation."""
import copy
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import gopevik_configs as gc
import plain_gopevik as pg
import trace_tools

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# max |logit difference| relative to the largest |logit|
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
# Every recurrent head's output is divided by its own length, and so is every part of a branch's output; a random model
# of several such layers multiplies rounding, at some tokens many times more than at others.  So a row may also differ by
# ``ALLOW`` times what the statement itself moves there when every weight gets relative noise of the size of the dtype's
# rounding (a lost key, a wrong page or a lost state moves most rows by far more).
NOISE = {"float32": 2e-7, "bfloat16": 2e-3}
ALLOW = 4.0
# bfloat16: one row in fifty may reach ``STRAY_FACTOR`` times that (two draws of noise do not meet every jump).
STRAY = {"float32": 0.0, "bfloat16": 0.02}
STRAY_FACTOR = 4.0
LENGTHS = {"A": [1, 2, 15, 16, 17, 33, 63, 64, 65, 150], "B": [3, 31, 32, 48, 97, 129, 210]}


class Expected(list):
    """The statement's logits per sequence, and what it allows per dtype and position."""
    allow = None

    def __add__(self, other):
        out = Expected(list(self) + list(other))
        out.allow = {d: self.allow[d] + other.allow[d] for d in self.allow}
        return out

    def __getitem__(self, i):
        if not isinstance(i, slice):
            return super().__getitem__(i)
        out = Expected(super().__getitem__(i))
        out.allow = {d: self.allow[d][i] for d in self.allow}
        return out


def expected(cfg, w, seqs):
    want = Expected(pg.forward(cfg, w, s).numpy() for s in seqs)
    gen = torch.Generator().manual_seed(1)
    want.allow = {}
    for dtype, eps in NOISE.items():
        rows = [np.zeros(len(s)) for s in seqs]
        for _ in range(2):
            noisy = {k: v.double() * (1 + eps * torch.randn(v.shape, generator=gen, dtype=torch.float64)) for k, v in w.items()}
            for r, s in enumerate(seqs):
                rows[r] = np.maximum(rows[r], np.abs(pg.forward(cfg, noisy, s).numpy() - want[r]).max(axis=-1))
        want.allow[dtype] = [ALLOW * x for x in rows]
    return want


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> folder, config, weights, sequences, expected logits."""
    out = {}
    for i, (name, cfg) in enumerate(gc.CONFIGS.items()):
        rng = random.Random(700 + i)
        seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in LENGTHS[name]]
        folder = gc.make_folder(cfg, str(tmp_path_factory.mktemp(f"g{name}")), seed=53 + i, edit=gc.steady)
        cfg_read, w = gc.read_folder(folder)
        out[name] = (folder, cfg_read, w, seqs, expected(cfg_read, w, seqs))
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


def run(runner, tr, want, dtype, out_dir, stray=None):
    got = trace_tools.run_inprocess(runner, tr, str(out_dir))
    trace_tools.compare(tr, got, want, TOL[dtype], stray=STRAY[dtype] if stray is None else stray, stray_factor=STRAY_FACTOR,
                        allow=want.allow[dtype])
    return got


def run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=128, tail=20, sizes=(7, 2, 24, 3, 2, 16, 5, 2, 31, 2),
                 stray=None, **kw):
    runner = make_runner(folder, dtype, max_tokens, **kw)
    for k, tr in enumerate((trace_tools.whole(seqs), trace_tools.portions(seqs, sizes=sizes),
                            trace_tools.decode_tail(seqs, tail=tail))):
        run(runner, tr, want, dtype, tmp_path / f"o{k}", stray)
    all_free(runner)


# ---------------------------------------------------------------------------------------------------- the kernels alone
@pytest.mark.parametrize("D,post_groups,pre_groups", [(64, 4, 4), (96, 3, 3), (2048, 8, 8), (4096, 1, 4), (4096, 16, 1),
                                                       (16384, 2, 2), (40, 4, 4), (66, 3, 6), (100, 1, 5), (36, 1, 36),
                                                       (8192, 128, 64), (8192, 1, 2), (12288, 3, 3), (384, 3, 1), (1536, 2, 4)])
@pytest.mark.parametrize("form", ["parts", "bf16", "float32"])
def test_group_add_norm(D, post_groups, pre_groups, form, guard_regions):
    """The grouped norm of a branch's output (partial sums, a bias), added, and the grouped norm of the sum; the parts
    have sizes of their own (one is a thousand times the others)."""
    from qwen_decoder_b200 import kernels
    gen = torch.Generator().manual_seed(D + post_groups)
    R = 5 if form != "bf16" else 150                            # few rows and many
    rnd = lambda *s: torch.randn(s, generator=gen)
    x, bias, pw, w = rnd(R, D), rnd(D), rnd(D), rnd(D)
    delta = rnd(3, R, D) if form == "parts" else rnd(R, D)
    delta[..., :D // post_groups] *= 1000.0
    if form == "bf16":
        delta = delta.bfloat16()
    y = (delta.double().sum(0) if form == "parts" else delta.double()) + bias.double()
    want_x = x.double() + pg.group_norm(y, pw.double(), 1e-5, post_groups)
    want_h = pg.group_norm(want_x, w.double(), 2e-3, pre_groups)
    for dt, rows, back in ((torch.float32, None, True), (torch.bfloat16, None, True), (torch.float32, [4, 1], False)):
        xd = x.to(DEV)
        rd = torch.tensor(rows, dtype=torch.int32, device=DEV) if rows else None
        out = torch.empty((len(rows) if rows else R, D), dtype=dt, device=DEV)
        kernels.group_add_norm(xd, delta.to(DEV), (pw.to(DEV), 1e-5, post_groups), bias.to(DEV), w.to(DEV), 2e-3, pre_groups, out,
                               rows=rd, write_back=back)
        assert torch.allclose(xd.cpu().double(), want_x if back else x.double(), rtol=1e-5, atol=1e-4)
        assert torch.allclose(out.cpu().double(), want_h[rows] if rows else want_h, rtol=2e-2 if dt == torch.bfloat16 else 1e-5, atol=1e-4)
    xd = x.to(DEV)                                              # the addition alone, with and without the norm
    kernels.group_add_norm(xd, delta.to(DEV), (pw.to(DEV), 1e-5, post_groups), bias.to(DEV))
    assert torch.allclose(xd.cpu().double(), want_x, rtol=1e-5, atol=1e-4)
    kernels.group_add_norm(xd, delta.to(DEV), None, bias.to(DEV))
    assert torch.allclose(xd.cpu().double(), want_x + y, rtol=1e-5, atol=5e-3)


def _step(lens, slots):
    """What the linear-attention kernels read of a step's context."""
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device=DEV)
    req = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(lens)).to(torch.int32).to(DEV)
    return SimpleNamespace(num_requests=len(lens), token_request=req, cu_tokens=cu,
                           state_slots=torch.tensor(slots, dtype=torch.int32, device=DEV))


@pytest.mark.parametrize("delta_rule", [False, True])
@pytest.mark.parametrize("H,G,d,dv", [(2, 2, 16, 8), (4, 2, 64, 64), (3, 1, 20, 100), (2, 2, 128, 130), (2, 1, 256, 32),
                                      (1, 1, 7, 5), (6, 3, 96, 48), (4, 4, 33, 12), (2, 2, 48, 300)])
def test_linear_scan(H, G, d, dv, delta_rule, guard_regions):
    """Portions of unequal length and single tokens against the recurrence in float64, from states that are not zero; a
    state slot that no request of the step has stays as it was; the same tokens in two steps give the same bits."""
    from qwen_decoder_b200 import kernels
    gen = torch.Generator().manual_seed(H * 1000 + d + dv)
    rnd = lambda *s: torch.randn(s, generator=gen)
    DP, off = kernels.linear_pad(d), 4
    n = off + H * d * dv + 3
    state0 = rnd(5, n)
    for lens, slots in (([1, 37, 16, 2], [3, 0, 4, 1]), ([1, 1, 1], [2, 4, 0]), ([70], [1])):
        T = sum(lens)
        q, k = rnd(T, G, d), torch.nn.functional.normalize(rnd(T, G, d), dim=-1)
        v, gate, norm = rnd(T, H * dv + 3), rnd(T, H * dv + 5), rnd(dv)
        g, beta = torch.rand((T, H), generator=gen), torch.rand((T, H), generator=gen)
        pad = lambda t: torch.nn.functional.pad(t, (0, DP - d)).to(DEV).contiguous()
        S = state0[:, off:off + H * d * dv].double().reshape(5, H, dv, d).clone()
        o = torch.zeros((T, H, dv), dtype=torch.float64)
        t = 0
        for ln, sl in zip(lens, slots):
            for _ in range(ln):
                for h in range(H):
                    kk, qq = k[t, h // (H // G)].double(), q[t, h // (H // G)].double()
                    S[sl, h] *= float(g[t, h])
                    x = v[t, h * dv:(h + 1) * dv].double()
                    if delta_rule:
                        x = float(beta[t, h]) * (x - S[sl, h] @ kk)
                    S[sl, h] += x[:, None] * kk[None, :]
                    o[t, h] = S[sl, h] @ qq
                t += 1
        want = pg.rms_div(o, 1e-4) * norm.double() * 0.7
        want = want.reshape(T, H * dv) * pg.silu(gate[:, :H * dv].double())
        ctx = _step(lens, slots)
        state = state0.to(DEV)
        out = torch.zeros((T, H * dv + 2), device=DEV)
        args = lambda a, b: (pad(q[a:b]), pad(k[a:b]), v[a:b].to(DEV)[:, :H * dv], g[a:b].to(DEV).contiguous(),
                             beta[a:b].to(DEV).contiguous() if delta_rule else None, H, d, dv)
        kernels.linear_scan(*args(0, T), state, off, ctx, True, gate.to(DEV)[:, :H * dv], norm.to(DEV), 1e-4, 0.7, out[:, :H * dv])
        # an output is divided by its own head's length, the state grows with the tokens: relative to the largest
        assert float((out[:, :H * dv].cpu().double() - want).abs().max()) <= 2e-4 * float(want.abs().max())
        assert not out[:, H * dv:].any()
        got = state.cpu().double()
        full = state0.double().clone()
        full[:, off:off + H * d * dv] = S.reshape(5, -1)
        assert float((got - full).abs().max()) <= 2e-5 * float(full.abs().max())
        for sl in set(range(5)) - set(slots):
            assert torch.equal(got[sl], state0[sl].double())
        assert torch.equal(got[:, :off], state0[:, :off].double()) and torch.equal(got[:, off + H * d * dv:], state0[:, off + H * d * dv:].double())
        if lens == [70]:                                        # cut into 1 + 20 + 49: the same state and outputs
            st2, out2 = state0.to(DEV), torch.zeros_like(out)
            for a, b in ((0, 1), (1, 21), (21, 70)):
                kernels.linear_scan(*args(a, b), st2, off, _step([b - a], slots), True, gate.to(DEV)[a:b, :H * dv], norm.to(DEV), 1e-4,
                                    0.7, out2[a:b, :H * dv])
            assert float((st2 - state).abs().max()) <= 1e-5 * float(full.abs().max())
            assert float((out2 - out).abs().max()) <= 1e-4 * float(want.abs().max())
            assert not torch.equal(st2, state0.to(DEV))
            kernels.linear_scan(*args(0, T), st2, off, ctx, False, gate.to(DEV)[:, :H * dv], None, 1e-4, 0.7, out2[:, :H * dv])
            assert float((st2 - state).abs().max()) <= 1e-5 * float(full.abs().max())      # a run that does not write


@pytest.mark.parametrize("T", [1, 5, 8])
def test_biases_in_the_few_token_feed_forward_kernels(T, guard_regions):
    """Gate, up and down biases through every form that takes a few tokens, and through the library products."""
    from qwen_decoder_b200 import kernels
    from qwen_decoder_b200.parts.mlp import SwiGLU
    from qwen_decoder_b200.weights.loader import TensorSource
    for D, F, n in ((256, 1536, T), (2304, 512, T), (128, 264, 16), (512, 640, 12), (256, 512, 100), (96, 40, 70)):
        gen = torch.Generator().manual_seed(D + F + n)
        part = SwiGLU(D, F, prefix="", names=("gate", "up", "down"), weight_suffix="", bias=True, bias_suffix=".b")
        w = {s.name: (torch.randn(s.shape, generator=gen) * (0.5 if s.name.endswith(".b") else 0.05)).bfloat16() for s in part.tensor_specs()}
        x = torch.randn((n, D), generator=gen).bfloat16()
        want = pg.gated_ff(x.double(), {k: v.double() for k, v in w.items()}, "")
        for dt, tol in ((torch.bfloat16, 2e-2), (torch.float32, 1e-5)):
            part.bind(TensorSource.from_dict(w), dt, torch.device(DEV))
            delta, bias = part.forward_without_bias(x.to(DEV, dt), None)
            got = (delta.double().sum(0) if delta.dim() == 3 else delta.double()) + bias.double()
            assert float((got.cpu() - want).abs().max()) <= tol * float(want.abs().max())
            assert torch.allclose(part.forward(x.to(DEV, dt), None).double().cpu(), got.cpu(), rtol=1e-3, atol=1e-3)
    gen = torch.Generator().manual_seed(3)
    p, b = torch.randn((3, T, 80), generator=gen), torch.randn((80,), generator=gen)
    out = torch.empty((T, 40), dtype=torch.bfloat16, device=DEV)
    kernels.swiglu_partial(p.to(DEV), out, b.to(DEV))
    z = p.double().sum(0) + b.double()
    assert torch.allclose(out.cpu().double(), pg.silu(z[:, :40]) * z[:, 40:], rtol=1e-2, atol=1e-2)


# ------------------------------------------------------------------------------------------------- each mechanism alone
L, R = gc.left(2, 1, 8, 8, 30), gc.right(2, 16, 8)
ONE_LAYER = {
    # name: (mixer, feed-forward, width, groups); a scale of 0 leaves one side of a parallel mixer out
    "blocks_of_five": (gc.par(gc.left(4, 2, 16, 24, 5, factor=3.0, scale=0.6), R, right_scale=0.0), None, 64, 4),
    "blocks_of_a_page_part_rotated": (gc.par(gc.left(2, 2, 24, 8, 16, rot_dims=12, base=50.0), R, right_scale=0.0), None, 64, 1),
    "blocks_of_sixty_four_wide_heads": (gc.par(gc.left(2, 1, 128, 64, 64, factor=8.0, scale=0.06), R, right_scale=0.0), None, 64, 2),
    "blocks_of_one": (gc.par(gc.left(3, 3, 10, 6, 1), R, right_scale=0.0), None, 66, 3),
    "blocks_longer_than_the_prompt_many_heads": (gc.par(gc.left(40, 2, 8, 16, 1000, rot_dims=4), R, right_scale=0.0), None, 48, 4),
    "a_head_of_odd_size_without_rotation": (gc.par(dict(gc.left(2, 1, 9, 7, 40), rot=None), R, right_scale=0.0), None, 40, 4),
    "a_stretch_of_one": (gc.par(gc.left(2, 2, 8, 8, 33, factor=1.0, base=20.0), R, right_scale=0.0), None, 64, 8),
    "retention_one_head": (gc.par(L, gc.right(1, 64, 64), left_scale=0.0), None, 64, 4),
    "retention_part_rotated_values_larger": (gc.par(L, gc.right(3, 24, 40, rot_dims=10, base=30.0), left_scale=0.0, right_scale=1.7), None, 64, 4),
    "retention_decays_of_0_and_1": (gc.par(L, gc.right(4, 8, 12, decay=[0.0, 1.0, 0.5, 0.999]), left_scale=0.0), None, 64, 4),
    "retention_heads_of_136": (gc.par(L, gc.right(1, 136, 8), left_scale=0.0, right_scale=0.3), None, 64, 4),
    "retention_without_rotation_odd": (gc.par(L, dict(gc.right(2, 17, 9), rot=None), left_scale=0.0), None, 36, 3),
    "side_by_side": (gc.par(gc.left(3, 1, 24, 8, 33), gc.right(3, 24, 16), 0.7, 1.4), None, 72, 4),
    "delta_four_taps": (gc.delta(4, 2, 16, 24, 4), None, 64, 4),
    "delta_one_tap_one_head": (gc.delta(1, 1, 40, 8, 1), None, 64, 4),
    "delta_two_taps_many_values_per_key_head": (gc.delta(8, 1, 12, 20, 2), None, 64, 4),
    "delta_seven_taps_odd_sizes": (gc.delta(3, 3, 21, 13, 7), None, 60, 5),
    "delta_wide_heads": (gc.delta(2, 2, 128, 96, 4), dict(kind="dense", ff=32), 64, 4),
    "delta_heads_of_200": (gc.delta(2, 1, 200, 24, 3), None, 64, 4),
    "dense": (gc.par(L, R), gc.dense(88), 64, 4),
    "dense_odd": (gc.delta(2, 2, 8, 8, 2), gc.dense(50), 100, 10),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_each_mechanism_alone(name, dtype, tmp_path):
    """One layer: a prompt at once, in portions, and its tail token by token."""
    mix, mlp, width, groups = ONE_LAYER[name]
    cfg = gc.one_layer(mix, mlp, width=width, groups=groups)
    folder = gc.make_folder(cfg, str(tmp_path / "m"), seed=sum(map(ord, name)), std=0.15)
    cfg, w = gc.read_folder(folder)
    rng = random.Random(len(name))
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1, 2, 37, 90)]
    run_all_ways(folder, dtype, seqs, expected(cfg, w, seqs), tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_whole_and_decode_tail(models, name, dtype, tmp_path):
    folder, cfg, w, seqs, want = models[name]
    runner = make_runner(folder, dtype, held(seqs), page_size=32 if name == "B" else 16)
    for k, tr in enumerate((trace_tools.whole(seqs), trace_tools.decode_tail(seqs, tail=40))):
        run(runner, tr, want, dtype, tmp_path / f"o{k}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_down_to_two_tokens(models, name, dtype, tmp_path):
    folder, cfg, w, seqs, want = models[name]
    runner = make_runner(folder, dtype, held(seqs), page_size=16 if name == "B" else 24)     # 24: no divisor of a key tile
    for k, sizes in enumerate(((7, 2, 24, 3, 2, 16, 5, 2, 31, 2), (2,), (64, 1, 3), (1, 1, 2, 1))):
        run(runner, trace_tools.portions(seqs, sizes=sizes), want, dtype, tmp_path / f"o{k}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype, tmp_path):
    """Unequal requests side by side, portions beside single tokens, in a pool of about two of the longest with three
    state slots: every page and every slot serves several requests in turn.  A key read from a page's former owner, a
    recurrent state or a convolution's kept inputs left over from a slot's former owner show against the statement."""
    folder, cfg, w, seqs, want = models[name]
    seqs2, want2 = seqs + seqs[::-1], want + want[::-1]
    max_tokens = 2 * held(seqs)
    runner = make_runner(folder, dtype, max_tokens, max_requests=3)
    tr = trace_tools.mixed(seqs2, max_tokens, seed=11, max_live=3)
    assert sum(len(s["entries"]) > 1 for s in tr.steps) > 5
    run(runner, tr, want2, dtype, tmp_path)
    all_free(runner)


def test_a_request_alone_and_in_a_batch_agree(models, tmp_path):
    """float32: the same rows from a batch of unequal requests and from each request alone differ by rounding
    of sums at most (far less than from the plain statement)."""
    folder, cfg, w, seqs, want = models["A"]
    runner = make_runner(folder, "float32", 4 * held(seqs))
    a = trace_tools.whole(seqs)
    ga = trace_tools.run_inprocess(runner, a, str(tmp_path / "a"))
    b = trace_tools.mixed(seqs, 4 * held(seqs), seed=3, max_live=4)
    gb = trace_tools.run_inprocess(runner, b, str(tmp_path / "b"))
    rows_a = {rp: ga[s][i] for s, rows in a.expect.items() for i, rp in enumerate(rows)}
    rows_b = {rp: gb[s][i] for s, rows in b.expect.items() for i, rp in enumerate(rows)}
    scale = max(float(np.abs(x).max()) for x in want)
    assert max(float(np.abs(rows_a[k] - rows_b[k]).max()) for k in rows_b) <= 3e-6 * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_and_first_tokens(models, name, dtype, tmp_path):
    """Two tokens of prompt, then 300 tokens one by one across many pages, blocks and key tiles: the states are carried
    300 times; the first positions are compared one by one."""
    folder, cfg, w, _, _ = models[name]
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
    d = np.abs(pg.forward(c, ww, seq).numpy() - want).max(axis=-1)
    return d > 3 * TOL["float32"] * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_keys_at_the_edges_of_blocks(dtype, tmp_path, monkeypatch):
    """Scores sharpened so that single keys (or the one in the denominator) take most of the weight: prompts that end just
    before, at and just after page, key-tile and block borders, their tails decoded token by token.  The statement is
    shown to depend on the edge and on the one."""
    f = 1.0 if dtype == "float32" else 0.45
    cfg = gc.one_layer(gc.par(gc.left(4, 2, 16, 40, 96, base=200.0, factor=4.0, scale=1.0), gc.right(1, 8, 8), right_scale=0.0),
                       None, vocab=400, width=48)

    def sharpen(t):
        t["l0.mix.left.q"] = (t["l0.mix.left.q"].float() * 0.8 * f).to(torch.bfloat16)
    folder = gc.make_folder(cfg, str(tmp_path / "m"), seed=5, std=0.2, edit=sharpen)
    cfg, w = gc.read_folder(folder)
    rng = random.Random(8)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (95, 96, 97, 193, 400)]
    want = expected(cfg, w, seqs)
    bigger = lambda c: c["layers"][0]["mixer"]["left"]["mask"].__setitem__("size", 97)
    assert moved(cfg, w, seqs[-1], want[-1], change_cfg=bigger).mean() > 0.1
    with monkeypatch.context() as m:
        m.setattr(pg, "softmax_plus_one", lambda s, mask: torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1))
        assert moved(cfg, w, seqs[-1], want[-1]).mean() > 0.1
    runner = make_runner(folder, dtype, 512)
    for i, tr in enumerate((trace_tools.whole(seqs), trace_tools.decode_tail(seqs, tail=36),
                            trace_tools.portions(seqs, sizes=(100, 2, 3, 64)))):
        run(runner, tr, want, dtype, tmp_path / f"o{i}")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["retention", "delta"])
def test_a_token_far_back_in_the_state(kind, dtype, tmp_path):
    """One token hundreds of positions back whose write stays readable: slow decays, and a key and value that stand out.
    The statement's logits at the end depend on that token; a state lost, reset or left over on the way shows."""
    if kind == "retention":
        mix = gc.par(gc.left(1, 1, 8, 8, 4), gc.right(2, 16, 24, rot_dims=2, base=1e9, decay=[0.999, 0.9999]), left_scale=0.0)
    else:
        mix = gc.delta(4, 2, 24, 16, 4)
    cfg = gc.one_layer(mix, None, vocab=300, width=48)

    def edit(t):
        if kind == "delta":                         # decays near 1 and small step sizes: writes last
            t["l0.mix.A_log"].fill_(-3.0)
            t["l0.mix.dt_bias"].fill_(-4.0)
            t["l0.mix.b"] *= 0.1
        v = "l0.mix.right.v" if kind == "retention" else "l0.mix.v"
        for tok in range(300):                      # one channel belongs to token 7 alone; the values read it strongly
            t["embed"][tok][0] = 30.0 if tok == 7 else 0.0
        t[v][:, 0] = t[v][:, 0] * 8.0
        t[v][:, 1:] = t[v][:, 1:] * 0.1             # everyone else writes little
    folder = gc.make_folder(cfg, str(tmp_path / "m"), seed=9, std=0.2, edit=edit)
    cfg, w = gc.read_folder(folder)
    rng = random.Random(6)
    seq = [rng.choice([x for x in range(300) if x != 7]) for _ in range(420)]
    seq[33] = 7
    seqs = [seq, seq[:330]]
    want = expected(cfg, w, seqs)
    other = list(seq)
    other[33] = 8
    d = np.abs(pg.forward(cfg, w, other).numpy()[300:] - want[0][300:]).max(axis=-1)
    assert (d > 2 * np.maximum(TOL[dtype] * np.abs(want[0]).max(), want.allow[dtype][0][300:])).mean() > 0.3
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=448, tail=60, sizes=(100, 2, 3, 64, 1))
    runner = make_runner(folder, dtype, 2 * 448, max_requests=2)
    tr = trace_tools.mixed(seqs + seqs[::-1], 2 * 448, seed=2, max_live=2, portion_sizes=(2, 9, 40))
    run(runner, tr, want + want[::-1], dtype, tmp_path / "mixed")
    all_free(runner)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoding_over_a_long_block(dtype, tmp_path):
    """A thousand keys of the query's own block behind each decoded token: its keys are shared among many CTAs whose
    partial results (values of a size that is no multiple of a warp) are added up with the one in the denominator and
    gated element by element; alone and side by side."""
    cfg = gc.one_layer(gc.par(gc.left(4, 2, 32, 40, 1060, base=5000.0, scale=0.9), gc.right(2, 16, 16), 1.0, 0.5), None, vocab=150)
    folder = gc.make_folder(cfg, str(tmp_path / "m"), seed=12, std=0.15)
    cfg, w = gc.read_folder(folder)
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


# -------------------------------------------------------------------------------------------------- the engine around it
def test_one_product_for_both_sides_and_two_agree(models, tmp_path, monkeypatch):
    """The two sides of a parallel mixer read one stacked product; with a product of their own each they give the same."""
    from qwen_decoder_b200.parts.side_by_side import SideBySide
    folder, cfg, w, seqs, want = models["A"]
    outs = []
    for shared in (True, False):
        runner = make_runner(folder, "float32", held(seqs))
        sides = [layer.mixer for layer in runner.model.layers if isinstance(layer.mixer, SideBySide)]
        assert len(sides) == 3 and all(s.inp is not None for s in sides)
        if not shared:
            for s in sides:
                for m in s.mixers:
                    m.stacked = m.stacked.clone()
                monkeypatch.setattr(s, "inp", None)
        outs.append(run(runner, trace_tools.decode_tail(seqs, tail=10), want, "float32", tmp_path / f"o{shared}"))
    scale = max(float(np.abs(x).max()) for x in want)
    assert max(float(np.abs(outs[0][s] - outs[1][s]).max()) for s in outs[0]) <= 3e-6 * scale


def test_greedy_generation_through_the_engine(models):
    """``Engine.generate`` (scheduler, portions of prompts, batched decoding as replayed graphs, the sampler's
    argmax) against greedy decoding with the plain statement, for prompts of unequal length at once."""
    from qwen_decoder_b200.engine import Engine, SamplingParams
    folder, cfg, w, seqs, _ = models["A"]
    prompts = [seqs[2], seqs[5][:20], seqs[4], seqs[1], seqs[9][:50]]
    new = 12
    engine = Engine(folder, dtype="float32", max_batch=3, max_prefill_tokens_per_step=24, max_total_tokens=64,
                    num_pages=40, page_size=16, max_positions=256)
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    for prompt, out in zip(prompts, outs):
        seq = list(prompt)
        for _ in range(new):
            logits = pg.forward(cfg, w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            assert float(top2[0] - top2[1]) > 1e-4, "a close call: choose another seed for this test"
            seq.append(int(torch.argmax(logits)))
        assert out == seq[len(prompt):]
    all_free(engine.runner)
    # bfloat16 with replayed graphs: every token the engine chose is, for the statement, the best one or within the
    # rounding of it (a near-tie may go either way, after which the statement follows the engine's sequence)
    e16 = Engine(folder, dtype="bfloat16", max_batch=4, max_prefill_tokens_per_step=32, max_total_tokens=64,
                 num_pages=40, page_size=16, max_positions=256)
    for prompt, out in zip(prompts, e16.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))):
        seq = list(prompt)
        assert len(out) == new
        for tok in out:
            logits = pg.forward(cfg, w, seq)[-1]
            assert float(logits.max() - logits[tok]) <= 2 * TOL["bfloat16"] * float(logits.abs().max())
            seq.append(tok)
    all_free(e16.runner)


def test_the_programs_take_the_folder(models, tmp_path):
    """``bin/decoder_main`` and ``bin/trace_run`` as separate processes on a Gopevik folder: the command line's greedy
    tokens are the statement's, and a replayed trace with four live requests in a small pool gives its logits."""
    import os
    import subprocess
    import sys
    root = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..")
    folder, cfg, w, seqs, want = models["A"]
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
            logits = pg.forward(cfg, w, seq)[-1]
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
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_models_drawn_at_random(seed, dtype, tmp_path):
    """Layers of either kind in any order with sizes, taps, blocks, decays, constants and feed-forwards drawn anew for
    every layer: whole, in portions, with decoded tails, and as mixed batches in a small pool with three state slots."""
    cfg = gc.drawn(seed)
    folder = gc.make_folder(cfg, str(tmp_path / "m"), seed=100 + seed, std=0.13, edit=gc.steady)
    cfg, w = gc.read_folder(folder)
    rng = random.Random(seed)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1, 2, 19, 64, 65, 141)]
    want = expected(cfg, w, seqs)
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=192, tail=30, page_size=16 if seed % 2 else 32)
    max_tokens = 2 * held(seqs)
    runner = make_runner(folder, dtype, max_tokens, max_requests=3)
    tr = trace_tools.mixed(seqs + seqs[::-1], max_tokens, seed=seed, max_live=3)
    run(runner, tr, want + want[::-1], dtype, tmp_path / "mixed")
    all_free(runner)


LARGER = gc.config(420, 192, 1e-5, 6, [
    (gc.par(gc.left(6, 2, 128, 96, 256, rot_dims=64, base=2e5), gc.right(3, 64, 128), 1.1, 0.9), gc.dense(320)),
    (gc.delta(8, 4, 64, 96, 4), gc.dense(256)),
    (gc.par(gc.left(4, 4, 64, 128, 100, factor=2.0), gc.right(2, 128, 64, rot_dims=32)), None),
    (gc.delta(6, 2, 128, 64, 3), None),
])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_larger_model_with_long_prompts(dtype, tmp_path):
    """Heads of 128 and 64 with values of 96, 128 and 64, prompts of up to 700 tokens over blocks of 256 and 100: several
    key tiles per query tile, single tokens whose keys are shared among CTAs, every way of cutting, and a mixed batch in a
    small pool."""
    folder = gc.make_folder(LARGER, str(tmp_path / "m"), seed=31, std=0.1, edit=gc.steady)
    cfg, w = gc.read_folder(folder)
    rng = random.Random(14)
    seqs = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (700, 257, 384, 129, 513)]
    want = expected(cfg, w, seqs)
    run_all_ways(folder, dtype, seqs, want, tmp_path, max_tokens=704, tail=40, sizes=(100, 2, 3, 64, 200, 7))
    runner = make_runner(folder, dtype, 1408, max_requests=3, page_size=32)
    tr = trace_tools.mixed(seqs, 1408, seed=5, max_live=3, prompt_frac=0.8, portion_sizes=(2, 9, 33, 64, 130))
    run(runner, tr, want, dtype, tmp_path / "mixed")
    all_free(runner)
