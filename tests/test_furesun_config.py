"""Furesun's configuration, description, cache layout, position tables, what its parts refuse, and the statement's own
mechanisms against hand-made cases (no GPU)."""
import copy
import math

import pytest
import torch

import furesun_configs as fc
import plain_furesun as pf
from qwen_decoder_b200.cache import CacheManager, FixedState, PagedKV, PagedRows
from qwen_decoder_b200.config import ConfigError, config_from_dict, describe_model
from qwen_decoder_b200.parts.block import PostNormBlock
from qwen_decoder_b200.parts.linear_attention import LinearAttention
from qwen_decoder_b200.parts.masked_attention import MaskedAttention
from qwen_decoder_b200.parts.model import build_model
from qwen_decoder_b200.parts.norm import RMSNorm
from qwen_decoder_b200.parts.rotary import Rotary


def test_round_trip_and_description():
    cfg = config_from_dict(fc.FA)
    assert cfg.architecture == "Furesun" and cfg.vocab_size == 310 and cfg.hidden_size == 96 and cfg.logit_softcap == 15.0
    assert config_from_dict(cfg.to_dict()) == cfg
    assert config_from_dict(fc.FB).logit_softcap is None and config_from_dict(config_from_dict(fc.FB).to_dict()) == config_from_dict(fc.FB)
    spec = describe_model(cfg)
    assert spec.lm_head_tensor == "head" and spec.logit_softcap == 15.0 and [l.block for l in spec.layers] == ["post_norm"] * 6
    assert [l.mixer.name for l in spec.layers] == ["masked_attention", "linear_attention", "masked_attention", "latent_attention",
                                                   "masked_attention", "linear_attention"]
    assert sorted(spec.layers[0].norms) == ["feed_forward_out", "mixer_out"] and sorted(spec.layers[2].norms) == ["mixer_out"]
    assert [e.cache_of for e in spec.schedule] == [None, None, 0, None, 0, None]
    a, b, c = (spec.layers[i].mixer.params for i in (0, 2, 4))
    assert (a["mask_size"], b["mask_size"], c["mask_size"]) == (20, 37, 5)
    assert a["cache_window"] == b["cache_window"] == c["cache_window"] == 37        # the widest window over these keys
    assert a["sink_score"] == 0.0 and a["softcap"] == 3.0 and a["qk_norm"] == "whole" and not a["shares_kv"] and b["shares_kv"]
    m = spec.layers[1].mixer.params
    assert m["gate_cap"] == 7.0 and m["q_scale"] == pytest.approx(20 ** -0.5) and m["output_gate"] == "sigmoid"
    assert spec.layers[1].feed_forward.params["activation"] == "gelu_tanh"
    e = spec.layers[3].feed_forward.params
    assert e["routing"] == "top_sigmoid_norm" and e["routing_scale"] == 0.7 and e["shared_size"] == 0
    l = spec.layers[3].mixer.params
    assert l["q_rank"] == 0 and l["window"] == 33 and not l["output_gate"] and spec.positions[l["position"]].params["pairing"] == "half"
    names = {s.name: tuple(s.shape) for s in build_model(spec).tensor_specs()}
    assert names["l0.mix.q"] == (96, 96) and names["l0.mix.k"] == (48, 96) and names["l0.mix.v"] == (72, 96)
    assert names["l0.mix.q.norm"] == (96,) and names["l0.mix.k.norm"] == (48,) and names["l0.mix.o"] == (96, 144)
    assert names["l2.mix.q"] == (48, 96) and names["l2.mix.q.norm"] == (48,) and names["l2.mix.o"] == (96, 72)
    assert not [n for n in names if n.startswith(("l2.mix.k", "l2.mix.v", "l4.mix.k", "l4.mix.v"))]
    assert names["l1.mix.i"] == names["l1.mix.f"] == (3, 96) and names["l1.mix.i.b"] == names["l1.mix.f.b"] == (3,)
    assert names["l1.mix.norm"] == (72,) and names["l1.mix.g"] == (72, 96) and "l1.mix.A_log" not in names
    assert names["l3.mix.q"] == (128, 96) and names["l3.mix.dkv"] == (48, 96) and names["l3.mix.dkv.norm"] == (40,)
    assert names["l3.mix.uk"] == (96, 40) and names["l3.mix.uv"] == (64, 40) and names["l3.mix.o"] == (96, 64)
    assert "l3.mix.dq" not in names and "l3.mix.g" not in names
    assert names["l0.mlp.router"] == (5, 96) and names["l0.mlp.e4.down"] == (96, 24) and names["l0.mlp.shared.up"] == (40, 96)
    assert "l0.mlp.router.b" not in names and "l3.mlp.shared.up" not in names and "l2.norm2" not in names
    assert names["final.norm"] == (96,) and names["head"] == (310, 96) and names["l1.norm1"] == names["l1.norm2"] == (96,)


def test_cache_layout_pages_and_state_rows():
    layout = build_model(describe_model(config_from_dict(fc.FA))).cache_layout()
    assert [g.need for g in layout.groups] == [PagedKV(3, 16, 37, v_dim=24), PagedRows(48, 33)]
    assert [g.entries for g in layout.groups] == [[0], [3]] and layout.owners[2] == layout.owners[4] == 0
    pad4 = lambda n: (n + 3) // 4 * 4
    assert layout.fixed_needs == [FixedState((pad4(3 * 25 * 20 + 3),)), FixedState((pad4(2 * 13 * 32 + 2),))]
    cm = CacheManager(layout, num_pages=8, page_size=16, max_requests=2)
    a = cm.open("a")
    cm.ensure(a, 60)
    cm.commit(a, 60)                    # the next token sees positions 24.. of the first group and 28.. of the second
    assert [p.num_free for p in cm.pools] == [5, 5]
    cm.ensure(a, 69)
    cm.commit(a, 9)                     # 33.. and 37..
    assert [p.num_free for p in cm.pools] == [5, 5]
    cm.close(a)
    cm.check()


def test_tables_of_stretched_half_split_positions():
    sc = fc.ramp(8.0, 48, 16.0, 0.7)
    part = Rotary(head_dim=24, rotary_dim=20, base=300.0, pairing="half", scaling=sc)
    part.prepare(200, torch.device("cpu"))
    x = torch.randn((200, 2, 24), dtype=torch.float64)
    want = pf.turn(x, {"base": 300.0, "dims": 20, "scaling": sc}, True)
    cos, sin = part.cos.double()[:, None], part.sin.double()[:, None]
    u, v = x[..., :10], x[..., 10:20]
    assert torch.allclose(u * cos - v * sin, want[..., :10], atol=1e-5) and torch.allclose(v * cos + u * sin, want[..., 10:20], atol=1e-5)
    assert float(part.cos[0, 0]) == pytest.approx(0.1 * math.log(8.0) + 1.0)


def test_parts_refuse_what_they_cannot_run():
    with pytest.raises(ValueError):
        LinearAttention(64, 4, 16, num_kv_heads=2, gate_cap=10.0)
    with pytest.raises(ValueError):
        LinearAttention(64, 2, 16, gate_cap=0.0)
    with pytest.raises(ValueError):
        LinearAttention(64, 2, 16, gate_cap=5.0, decay=[0.9, 0.8])
    with pytest.raises(ValueError):
        LinearAttention(64, 2, 16, decay=[0.9, 0.8], output_gate="tanh")
    with pytest.raises(ValueError):
        MaskedAttention(64, 2, 1, 8, softcap=-1.0)
    with pytest.raises(ValueError):
        MaskedAttention(64, 2, 1, 8, shares_kv=True, conv_taps=2)
    with pytest.raises(ValueError):
        MaskedAttention(64, 2, 1, 8, mask="window", mask_size=9, cache_window=8)
    with pytest.raises(ValueError):
        PostNormBlock(None, None, {})
    with pytest.raises(ValueError):
        PostNormBlock(None, None, {"mixer_out": RMSNorm(8, 1e-5)})



@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("scaling", fc.ramp(2, 3, 4, 1)), "scaling"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), "size"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("softcap", 0.0), "softcap"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("kv_from", 2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("kv_from", 1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].__setitem__("kv_from", 2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("vdim", 8), "vdim"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("gate_cap", -3.0), "gate_cap"),
    (lambda c: c["layers"][3]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][3]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("dims", 10), "dims"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "gated"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_errors_name_the_key(edit, word):
    cfg = copy.deepcopy(fc.FA)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert word in str(e.value)


def test_drawn_models_describe():
    kinds = set()
    for seed in range(1, 13):
        spec = describe_model(config_from_dict(fc.drawn(seed)))
        build_model(spec).cache_layout()
        kinds |= {l.mixer.name for l in spec.layers} | ({"shared"} if any(e.cache_of is not None for e in spec.schedule) else set())
    assert kinds == {"masked_attention", "latent_attention", "linear_attention", "shared"}


def test_the_statement_sees_its_own_mechanisms():
    """The statement's parts against hand-made cases: a window's edge, the one in the denominator, the gates, the running
    maximum and the normaliser, the router's weights."""
    assert pf.window(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False],
                                        [False, False, True, True]]
    s = torch.tensor([[0.0, 1.0], [50.0, -60.0]], dtype=torch.float64)
    p, e = pf.softmax_plus_one(s, torch.ones(2, 2, dtype=torch.bool)), torch.exp(s[0])
    assert torch.allclose(p[0], e / (1 + e.sum())) and p[1, 0] == pytest.approx(1.0)
    # one head of size 1, forget gates of log(1/2), input gates of 0: S_t = S_(t-1) / 2 + k v in true terms, n alike
    one = lambda v: torch.tensor([[v]], dtype=torch.float64)
    cap, half = 40.0, 0.0                                           # logsigmoid(0) = log(1/2)
    w = {"q": one(1.0), "k": one(1.0), "v": one(1.0), "g": one(1.0), "o": one(1.0), "norm": one(1.0)[0],
         "i": one(0.0), "f": one(0.0), "i.b": one(0.0)[0], "f.b": one(half)[0]}
    h = torch.tensor([[1.0], [2.0], [-3.0]], dtype=torch.float64)
    y = pf.mlstm(h, {"heads": 1, "dim": 1, "vdim": 1, "gate_cap": cap}, w, "", 0.7, {})
    S = n = 0.0
    want = []
    for x in (1.0, 2.0, -3.0):
        S, n = 0.5 * S + x * x, 0.5 * n + x
        o = S * x / max(abs(n * x), 1.0)                            # in true terms the floor is 1, the 1e-6 next to nothing
        want.append(o / math.sqrt(o * o + 0.7) / (1 + math.exp(-x)))
    assert torch.allclose(y[:, 0], torch.tensor(want, dtype=torch.float64), rtol=1e-5)
    # the router: the two largest of three, their sigmoids over their sum, times the constant
    x = torch.tensor([[1.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[0.0], [2.0], [-1.0]], dtype=torch.float64)}
    for i in range(3):
        w |= {f"e{i}.gate": one(1.0), f"e{i}.up": one(float(i + 1)), f"e{i}.down": one(1.0)}
    a, b = 0.5, 1 / (1 + math.exp(-2.0))
    y = pf.experts(x, {"router": {"top": 2, "scale": 3.0}}, w, "")
    assert float(y) == pytest.approx(3.0 * (a * 1 + b * 2) / (a + b) * float(pf.silu(x)))
