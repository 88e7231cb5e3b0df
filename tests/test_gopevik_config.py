"""Gopevik's configuration, description, cache layout, position tables, and what its parts refuse (no GPU)."""
import copy

import pytest
import torch

import gopevik_configs as gc
import plain_gopevik as pg
from qwen_decoder_b200.cache import CacheManager, FixedState, PagedKV
from qwen_decoder_b200.config import ConfigError, config_from_dict, describe_model
from qwen_decoder_b200.parts.linear import pad_rows
from qwen_decoder_b200.parts.linear_attention import LinearAttention
from qwen_decoder_b200.parts.masked_attention import MaskedAttention
from qwen_decoder_b200.parts.model import build_model
from qwen_decoder_b200.parts.norm import GroupRMSNorm
from qwen_decoder_b200.parts.rotary import Rotary


def test_round_trip_and_description():
    cfg = config_from_dict(gc.GA)
    assert cfg.architecture == "Gopevik" and cfg.vocab_size == 310 and cfg.hidden_size == 96 and cfg.norm_groups == 3
    assert config_from_dict(cfg.to_dict()) == cfg
    spec = describe_model(cfg)
    assert spec.lm_head_tensor == "head" and [l.block for l in spec.layers] == ["pre_post_norm"] * 5
    assert [l.mixer.name for l in spec.layers] == ["side_by_side", "linear_attention", "side_by_side", "linear_attention", "side_by_side"]
    assert [sorted(l.norms) for l in spec.layers][0] == ["feed_forward_out", "input", "mixer_out", "post_mixer"]
    assert sorted(spec.layers[3].norms) == ["input", "mixer_out"] and spec.layers[3].feed_forward is None
    assert all(n.params["groups"] == 3 for l in spec.layers for n in l.norms.values()) and spec.final_norm.params["groups"] == 3
    l, r = (b["params"] for b in spec.layers[0].mixer.params["branches"])
    assert l["mask"] == "chunk" and l["mask_size"] == 20 and l["sink_score"] == 0.0 and l["output_gate"] == "element"
    assert r["decay"] == tuple(gc.decays(2)) and r["k_scale"] == pytest.approx(24 ** -0.5) and not r.get("delta_rule")
    assert [b["scale"] for b in spec.layers[0].mixer.params["branches"]] == [0.8, 1.3]
    names = {s.name: tuple(s.shape) for s in build_model(spec).tensor_specs()}
    assert names["l0.mix.left.q"] == (96, 96) and names["l0.mix.left.k"] == (48, 96) and names["l0.mix.left.v"] == (72, 96)
    assert names["l0.mix.left.g"] == (6 * 24, 96) and names["l0.mix.left.o"] == (96, 6 * 24)
    assert names["l0.mix.right.q"] == names["l0.mix.right.k"] == (48, 96) and names["l0.mix.right.v"] == (80, 96)
    assert names["l0.mix.right.g"] == (80, 96) and names["l0.mix.right.o"] == (96, 80)
    assert names["l1.mix.q"] == (40, 96) and names["l1.mix.v"] == (144, 96) and names["l1.mix.v.conv"] == (144, 2)
    assert names["l1.mix.b"] == names["l1.mix.a"] == (6, 96) and names["l1.mix.A_log"] == names["l1.mix.dt_bias"] == (6,)
    assert names["l1.mix.norm"] == (24,) and names["l1.mix.g"] == (144, 96) and names["l1.mix.o"] == (96, 144)
    assert names["l1.mlp.gate.b"] == (56,) and names["l1.mlp.down.b"] == (96,) and names["l1.mlp.down"] == (96, 56)
    assert "l3.norm2" not in names and "l3.norm2b" not in names and names["l3.norm1b"] == (96,)
    assert names["final.norm"] == (96,) and names["head"] == (310, 96) and names["embed"] == (310, 96)
    assert "l0.mix.right.norm" not in names and "l0.mix.right.A_log" not in names and "l0.mix.left.q.b" not in names


def test_cache_layout_pages_and_state_rows():
    layout = build_model(describe_model(config_from_dict(gc.GA))).cache_layout()
    assert [g.need for g in layout.groups] == [PagedKV(3, 16, None, v_dim=24), PagedKV(1, 24, None, v_dim=8), PagedKV(2, 32, None, v_dim=32)]
    pad4 = lambda n: (n + 3) // 4 * 4
    assert layout.fixed_needs == [FixedState((2 * 24 * 40,)), FixedState((pad4(6 * 20 * 24 + 1 * (2 * 40 + 144)),)),
                                  FixedState((5 * 8 * 16,)), FixedState((pad4(3 * 40 * 8 + 4 * (2 * 120 + 24)),)), FixedState((64 * 12,))]
    assert sorted(layout.paged) == [0, 2, 4] and sorted(layout.fixed) == [0, 1, 2, 3, 4]
    cm = CacheManager(layout, num_pages=8, page_size=16, max_requests=2)
    a = cm.open("a")
    cm.ensure(a, 40)
    cm.commit(a, 40)
    cm.close(a)
    cm.check()


def test_tables_of_evenly_stretched_positions():
    part = Rotary(head_dim=32, rotary_dim=24, base=500.0, pairing="half", scaling={"kind": "linear", "factor": 2.5})
    part.prepare(300, torch.device("cpu"))
    x = torch.randn((300, 2, 32), dtype=torch.float64)
    want = pg.turn(x, {"base": 500.0, "dims": 24, "scaling": {"factor": 2.5}})
    cos, sin = part.cos.double()[:, None], part.sin.double()[:, None]
    u, v = x[..., :12], x[..., 12:24]
    assert torch.allclose(u * cos - v * sin, want[..., :12], atol=1e-5)
    assert torch.allclose(v * cos + u * sin, want[..., 12:24], atol=1e-5)
    with pytest.raises(ValueError):
        Rotary(head_dim=8, rotary_dim=8, base=10.0, scaling={"kind": "linear", "factor": 0.0})


def test_padded_rows():
    w = torch.randn(11, 4)
    p = pad_rows(w, 8)
    assert p.shape == (16, 4) and torch.equal(p[:11], w) and not p[11:].any()
    assert pad_rows(p, 8).shape == (16, 4)


def test_parts_refuse_what_they_cannot_run():
    with pytest.raises(ValueError):
        GroupRMSNorm(10, 1e-5, groups=4)
    with pytest.raises(ValueError):
        LinearAttention(64, 4, 16, num_kv_heads=3)
    with pytest.raises(ValueError):
        LinearAttention(64, 4, 16, decay=[0.9])
    with pytest.raises(ValueError):
        LinearAttention(64, 1, 300)
    with pytest.raises(ValueError):
        MaskedAttention(64, 2, 2, 8, output_gate="row")


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("mask"), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("decay"), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("decay", [0.9]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"]["rot"].__setitem__("scaling", {"factor": 2.0}), "scaling"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["norm"].pop("groups"), "groups"),
    (lambda c: c["norm"].__setitem__("groups", 7), "groups"),
    (lambda c: c.pop("norm"), "eps"),
])
def test_errors_name_the_key(edit, word):
    cfg = copy.deepcopy(gc.GA)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert word in str(e.value)


def test_the_statement_sees_its_own_mechanisms():
    """The statement's parts against hand-made cases: a block's edge, the one in the softmax's denominator, the order of
    decay, write and read in the recurrences."""
    mask = pg.same_block(5, 2)
    assert mask.tolist() == [[True, False, False, False, False], [True, True, False, False, False], [False, False, True, False, False],
                             [False, False, True, True, False], [False, False, False, False, True]]
    s = torch.tensor([[0.0, 1.0], [50.0, -60.0]], dtype=torch.float64)
    p = pg.softmax_plus_one(s, torch.ones(2, 2, dtype=torch.bool))
    e = torch.exp(s[0])
    assert torch.allclose(p[0], e / (1 + e.sum())) and p[1, 0] == pytest.approx(1.0)
    # one head of size 1: S_t = 0.5 S_(t-1) + k v, read after the write
    w = {"q": [[1.0]], "k": [[1.0]], "v": [[1.0]], "g": [[1.0]], "o": [[1.0]]}
    w = {k: torch.tensor(v, dtype=torch.float64) for k, v in w.items()}
    h = torch.tensor([[1.0], [2.0]], dtype=torch.float64)
    y = pg.retention(h, {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, w, "", 1e-3)
    o = torch.tensor([1.0, 2.0 * (0.5 * 1.0 + 4.0)], dtype=torch.float64)
    assert torch.allclose(y[:, 0], o / torch.sqrt(o * o + 1e-3) * pg.silu(h[:, 0]))
