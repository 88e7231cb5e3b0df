"""``Furesun``: a decoder whose ``config.json`` lists its layers one by one.

A layer has a norm after each branch and none before it: the branches read the residual sum itself,
x += n1(mixer(x)), x += n2(ff(x)) (a layer whose ``mlp`` is null ends after the mixer).  Three mixers:

* ``latent_attention``: keys and values of all heads expanded from one cached row per token; no query latent; a rotated
  part of half-split pairs, shared by the heads' keys, at rates stretched by ``rot.scaling``; the last ``mask.size`` keys;
* ``attention``: grouped queries; q and k normed over the whole projection; adjacent pairs turn; scores capped by tanh; the
  last ``mask.size`` keys; one added to the softmax's denominator.  A layer with ``kv_from``: j has no keys and values of its
  own and reads those of layer j;
* ``mlstm``: a matrix memory per head with exponential gates, a running maximum and a normaliser; every head's output
  divided by its root mean square, times weights over all heads, gated by a sigmoid.

Feed-forwards: dense gated by gelu (its tanh form), routed experts gated by silu (the largest sigmoid scores, divided by
their sum, times a constant) with an optional shared expert, or none.  The logits are capped by tanh.

Keys read from ``config.json``: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` (absent or null: no
cap), ``layers[i].type`` / ``.mixer`` / ``.mlp`` (and, optional, ``max_positions`` and ``eos_token_id``).  Tensor names:
``embed``, ``head``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``; linear weights are [out, in] with
no suffix, the gates' biases ``l<i>.mix.i.b|f.b``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .veterax import DEFAULT_MAX_POSITIONS, _need

_MIXER_SIZES = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank"),
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "mlstm": ("heads", "dim", "vdim"),
}
_RAMP = ("factor", "original", "fast", "slow")


def _positive(d, key: str, where: str) -> float:
    v = _need(d, key, where, float)
    if v <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _check_rot(rot, dim: int, where: str, scaling: bool) -> None:
    if rot is None:
        return
    dims = _need(rot, "dims", where)
    _positive(rot, "base", where)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.dims ({dims}) must be even and at most {dim}")
    if rot.get("scaling") is not None:
        if not scaling:
            raise ConfigError(f"config.json: {where}.scaling: this mixer's rotation has no scaling")
        for k in _RAMP:
            _positive(rot["scaling"], k, f"{where}.scaling")


def _check_layer(i: int, layer, layers) -> None:
    where = f"layers[{i}]"
    kind = layer.get("type") if isinstance(layer, Mapping) else None
    if kind not in _MIXER_SIZES:
        raise ConfigError(f"config.json: {where}.type must be one of {sorted(_MIXER_SIZES)}, got {kind!r}")
    m, mw = layer.get("mixer"), f"{where}.mixer"
    for k in _MIXER_SIZES[kind]:
        _need(m, k, mw)
    if kind == "mlstm":
        _positive(m, "gate_cap", mw)
    else:
        _need(m, "scale", mw, float)
        _need(m.get("mask"), "size", f"{mw}.mask")
        _check_rot(m.get("rot"), m["rot_dim"] if kind == "latent_attention" else m["dim"], f"{mw}.rot",
                   kind == "latent_attention")
    if kind == "attention":
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {mw}.kv_heads ({m['kv_heads']}) must divide heads ({m['heads']})")
        if m.get("softcap") is not None:
            _positive(m, "softcap", mw)
        _check_kv_from(i, m, mw, layers)
    _check_mlp(layer.get("mlp"), f"{where}.mlp")


def _check_kv_from(i: int, m, where: str, layers) -> None:
    j = m.get("kv_from")
    if j is None:
        return
    if isinstance(j, bool) or not isinstance(j, int) or not (0 <= j < i):
        raise ConfigError(f"config.json: {where}.kv_from must name an earlier layer, got {j!r}")
    src = layers[j].get("mixer") if layers[j].get("type") == "attention" else None
    if src is None or src.get("kv_from") is not None:
        raise ConfigError(f"config.json: {where}.kv_from: layer {j} has no keys and values of its own")
    for k in ("kv_heads", "dim", "vdim"):
        if m[k] != src[k]:
            raise ConfigError(f"config.json: {where}.kv_from: layer {j} has another {k} ({src[k]}, here {m[k]})")


def _check_mlp(f, where: str) -> None:
    if f is None:
        return
    kind = f.get("kind") if isinstance(f, Mapping) else None
    if kind == "dense":
        _need(f, "ff", where)
        return
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind must be 'dense' or 'moe', got {kind!r}")
    _need(f.get("expert"), "ff", f"{where}.expert")
    r = f.get("router")
    e, top = _need(r, "experts", f"{where}.router"), _need(r, "top", f"{where}.router")
    _need(r, "scale", f"{where}.router", float)
    if top > e:
        raise ConfigError(f"config.json: {where}.router.top ({top}) exceeds experts ({e})")
    if f.get("shared"):                         # absent, null or empty: no shared expert
        _need(f["shared"], "ff", f"{where}.shared")


@dataclass(frozen=True)
class FuresunConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[dict, ...]
    logit_softcap: Optional[float] = None
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()
    extra: dict = field(default_factory=dict, compare=False, hash=False)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "FuresunConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        for i, layer in enumerate(layers):
            _check_layer(i, layer, layers)
        cap = d.get("logit_softcap")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
        return cls(architecture=d.get("architecture") or d["architectures"][0],
                   vocab_size=_need(d, "vocab", "config"), hidden_size=_need(d, "width", "config"),
                   norm_eps=_positive(d.get("norm"), "eps", "norm"),
                   layers=tuple(copy.deepcopy(layer) for layer in layers),
                   logit_softcap=_positive(d, "logit_softcap", "config") if cap is not None else None,
                   max_position_embeddings=d.get("max_positions") or DEFAULT_MAX_POSITIONS, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [copy.deepcopy(layer) for layer in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d


def _position(positions: dict, rot, dim: int, pairing: str) -> Optional[str]:
    """The name under which the model keeps a rotation's tables (mixers with equal rotations share them)."""
    if rot is None:
        return None
    sc = rot.get("scaling")
    name = f"{pairing}{rot['dims']}of{dim}b{rot['base']!r}" + ("s" + "/".join(repr(sc[k]) for k in _RAMP) if sc else "")
    positions.setdefault(name, PartSpec("rotary", {
        "head_dim": dim, "rotary_dim": rot["dims"], "base": rot["base"], "pairing": pairing,
        "scaling": {k: sc[k] for k in _RAMP} if sc else None}))
    return name


def _mixer(cfg: FuresunConfig, i: int, kind: str, m: Mapping, positions: dict) -> PartSpec:
    common = {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "v_dim": m["vdim"], "eps": cfg.norm_eps,
              "prefix": "mix.", "weight_suffix": ""}
    if kind == "mlstm":
        return PartSpec("linear_attention", {
            **common, "head_dim": m["dim"], "q_scale": m["dim"] ** -0.5, "gate_cap": m["gate_cap"], "norm_weight": "all",
            "output_gate": "sigmoid"})
    if kind == "latent_attention":
        return PartSpec("latent_attention", {
            **common, "nope_dim": m["dim"], "rope_dim": m["rot_dim"], "q_rank": 0, "kv_rank": m["kv_rank"], "scale": m["scale"],
            "position": _position(positions, m.get("rot"), m["rot_dim"], "half"), "window": m["mask"]["size"],
            "output_gate": False})
    owner = m.get("kv_from") if m.get("kv_from") is not None else i
    reach = max(other["mixer"]["mask"]["size"] for n, other in enumerate(cfg.layers)     # the widest window over these keys
                if other["type"] == "attention" and (n == owner or other["mixer"].get("kv_from") == owner))
    return PartSpec("masked_attention", {
        **common, "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "scale": m["scale"], "qk_norm": "whole",
        "position": _position(positions, m.get("rot"), m["dim"], "adjacent"), "mask": "window", "mask_size": m["mask"]["size"],
        "cache_window": reach, "sink_score": 0.0, "softcap": m.get("softcap"), "shares_kv": m.get("kv_from") is not None})


def _feed_forward(cfg: FuresunConfig, f) -> Optional[PartSpec]:
    if f is None:
        return None
    common = {"hidden_size": cfg.hidden_size, "prefix": "mlp.", "weight_suffix": "", "names": ("gate", "up", "down")}
    if f["kind"] == "dense":
        return PartSpec("swiglu", {**common, "intermediate_size": f["ff"], "activation": "gelu_tanh"})
    shared, r = f.get("shared"), f["router"]
    return PartSpec("moe", {
        **common, "expert_size": f["expert"]["ff"], "num_experts": r["experts"], "top": r["top"], "routing": "top_sigmoid_norm",
        "routing_scale": r["scale"], "router_bias": False, "shared_size": shared["ff"] if shared else 0, "shared_gate": False})


def describe_furesun(cfg: FuresunConfig) -> ModelSpec:
    norm = lambda tensor: PartSpec("group_rmsnorm", {"size": cfg.hidden_size, "eps": cfg.norm_eps, "groups": 1, "tensor": tensor})
    positions, layers, schedule = {}, [], []
    for i, layer in enumerate(cfg.layers):
        ff = _feed_forward(cfg, layer.get("mlp"))
        norms = {"mixer_out": norm("norm1")}
        if ff is not None:
            norms["feed_forward_out"] = norm("norm2")
        layers.append(LayerSpec(prefix=f"l{i}.", block="post_norm",
                                mixer=_mixer(cfg, i, layer["type"], layer["mixer"], positions), feed_forward=ff, norms=norms))
        schedule.append(ScheduleEntry(layer=i, cache_of=layer["mixer"].get("kv_from")))
    return ModelSpec(
        hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size, max_positions=cfg.max_position_embeddings,
        embedding_tensor="embed", positions=positions, layers=layers, schedule=schedule, final_norm=norm("norm"),
        final_norm_prefix="final.", lm_head_tensor="head", logit_softcap=cfg.logit_softcap)


register_architecture("Furesun", FuresunConfig, describe_furesun)
