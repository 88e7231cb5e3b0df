"""``Gopevik``: a decoder whose ``config.json`` lists its layers one by one.

A layer has a norm before and a norm after each branch, x += n1b(mixer(n1(x))), x += n2b(ff(n2(x))) (a layer whose ``mlp``
is null ends after the mixer).  Every norm is an RMS norm in ``norm.groups`` equal parts of the row.  Two mixers:

* ``parallel``: ``left_scale`` * left + ``right_scale`` * right on the same input.  left is grouped-query attention with
  half-split rotary pairs at rates divided by ``rot.scaling.factor``, keys of the query's own block of ``mask.size``
  positions, one added to the softmax's denominator, and a sigmoid gate per output element; right is retention, linear
  attention with a fixed ``decay`` per head on rotated queries and keys, every head's output divided by its root mean square
  and gated by silu;
* ``delta``: the gated delta rule: q, k and v through a short convolution over ``conv`` tokens and silu, q and k of unit
  length per head, a decay and a step size per head and token computed from the input, ``heads`` value heads over
  ``kv_heads`` query/key heads, a norm with one weight for all heads, gated by silu.

Feed-forwards: dense gated (silu) with biases, or none.  The output matrix is a tensor of its own.

Keys read from ``config.json``: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``norm.groups``, ``layers[i].type`` /
``.mixer`` / ``.mlp`` (and, optional, ``max_positions`` and ``eos_token_id``).  Tensor names: ``embed``, ``head``,
``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*`` (``l<i>.mix.left.*`` and ``.right.*`` for the two side by side),
``l<i>.mlp.*``, ``final.norm``; linear weights are [out, in] with no suffix, biases ``<tensor>.b``.  The 1e-6 under the
root of the delta rule's unit vectors is the design's and stands in code.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .veterax import DEFAULT_MAX_POSITIONS, _need

MIXERS = ("parallel", "delta")
UNIT_EPS = 1e-6


def _check_rot(rot, dim: int, where: str, scaling: bool) -> None:
    if rot is None:
        return
    dims = _need(rot, "dims", where)
    if _need(rot, "base", where, float) <= 0:
        raise ConfigError(f"config.json: {where}.base must be positive")
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.dims ({dims}) must be even and at most dim ({dim})")
    sc = rot.get("scaling")
    if sc is not None:
        if not scaling:
            raise ConfigError(f"config.json: {where}.scaling: this mixer's rotation has no scaling")
        if _need(sc, "factor", f"{where}.scaling", float) <= 0:
            raise ConfigError(f"config.json: {where}.scaling.factor must be positive")


def _divides(m, where: str) -> None:
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.kv_heads ({m['kv_heads']}) must divide heads ({m['heads']})")


def _check_layer(i: int, layer) -> None:
    where = f"layers[{i}]"
    kind = layer.get("type") if isinstance(layer, Mapping) else None
    if kind not in MIXERS:
        raise ConfigError(f"config.json: {where}.type must be one of {MIXERS}, got {kind!r}")
    m = layer.get("mixer")
    if not isinstance(m, Mapping):
        raise ConfigError(f"config.json: {where}: required key 'mixer' is missing")
    where += ".mixer"
    if kind == "parallel":
        left, right = m.get("left"), m.get("right")
        for k in ("heads", "kv_heads", "dim", "vdim"):
            _need(left, k, f"{where}.left")
        _divides(left, f"{where}.left")
        _need(left, "scale", f"{where}.left", float)
        _need(left.get("mask"), "size", f"{where}.left.mask")
        _check_rot(left.get("rot"), left["dim"], f"{where}.left.rot", True)
        for k in ("heads", "dim", "vdim"):
            _need(right, k, f"{where}.right")
        _check_rot(right.get("rot"), right["dim"], f"{where}.right.rot", False)
        decay = right.get("decay")
        if not isinstance(decay, list) or len(decay) != right["heads"] or \
                any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
            raise ConfigError(f"config.json: {where}.right.decay must be a list of one number per head ({right['heads']})")
        for k in ("left_scale", "right_scale"):
            _need(m, k, where, float)
    else:
        for k in ("heads", "kv_heads", "dim", "vdim", "conv"):
            _need(m, k, where)
        _divides(m, where)
    f = layer.get("mlp")
    if f is None:
        return
    fk = f.get("kind") if isinstance(f, Mapping) else None
    if fk != "dense":
        raise ConfigError(f"config.json: layers[{i}].mlp.kind must be 'dense', got {fk!r}")
    _need(f, "ff", f"layers[{i}].mlp")


@dataclass(frozen=True)
class GopevikConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    norm_groups: int
    layers: Tuple[dict, ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()
    extra: dict = field(default_factory=dict, compare=False, hash=False)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "GopevikConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        for i, layer in enumerate(layers):
            _check_layer(i, layer)
        eps = _need(d.get("norm"), "eps", "norm", float)
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        groups, width = _need(d.get("norm"), "groups", "norm"), _need(d, "width", "config")
        if width % groups:
            raise ConfigError(f"config.json: norm.groups ({groups}) must divide width ({width})")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
        return cls(architecture=d.get("architecture") or d["architectures"][0],
                   vocab_size=_need(d, "vocab", "config"), hidden_size=width, norm_eps=eps, norm_groups=groups,
                   layers=tuple(copy.deepcopy(layer) for layer in layers),
                   max_position_embeddings=d.get("max_positions") or DEFAULT_MAX_POSITIONS, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
             "layers": [copy.deepcopy(layer) for layer in self.layers]}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d


def _position(positions: dict, m: Mapping) -> Optional[str]:
    """The name under which the model keeps this mixer's rotation tables (mixers with equal rotations share them)."""
    rot = m.get("rot")
    if rot is None:
        return None
    sc = rot.get("scaling")
    name = f"rot{rot['dims']}of{m['dim']}b{rot['base']!r}" + (f"/{sc['factor']!r}" if sc else "")
    positions.setdefault(name, PartSpec("rotary", {
        "head_dim": m["dim"], "rotary_dim": rot["dims"], "base": rot["base"], "pairing": "half",
        "scaling": {"kind": "linear", "factor": sc["factor"]} if sc else None}))
    return name


def describe_gopevik(cfg: GopevikConfig) -> ModelSpec:
    D, eps = cfg.hidden_size, cfg.norm_eps
    norm = lambda tensor: PartSpec("group_rmsnorm", {"size": D, "eps": eps, "groups": cfg.norm_groups, "tensor": tensor})
    positions, layers = {}, []
    for i, layer in enumerate(cfg.layers):
        m = layer["mixer"]
        if layer["type"] == "parallel":
            left, right = m["left"], m["right"]
            lp = {"hidden_size": D, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"],
                  "v_dim": left["vdim"], "scale": left["scale"], "position": _position(positions, left), "mask": "chunk",
                  "mask_size": left["mask"]["size"], "sink_score": 0.0, "output_gate": "element", "prefix": "left.",
                  "weight_suffix": ""}
            rp = {"hidden_size": D, "num_heads": right["heads"], "head_dim": right["dim"], "v_dim": right["vdim"], "eps": eps,
                  "position": _position(positions, right), "k_scale": right["dim"] ** -0.5, "decay": tuple(right["decay"]),
                  "prefix": "right.", "weight_suffix": ""}
            mixer = PartSpec("side_by_side", {"hidden_size": D, "prefix": "mix.", "weight_suffix": "", "branches": [
                {"name": "masked_attention", "params": lp, "scale": m["left_scale"]},
                {"name": "linear_attention", "params": rp, "scale": m["right_scale"]}]})
        else:
            mixer = PartSpec("linear_attention", {
                "hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                "v_dim": m["vdim"], "eps": eps, "conv_taps": m["conv"], "unit_eps": UNIT_EPS, "q_scale": m["dim"] ** -0.5,
                "delta_rule": True, "norm_weight": True, "prefix": "mix.", "weight_suffix": ""})
        norms = {"input": norm("norm1"), "mixer_out": norm("norm1b")}
        ff = None
        if layer.get("mlp") is not None:
            ff = PartSpec("swiglu", {"hidden_size": D, "intermediate_size": layer["mlp"]["ff"], "prefix": "mlp.",
                                     "names": ("gate", "up", "down"), "weight_suffix": "", "bias": True, "bias_suffix": ".b"})
            norms.update(post_mixer=norm("norm2"), feed_forward_out=norm("norm2b"))
        layers.append(LayerSpec(prefix=f"l{i}.", block="pre_post_norm", mixer=mixer, feed_forward=ff, norms=norms))
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab_size, max_positions=cfg.max_position_embeddings, embedding_tensor="embed",
        positions=positions, layers=layers, schedule=[ScheduleEntry(layer=i) for i in range(len(layers))],
        final_norm=norm("norm"), final_norm_prefix="final.", lm_head_tensor="head")


register_architecture("Gopevik", GopevikConfig, describe_gopevik)
