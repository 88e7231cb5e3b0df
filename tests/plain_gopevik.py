"""A plain, slow statement of the Gopevik design: whole sequences, no cache, float64, one function per mechanism.
It shares no code with the engine: it takes a plain configuration dict and a dict of tensors by name.

Notation.  D width, T tokens of one sequence at positions 0..T-1.  A linear weight W is stored [out, in] and applied
as x @ W^T.  n(y; w) is the grouped norm: y is cut into ``norm.groups`` equal consecutive parts, every part is divided
by its own sqrt(mean(part^2) + eps), and the whole is multiplied by w.

* layer:         x += n(mixer(n(x; norm1)); norm1b);  x += n(ff(n(x; norm2)); norm2b)   (the second only with an ``mlp``)
* parallel:      left_scale * chunk_attention(h) + right_scale * retention(h)
* chunk_attention: grouped queries, pairs (i, i + dims/2) turn at rates base^(-2i/dims) / factor, keys j <= i of the
                 same block of ``mask.size`` positions, p_j = exp(s_j) / (1 + sum exp(s_j)); the heads' values times
                 sigmoid(Wg h) element by element; Wo.
* retention:     q and k turn, k times dim^-1/2;  S <- decay_h S + k v^T,  o = S^T q;  every head's o is divided by its
                 root mean square;  times silu(Wg h);  Wo.
* delta:         q, k, v through a short causal convolution and silu; q and k of every head of unit length (1e-6 under
                 the root), q times dim^-1/2;  beta = sigmoid(Wb h),  g = exp(-exp(A_log) softplus(Wa h + dt_bias));
                 S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;  o / rms(o) * norm * silu(Wg h);  Wo.
* feed-forward:  Wd (silu(Wg h + bg) * (Wu h + bu)) + bd.
* output:        logits = Wh n(x; final.norm).
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

F64 = torch.float64


def rms_div(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def group_norm(y: torch.Tensor, weight: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    T, D = y.shape
    parts = [rms_div(part, eps) for part in torch.split(y, D // groups, dim=-1)]
    return torch.cat(parts, dim=-1) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def turn(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: pairs (i, i + dims/2) of the first ``dims`` elements turn by position * rate_i."""
    if not rot:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    rates = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    if rot.get("scaling"):
        rates = rates / float(rot["scaling"]["factor"])
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * rates[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j][None, :]
    return y


def same_block(T: int, size: int) -> torch.Tensor:
    """[T, T] True where query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def softmax_plus_one(s: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum over the visible j of exp(s_j)): a score of 0 with no value takes part."""
    s = s.masked_fill(~mask, float("-inf"))
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def chunk_attention(h, m: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = turn((h @ w[p + "q"].T).reshape(T, H, d), m.get("rot"))
    k = turn((h @ w[p + "k"].T).reshape(T, G, d), m.get("rot"))
    v = (h @ w[p + "v"].T).reshape(T, G, vd)
    mask = same_block(T, int(m["mask"]["size"]))
    out = []
    for i in range(H):
        g = i // (H // G)
        out.append(softmax_plus_one((q[:, i] @ k[:, g].T) * float(m["scale"]), mask) @ v[:, g])
    o = torch.cat(out, dim=-1) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def retention(h, m: dict, w, p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    q = turn((h @ w[p + "q"].T).reshape(T, H, d), m.get("rot"))
    k = turn((h @ w[p + "k"].T).reshape(T, H, d), m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, vd)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=F64)[:, None, None]
    S = torch.zeros((H, d, vd), dtype=F64)
    o = torch.zeros((T, H, vd), dtype=F64)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hij,hi->hj", S, q[t])
    return (rms_div(o, eps).reshape(T, H * vd) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, m: dict, w, p: str, eps: float) -> torch.Tensor:
    return float(m["left_scale"]) * chunk_attention(h, m["left"], w, p + "left.") + \
        float(m["right_scale"]) * retention(h, m["right"], w, p + "right.", eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_mixer(h, m: dict, w, p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k = unit(q.reshape(T, G, d)) * d ** -0.5, unit(k.reshape(T, G, d))
    q, k = (torch.repeat_interleave(t, H // G, dim=1) for t in (q, k))
    v = v.reshape(T, H, vd)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    S = torch.zeros((H, d, vd), dtype=F64)
    o = torch.zeros((T, H, vd), dtype=F64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hij,hi->hj", S, q[t])
    o = rms_div(o, eps) * w[p + "norm"]
    return (o.reshape(T, H * vd) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_ff(h, w, p: str) -> torch.Tensor:
    a = silu(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])
    return a @ w[p + "down"].T + w[p + "down.b"]


MIXERS = {"parallel": parallel_mixer, "delta": delta_mixer}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    w = {k: v.to(F64) for k, v in weights.items() if v.is_floating_point()}
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"]["groups"])
    n = lambda y, name: group_norm(y, w[name], eps, groups)
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        a = MIXERS[layer["type"]](n(x, p + "norm1"), layer["mixer"], w, p + "mix.", eps)
        x = x + n(a, p + "norm1b")
        if layer.get("mlp") is not None:
            x = x + n(gated_ff(n(x, p + "norm2"), w, p + "mlp."), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return n(x, "final.norm") @ w["head"].T
