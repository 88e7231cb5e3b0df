"""A plain, slow statement of the Furesun design: whole sequences, no cache, float64, one function per mechanism.
It shares no code with the engine: it takes a plain configuration dict and a dict of tensors by name.

Notation.  D width, T tokens of one sequence at positions 0..T-1.  A linear weight W is stored [out, in] and applied
as x @ W^T.  n(y; w) = y / sqrt(mean(y^2) + eps) * w.

* layer:         x += n(mixer(x); norm1);  x += n(ff(x); norm2)          (the second only with an ``mlp``)
* latent:        q = Wq x, per head [dim | rot_dim];  [c_raw | kr] = Wdkv x, c = n(c_raw; dkv.norm);  k_h = [Wuk_h c | kr],
                 v_h = Wuv_h c;  the rot_dim parts turn, pairs (i, i + dims/2), at stretched rates and with enlarged cosines
                 and sines;  the last ``mask.size`` keys, ordinary softmax;  Wo.
* attention:     grouped queries; q and k normed over all heads at once; pairs (2i, 2i+1) turn;  s = cap tanh(scale q.k / cap);
                 the last ``mask.size`` keys;  p_j = exp(s_j) / (1 + sum exp(s_j));  Wo.  With ``kv_from`` the keys (as the
                 named layer rotated them) and values are that layer's.
* mlstm:         i = cap tanh((Wi x + bi) / cap),  f = logsigmoid(cap tanh((Wf x + bf) / cap));  m' = max(f + m, i), m_0 = 0;
                 S <- exp(f + m - m') S + exp(i - m') k v^T, n <- alike with k alone;  o = S^T q / (max(|n.q|, exp(-m')) + 1e-6),
                 q times dim^-1/2;  every head's o divided by its root mean square;  times norm, times sigmoid(Wg x);  Wo.
* feed-forward:  dense Wd (gelu_tanh(Wg x) * (Wu x)), or the ``top`` experts of the largest sigmoid(Wr x), weighed by those
                 scores divided by their sum (+ 1e-20) times ``router.scale``, expert = Wd (silu(Wg x) * (Wu x)), plus a shared one.
* output:        cap tanh(Wh n(x; final.norm) / cap).
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Sequence

import torch

F64 = torch.float64


def rms_div(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def soft_cap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return z if cap is None else float(cap) * torch.tanh(z / float(cap))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def rates_and_size(rot: dict):
    """Every pair's rate, and what cosines and sines are multiplied by."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    at = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def turn(x: torch.Tensor, rot: Optional[dict], halves: bool) -> torch.Tensor:
    """x [T, heads, d]: the first ``dims`` elements turn; pairs (i, i + dims/2) with ``halves``, else (2i, 2i + 1)."""
    if not rot:
        return x
    dims = int(rot["dims"])
    f, size = rates_and_size(rot)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * f[None, :]
    cos, sin = size * torch.cos(ang)[:, None, :], size * torch.sin(ang)[:, None, :]
    y = x.clone()
    a, b = (slice(0, dims // 2), slice(dims // 2, dims)) if halves else (slice(0, dims, 2), slice(1, dims, 2))
    u, v = x[..., a], x[..., b]
    y[..., a] = u * cos - v * sin
    y[..., b] = v * cos + u * sin
    return y


def window(T: int, size: int) -> torch.Tensor:
    """[T, T] True where query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def softmax(s: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    return torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1)


def softmax_plus_one(s: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum over the visible j of exp(s_j))."""
    s = s.masked_fill(~mask, float("-inf"))
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def latent_attention(x, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, kept: dict) -> torch.Tensor:
    T = x.shape[0]
    H, dn, dr, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (x @ w[p + "q"].T).reshape(T, H, dn + dr)
    u = x @ w[p + "dkv"].T
    c = rms_div(u[:, :r], eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    kr = turn(u[:, None, r:], m.get("rot"), True)[:, 0]
    qr = turn(q[..., dn:], m.get("rot"), True)
    mask = window(T, int(m["mask"]["size"]))
    out = []
    for h in range(H):
        s = (q[:, h, :dn] @ k[:, h].T + qr[:, h] @ kr.T) * float(m["scale"])
        out.append(softmax(s, mask) @ v[:, h])
    return torch.cat(out, dim=-1) @ w[p + "o"].T


def attention(x, m: dict, w, p: str, eps: float, kept: dict) -> torch.Tensor:
    """``kept``: layer number -> (keys, values), for layers that read another one's."""
    T = x.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = turn((rms_div(x @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(T, H, d), m.get("rot"), False)
    if m.get("kv_from") is None:
        k = turn((rms_div(x @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(T, G, d), m.get("rot"), False)
        v = (x @ w[p + "v"].T).reshape(T, G, vd)
        kept["here"] = (k, v)
    else:
        k, v = kept[int(m["kv_from"])]
    mask = window(T, int(m["mask"]["size"]))
    out = []
    for i in range(H):
        g = i // (H // G)
        s = soft_cap((q[:, i] @ k[:, g].T) * float(m["scale"]), m.get("softcap"))
        out.append(softmax_plus_one(s, mask) @ v[:, g])
    return torch.cat(out, dim=-1) @ w[p + "o"].T


def mlstm(x, m: dict, w, p: str, eps: float, kept: dict) -> torch.Tensor:
    T = x.shape[0]
    H, d, vd, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = (x @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (x @ w[p + "k"].T).reshape(T, H, d)
    v = (x @ w[p + "v"].T).reshape(T, H, vd)
    i = soft_cap(x @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(soft_cap(x @ w[p + "f"].T + w[p + "f.b"], cap))
    S, n, mx = torch.zeros((H, d, vd), dtype=F64), torch.zeros((H, d), dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros((T, H, vd), dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + mx, i[t])
        keep, write = torch.exp(f[t] + mx - new), torch.exp(i[t] - new)
        mx = new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        nq = (n * q[t]).sum(dim=-1)
        o[t] = torch.einsum("hij,hi->hj", S, q[t]) / (torch.maximum(nq.abs(), torch.exp(-mx)) + 1e-6)[:, None]
    y = rms_div(o, eps).reshape(T, H * vd) * w[p + "norm"] * torch.sigmoid(x @ w[p + "g"].T)
    return y @ w[p + "o"].T


def gated(x, w, p: str, act) -> torch.Tensor:
    return (act(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def experts(x, f: dict, w, p: str) -> torch.Tensor:
    r = f["router"]
    s = torch.sigmoid(x @ w[p + "router"].T)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        best = torch.topk(s[t], int(r["top"])).indices
        total = s[t][best].sum() + 1e-20
        for e in best.tolist():
            out[t] += s[t][e] / total * float(r["scale"]) * gated(x[t:t + 1], w, f"{p}e{e}.", silu)[0]
    if f.get("shared"):
        out = out + gated(x, w, p + "shared.", silu)
    return out


def feed_forward(x, f: dict, w, p: str) -> torch.Tensor:
    return gated(x, w, p, gelu_tanh) if f["kind"] == "dense" else experts(x, f, w, p)


MIXERS = {"latent_attention": latent_attention, "attention": attention, "mlstm": mlstm}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    w = {k: v.to(F64) for k, v in weights.items() if v.is_floating_point()}
    eps = float(cfg["norm"]["eps"])
    n = lambda y, name: rms_div(y, eps) * w[name]
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + n(MIXERS[layer["type"]](x, layer["mixer"], w, p + "mix.", eps, kept), p + "norm1")
        if "here" in kept:
            kept[i] = kept.pop("here")
        if layer.get("mlp") is not None:
            x = x + n(feed_forward(x, layer["mlp"], w, p + "mlp."), p + "norm2")
        if layers_out is not None:
            layers_out.append(x.clone())
    return soft_cap(n(x, "final.norm") @ w["head"].T, cfg.get("logit_softcap"))
