"""Linear attention with a matrix state per head and one decay number per head and token: retention (a fixed decay per
head), the gated delta rule (a decay and a step size computed from the input), matrix memories with exponential gates and
a normaliser, and what lies between, as options.

With h the mixer's input [T, D], H heads of value size vd over G query/key heads of size d (head i uses query/key head
i // (H / G)):

    q, k, v = Wq h, Wk h, Wv h                     (``q`` [G*d, D], ``k`` alike, ``v`` [H*vd, D]; no biases)
    ``conv_taps`` > 0: every channel c of q, k, v <- silu(sum_j w[c, j] * (its value ``conv_taps`` - 1 - j tokens earlier)),
        zeros before the sequence's start (``<q|k|v>.conv`` [channels, taps])
    ``unit_eps``: every head of q and of k <- head / sqrt(sum(head^2) + unit_eps)
    ``position``: the first ``rotary_dim`` elements of every head of q and k turn by the token's position
    q <- q * q_scale;  k <- k * k_scale
    decay g per head and token: the constants ``decay`` (one per head), or with ``decay`` None
        g = exp(-exp(A_log) * softplus(Wa h + dt_bias))      (``a`` [H, D], ``A_log`` [H], ``dt_bias`` [H])
    S <- g S;   x = v, or with ``delta_rule`` x = beta (v - S^T k), beta = sigmoid(Wb h) (``b`` [H, D]);
    S <- S + k x^T;   o = S^T q
    out = Wo [o / sqrt(mean(o^2) + eps) of every head (* ``norm`` [vd], one for all heads, with ``norm_weight``; [H*vd] with
        ``norm_weight`` = "all") * silu(Wg h)]      (``output_gate`` = "sigmoid": sigmoid(Wg h))

``gate_cap`` c (no decay, no delta rule, as many query/key heads as value heads) gives a head exponential gates, a running
maximum m that starts at 0, and a normaliser n [d] that starts at zero:
    i = c tanh((Wi h + bi) / c),  f = logsigmoid(c tanh((Wf h + bf) / c))      (``i`` [H, D], ``i.b`` [H]; ``f`` alike)
    m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T,  n <- e^(f + m - m') n + e^(i - m') k
    o = S^T q / (max(|n . q|, e^-m') + 1e-6)

Per request, one float32 state row: the heads' matrices S [H, vd, d] (a value column's d numbers side by side; with
exponential gates [H, vd + 1, d], n as one more column, and then the H maxima), then the last ``conv_taps`` - 1 projected
rows [q | k | v] before the convolution; a fresh row is zero.  All projections of h are one stacked product with float32
sums; everything between them and the rounded input of the output matrix is float32 in both engine dtypes
(``csrc/linear_scan.cu``).  The recurrence runs in the tokens' order, the delta rule of longer portions in runs of four
tokens (the same rule written out).  Single tokens whose q and k need nothing but their constants are read where the
product left them: the step is one launch.

``inner`` computes everything up to the output projection into a tensor the caller gives, times ``out_scale``.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from .. import kernels
from ..cache import FixedState
from ..config.registry import register_part
from ..weights.loader import TensorSource, TensorSpec
from .base import Mixer, RunCacheView
from .linear import Linear, pad_rows
from . import matmul_backend


OUTPUT_GATES = {"silu": 0, "sigmoid": 1}


@register_part("mixer", "linear_attention")
class LinearAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, v_dim: Optional[int] = None,
                 num_kv_heads: Optional[int] = None, eps: float = 1e-6, conv_taps: int = 0,
                 unit_eps: Optional[float] = None, position=None, q_scale: float = 1.0, k_scale: float = 1.0,
                 decay: Optional[Sequence[float]] = None, delta_rule: bool = False, norm_weight=False,
                 gate_cap: Optional[float] = None, output_gate: str = "silu", prefix: str = "mix.", weight_suffix: str = "", output_projection: bool = True):
        G = num_kv_heads or num_heads
        if num_heads % G:
            raise ValueError(f"linear_attention: query/key heads ({G}) must divide heads ({num_heads})")
        if decay is not None and len(decay) != num_heads:
            raise ValueError(f"linear_attention: {len(decay)} decays for {num_heads} heads")
        if norm_weight not in (False, True, "all") or output_gate not in OUTPUT_GATES:
            raise ValueError(f"linear_attention: norm_weight is False, True or 'all', output_gate one of {sorted(OUTPUT_GATES)}")
        if gate_cap is not None and (not gate_cap > 0 or G != num_heads or delta_rule or decay is not None):
            raise ValueError("linear_attention: gate_cap is positive and goes with as many query/key heads as heads, without "
                             "a decay or the delta rule")
        self.gate_cap, self.gate_kind = gate_cap, OUTPUT_GATES[output_gate]
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, G
        self.head_dim, self.v_dim = head_dim, v_dim or head_dim
        if self.head_dim > kernels.LINEAR_PADS[-1] or self.v_dim > kernels.LINEAR_MAX_VDIM:
            raise ValueError(f"linear_attention: query/key heads up to {kernels.LINEAR_PADS[-1]}, values up to {kernels.LINEAR_MAX_VDIM}")
        self.eps, self.conv_taps, self.unit_eps = float(eps), int(conv_taps or 0), unit_eps
        self.position, self.q_scale, self.k_scale = position, float(q_scale), float(k_scale)
        self.fixed_decay = [float(x) for x in decay] if decay is not None else None
        self.delta_rule, self.norm_weight = bool(delta_rule), norm_weight
        self.prefix, self.sfx = prefix, weight_suffix
        H, d, vd = num_heads, head_dim, self.v_dim
        self.channels = 2 * G * d + H * vd
        pieces = [(f"{prefix}q", G * d), (f"{prefix}k", G * d), (f"{prefix}v", H * vd), (f"{prefix}g", H * vd)]
        at = self.channels + H * vd
        self.b_off = self.a_off = -1                    # columns of the stacked product
        if self.delta_rule:
            pieces.append((f"{prefix}b", H))
            self.b_off, at = at, at + H
        self.i_off = self.f_off = -1
        if self.gate_cap is not None:
            pieces += [(f"{prefix}i", H), (f"{prefix}f", H)]
            self.i_off, self.f_off, at = at, at + H, at + 2 * H
        self.computed_decay = self.fixed_decay is None and self.gate_cap is None
        if self.computed_decay:
            pieces.append((f"{prefix}a", H))
            self.a_off, at = at, at + H
        self.inp = Linear(hidden_size, pieces, bias=False, weight_suffix=weight_suffix)
        self.inner_size = H * vd
        self.out = Linear(H * vd, [(f"{prefix}o", hidden_size)], bias=False, weight_suffix=weight_suffix) \
            if output_projection else None
        self.out_stem = f"{prefix}o"
        self.stacked = self.stacked_bias = None
        self.conv_w = self.A_log = self.dt_bias = self.decay = self.norm = self.i_bias = self.f_bias = None

    # ---- what it keeps -------------------------------------------------------
    def matrix_size(self) -> int:
        """Numbers of a state row before the kept inputs: S, and with exponential gates n and the maxima."""
        H = self.num_heads
        return H * self.v_dim * self.head_dim + (H * self.head_dim + H if self.gate_cap is not None else 0)

    def state_size(self) -> int:
        n = self.matrix_size()
        if self.conv_taps > 1:
            n += (self.conv_taps - 1) * self.channels
        return (n + 3) // 4 * 4                         # rows of S then start on 16-byte boundaries

    def paged_need(self):
        return None

    def cache_need(self):
        return FixedState((self.state_size(),), torch.float32)

    # ---- tensors ---------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        p, H, G, d, vd = self.prefix, self.num_heads, self.num_kv_heads, self.head_dim, self.v_dim
        specs = self.inp.tensor_specs()
        if self.out is not None:
            specs += self.out.tensor_specs()
        if self.conv_taps:
            specs += [TensorSpec(f"{p}{n}.conv", (c, self.conv_taps), init="uniform:-0.5:0.5")
                      for n, c in (("q", G * d), ("k", G * d), ("v", H * vd))]
        if self.gate_cap is not None:
            specs += [TensorSpec(f"{p}i.b", (H,), init="uniform:-2.0:2.0"), TensorSpec(f"{p}f.b", (H,), init="uniform:2.0:6.0")]
        if self.computed_decay:
            specs += [TensorSpec(f"{p}A_log", (H,), init="uniform:-2.0:1.0"),
                      TensorSpec(f"{p}dt_bias", (H,), init="uniform:-3.0:0.0")]
        if self.norm_weight:
            specs.append(TensorSpec(f"{p}norm", (H * vd if self.norm_weight == "all" else vd,), init="around_one"))
        return specs

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.inp.bind(source, dtype, device)
        self.stacked = pad_rows(self.inp.weight, 8)
        self.inp.weight = None
        if self.out is not None:
            self.out.bind(source, dtype, device)
        p = self.prefix
        f32 = lambda n: source.get(n).to(device=device, dtype=torch.float32).contiguous()
        if self.conv_taps:
            self.conv_w = torch.cat([f32(f"{p}{n}.conv") for n in ("q", "k", "v")], dim=0).contiguous()
        if self.gate_cap is not None:
            self.i_bias, self.f_bias = f32(f"{p}i.b"), f32(f"{p}f.b")
        elif self.computed_decay:
            self.A_log, self.dt_bias = f32(f"{p}A_log"), f32(f"{p}dt_bias")
        else:
            self.decay = torch.tensor(self.fixed_decay, dtype=torch.float32, device=device)
        if self.norm_weight:
            self.norm = f32(f"{p}norm")

    # ---- compute -----------------------------------------------------------------
    def inner(self, x: torch.Tensor, ctx, cache, out: torch.Tensor, out_scale: float = 1.0,
              u: Optional[torch.Tensor] = None) -> None:
        """Everything before the output projection: out [T, H * vd] (rows may be strided) in x's dtype.  ``u``: the
        stacked product's float32 sums, if the caller has made them (with products of other mixers of the same x)."""
        H, G, d, vd = self.num_heads, self.num_kv_heads, self.head_dim, self.v_dim
        st, off = (cache.state, cache.state_off) if isinstance(cache, RunCacheView) else (cache, 0)
        if u is None:
            u = torch.empty((x.shape[0], self.stacked.shape[0]), dtype=torch.float32, device=x.device)
            matmul_backend.linear(x, self.stacked, None, u)               # [q | k | v | gate | b | a]
        pos = self.position
        rope = (pos.rotary_dim, pos.pairing_code, pos.cos, pos.sin) if pos is not None else (0, 0, None, None)
        tail = (u[:, self.channels:self.channels + H * vd], self.norm, self.eps, out_scale, out, self.gate_kind)
        single = x.shape[0] == ctx.num_requests
        exp_gates = in_factor = low = g = None
        if self.gate_cap is not None:
            exp_gates = kernels.ExpGates(u, self.i_off, self.f_off, self.i_bias, self.f_bias, self.gate_cap,
                                         off + H * (vd + 1) * d)
            if not single:
                g, in_factor, low = kernels.linear_exp_gates(exp_gates, H, st.state, ctx, st.write)
        if single and not (self.conv_taps or self.unit_eps is not None or pos is not None or self.delta_rule or self.computed_decay):
            # q and k need nothing but their constants: the step reads them where the product left them
            kernels.linear_scan(u[:, :G * d], u[:, G * d:2 * G * d], u[:, 2 * G * d:self.channels], self.decay, None, H, d, vd,
                                st.state, off, ctx, st.write, *tail, exp_gates=exp_gates, q_scale=self.q_scale,
                                k_scale=self.k_scale)
            return
        q, k, v, beta, made = kernels.linear_prep(
            u, H, G, d, vd, self.conv_w, st.state, off + self.matrix_size(), ctx, st.write, self.unit_eps, *rope, self.q_scale,
            self.k_scale, self.b_off, self.a_off, self.A_log, self.dt_bias, k_mul=in_factor)
        g = g if g is not None else made if made is not None else self.decay
        kernels.linear_scan(q, k, v, g, beta, H, d, vd, st.state, off, ctx, st.write, *tail, exp_gates=exp_gates, low=low)

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        y = torch.empty((x.shape[0], self.inner_size), dtype=x.dtype, device=x.device)
        self.inner(x, ctx, cache, y)
        return self.out.forward_partial(y)
