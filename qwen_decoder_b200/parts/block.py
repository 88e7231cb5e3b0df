"""The pre-norm residual block: x += mixer(norm(x)); x += feed_forward(norm(x))
(gpu_decoder.cu:321-497: norm, attention, residual, norm, feed-forward, residual).
A branch's output is left pending on the stream and added by the next norm's kernel.
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch

from ..cache import FixedState
from ..config.registry import register_part
from ..weights.loader import TensorSource, TensorSpec
from .. import kernels
from .base import Block, FeedForward, Mixer, Norm, ResidualStream, RunCacheView
from . import matmul_backend
from .linear import Linear


@register_part("block", "pre_norm")
class PreNormBlock(Block):
    norm_roles = ("input", "post_mixer")

    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm]):
        missing = [r for r in self.norm_roles if r not in norms]
        if missing:
            raise ValueError(f"pre_norm block needs norms {self.norm_roles}, missing {missing}")
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.input_norm = norms["input"]
        self.post_mixer_norm = norms["post_mixer"]

    def parts(self):
        return [self.input_norm, self.mixer, self.post_mixer_norm, self.feed_forward]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()]

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        for p in self.parts():
            p.bind(source, dtype, device)

    def native_params(self):
        if type(self) is not PreNormBlock:
            return None          # a subclass may run its parts in another order: it answers for itself
        n1, mx = self.input_norm.native_params(), self.mixer.native_params()
        n2, ff = self.post_mixer_norm.native_params(), self.feed_forward.native_params()
        if None in (n1, mx, n2, ff) or not all(k in mx for k in ("wqkv", "wo", "H", "G", "d")) \
                or not all(k in ff for k in ("wgu", "wd", "F")) or "weight" not in n1 or "weight" not in n2:
            return None
        if not (n1["size"] == n2["size"] == mx["D"] == ff["D"]):
            return None
        out = dict(mx)
        # what runs in which order: native code that restates one composition takes that one only
        out["composition"] = "/".join(["pre_norm", str(mx.get("kind")), str(ff.get("kind")), str(n1.get("kind")),
                                       str(n2.get("kind"))])
        out.update(F=ff["F"], wgu=ff["wgu"], wd=ff["wd"], norm1_w=n1["weight"], eps1=n1["eps"],
                   norm2_w=n2["weight"], eps2=n2["eps"])
        return out

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        h = self.input_norm.forward(stream, self.dtype)
        stream.push(self.mixer.forward(h, ctx, cache))
        h = self.post_mixer_norm.forward(stream, self.dtype)
        stream.push(self.feed_forward.forward(h, ctx))


@register_part("block", "pre_norm_scaled")
class ScaledPreNormBlock(PreNormBlock):
    """The pre-norm block with a layer scale: each branch's output is multiplied, element by element along
    the hidden size, by a learned vector before it joins the residual sum,
    x += s1 * mixer(norm(x)); x += s2 * feed_forward(norm(x)).  The multiplication happens in float32 inside
    the kernel that adds the branch (the next norm's).  A layer may have no feed-forward: the block then ends
    after the mixer and needs no second norm."""

    def __init__(self, mixer: Mixer, feed_forward, norms: Dict[str, Norm], size: int, prefix: str = "",
                 scale_names=("ls1", "ls2")):
        if feed_forward is None:
            norms = dict(norms)
            norms.setdefault("post_mixer", None)
        super().__init__(mixer, feed_forward, norms)
        self.size = size
        self.prefix = prefix
        self.scale_names = tuple(scale_names)
        self.mixer_scale = None
        self.ff_scale = None

    def parts(self):
        return [p for p in super().parts() if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        specs = super().tensor_specs()
        specs.append(TensorSpec(f"{self.prefix}{self.scale_names[0]}", (self.size,), init="around_one"))
        if self.feed_forward is not None:
            specs.append(TensorSpec(f"{self.prefix}{self.scale_names[1]}", (self.size,), init="around_one"))
        return specs

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        super().bind(source, dtype, device)
        get = lambda n: source.get(f"{self.prefix}{n}").to(device=device, dtype=torch.float32).contiguous()
        self.mixer_scale = get(self.scale_names[0])
        if self.feed_forward is not None:
            self.ff_scale = get(self.scale_names[1])

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        h = self.input_norm.forward(stream, self.dtype)
        stream.push(self.mixer.forward(h, ctx, cache), self.mixer_scale)
        if self.feed_forward is not None:
            h = self.post_mixer_norm.forward(stream, self.dtype)
            stream.push(self.feed_forward.forward(h, ctx), self.ff_scale)


@register_part("block", "parallel_side")
class ParallelSideBlock(Block):
    """Two branches that read the same x, then an optional per-layer token input:

        x += mixer(norm1(x)) + feed_forward(norm2(x))                    (a layer may have no feed-forward)
        e = side_table[token, side_index * side_dim : (side_index + 1) * side_dim]
        y = Wp (gelu_tanh(Wg x) * e);   x += y / sqrt(mean(y^2) + eps) * ws

    The side table is one tensor for the whole model (``side_table``, [vocab, layers * side_dim]); a block keeps its
    own slice.  Tensors of the block: ``<prefix>side.gate`` [side_dim, D], ``<prefix>side.proj`` [D, side_dim],
    ``<prefix>side.norm`` [D].  With ``side_dim`` = 0 the block ends after the two branches.

    ``shared_norm``: there is one norm and both branches read its output, x += mixer(h) + feed_forward(h) with
    h = norm1(x).  ``mult``: a constant m on everything the layer adds, x += m (mixer + feed_forward) and
    x += m y / sqrt(mean(y^2) + eps) * ws.

    Nothing is added to the residual sum by a kernel of its own where the next kernel can do it: the branch outputs
    wait on the stream for the kernel that needs the new sum (the side input's, which also writes the rounded copy the
    gate product reads), and the side output waits, to be unit-normalised and added, for the next layer's norms.  When
    both norms are tanh norms one launch writes both."""
    norm_roles = ("input", "post_mixer")

    def __init__(self, mixer: Mixer, feed_forward, norms: Dict[str, Norm], size: int, eps: float = 1e-6,
                 side_dim: int = 0, side_index: int = 0, side_table: str = "side.embed", side_table_shape=None,
                 prefix: str = "", shared_norm: bool = False, mult: float = 1.0):
        if "input" not in norms or (feed_forward is not None and not shared_norm and "post_mixer" not in norms):
            raise ValueError("parallel_side block needs the norms 'input' and, with a feed-forward, 'post_mixer'")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.shared_norm, self.mult = bool(shared_norm), float(mult)
        self.norm1 = norms["input"]
        self.norm2 = norms.get("post_mixer") if feed_forward is not None and not shared_norm else None
        self.size, self.eps, self.prefix = size, float(eps), prefix
        self.side_dim, self.side_index, self.side_table = int(side_dim), int(side_index), side_table
        self.side_table_shape = tuple(side_table_shape) if side_table_shape else None
        if self.side_dim:
            if self.side_table_shape is None or (self.side_index + 1) * self.side_dim > self.side_table_shape[1]:
                raise ValueError("parallel_side block: the side table has no columns for this layer")
            self.gate = Linear(size, [(f"{prefix}side.gate", self.side_dim)], bias=False, weight_suffix="")
            self.proj = Linear(self.side_dim, [(f"{prefix}side.proj", size)], bias=False, weight_suffix="")
        self.side_rows = self.side_norm = None

    def parts(self):
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feed_forward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        specs = [s for p in self.parts() for s in p.tensor_specs()]
        if self.side_dim:
            specs += self.gate.tensor_specs() + self.proj.tensor_specs()
            specs += [TensorSpec(f"{self.prefix}side.norm", (self.size,), init="around_one"),
                      TensorSpec(self.side_table, self.side_table_shape)]      # declared by every layer that reads it
        return specs

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        for p in self.parts():
            p.bind(source, dtype, device)
        if self.side_dim:
            self.gate.bind(source, dtype, device)
            self.proj.bind(source, dtype, device)
            self.side_norm = source.get(f"{self.prefix}side.norm").to(device=device, dtype=torch.float32).contiguous()
            lo = self.side_index * self.side_dim
            self.side_rows = source.get(self.side_table)[:, lo:lo + self.side_dim].to(device=device, dtype=dtype).contiguous()

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        from .norm import RMSNorm, TanhNorm
        T, dev = stream.x.shape[0], stream.x.device
        n1, n2 = self.norm1, self.norm2
        if type(n1) in (TanhNorm, RMSNorm) and (n2 is None or type(n2) in (TanhNorm, RMSNorm)) and \
                stream.delta_scale is None and stream.delta_gate is None and stream.delta_post is None and \
                stream.delta_bias is None:
            h1 = torch.empty((T, self.size), dtype=self.dtype, device=dev)
            h2 = torch.empty((T, self.size), dtype=self.dtype, device=dev) if n2 is not None else None
            kernels.add_tanh_norm(stream.x, stream.pending(),
                                  [n1.launch_params(h1)] + ([n2.launch_params(h2)] if n2 is not None else []))
            stream.clear()
        else:
            h1 = n1.forward(stream, self.dtype)                      # adds what was pending
            h2 = n2.forward(stream, self.dtype) if n2 is not None else None
        a = self.mixer.forward(h1, ctx, cache)
        if self.feed_forward is not None:
            stream.push_pair(a, self.feed_forward.forward(h1 if self.shared_norm else h2, ctx), mult=self.mult)
        else:
            stream.push(a, mult=self.mult)
        if not self.side_dim:
            return
        # the new sum, and its copy in the engine's dtype for the gate product, in one launch
        xr = torch.empty((T, self.size), dtype=self.dtype, device=dev)
        kernels.add_tanh_norm(stream.x, stream.pending(), [], copy_out=xr)
        stream.clear()
        g = torch.empty((T, self.side_dim), dtype=self.dtype, device=dev)
        kernels.token_gate(self.gate.forward(xr, out_dtype=torch.float32), self.side_rows, ctx.tokens, g)
        stream.push(self.proj.forward_partial(g), unit=(self.side_norm, self.eps), mult=self.mult)


@register_part("block", "pre_norm_gated")
class GatedPreNormBlock(Block):
    """The pre-norm block whose branches join through a gate, and whose mixer reads its input through a short
    causal convolution over time:

        h = norm1(x);   x += sigmoid(Wg1 h + b1) * mixer(h + conv(h));
        h = norm2(x);   x += sigmoid(Wg2 h + b2) * feed_forward(h)               (a layer may have no feed-forward)
        conv(h)_t = sum_j w[:, j] * h_(t - taps + 1 + j), zeros before the sequence's start     (per channel, no bias)

    The gates read the normed input itself, before the convolution.  ``taps`` = 0 leaves the convolution out; with
    more than one tap the last taps - 1 inputs h of every request are part of its state: the block adds
    (taps - 1) x size float32 numbers to the run's per-request state row, after whatever the mixer keeps there.
    Tensors: ``<prefix>canon1`` [size, taps], ``<prefix>rg1`` [size, size] with ``<prefix>rg1.b``, and ``rg2`` alike.
    A branch's output waits on the stream with its gate's logits; the next norm's kernel multiplies, adds and norms."""
    norm_roles = ("input", "post_mixer")

    def __init__(self, mixer: Mixer, feed_forward, norms: Dict[str, Norm], size: int, taps: int = 0, prefix: str = "",
                 conv_name: str = "canon1", gate_names=("rg1", "rg2")):
        if "input" not in norms or (feed_forward is not None and "post_mixer" not in norms):
            raise ValueError("pre_norm_gated block needs the norms 'input' and, with a feed-forward, 'post_mixer'")
        if taps < 0:
            raise ValueError("pre_norm_gated block: taps must be 0 (no convolution) or more")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norm1 = norms["input"]
        self.norm2 = norms.get("post_mixer") if feed_forward is not None else None
        self.size, self.taps, self.prefix, self.conv_name = size, int(taps), prefix, conv_name
        self.gate1 = Linear(size, [(f"{prefix}{gate_names[0]}", size)], bias=True, weight_suffix="", bias_suffix=".b")
        self.gate2 = Linear(size, [(f"{prefix}{gate_names[1]}", size)], bias=True, weight_suffix="",
                            bias_suffix=".b") if feed_forward is not None else None
        self.conv_w = None
        self._mixer_need = mixer.cache_need()
        parts = self._mixer_need if isinstance(self._mixer_need, tuple) else \
            (self._mixer_need,) if self._mixer_need is not None else ()
        self._paged = [p for p in parts if not isinstance(p, FixedState)]
        fixed = [p for p in parts if isinstance(p, FixedState)]
        if any(f.dtype != torch.float32 for f in fixed) or len(fixed) > 1:
            raise ValueError("pre_norm_gated block: the mixer's per-request state must be one float32 row")
        self.state_off = math.prod(fixed[0].shape) if fixed else 0       # the block's share follows the mixer's

    def cache_need(self):
        if self.taps <= 1:
            return self._mixer_need
        return tuple(self._paged) + (FixedState((self.state_off + (self.taps - 1) * self.size,), torch.float32),)

    def parts(self):
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feed_forward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        specs = [s for p in self.parts() for s in p.tensor_specs()]
        specs += self.gate1.tensor_specs()
        if self.gate2 is not None:
            specs += self.gate2.tensor_specs()
        if self.taps:
            specs.append(TensorSpec(f"{self.prefix}{self.conv_name}", (self.size, self.taps), init="uniform:-0.5:0.5"))
        return specs

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        for p in self.parts():
            p.bind(source, dtype, device)
        self.gate1.bind(source, dtype, device)
        if self.gate2 is not None:
            self.gate2.bind(source, dtype, device)
        if self.taps:
            self.conv_w = source.get(f"{self.prefix}{self.conv_name}").to(device=device, dtype=torch.float32).contiguous()

    def _mixer_cache(self, cache):
        """The mixer's own view: what it would get in a block without a state of its own."""
        if self.taps <= 1 or not isinstance(cache, RunCacheView):
            return cache
        if isinstance(self._mixer_need, tuple):
            return cache                                # pages and the row; the mixer's share starts at 0
        if isinstance(self._mixer_need, FixedState):
            return cache.state
        return cache.paged                              # None for a mixer that caches nothing

    @staticmethod
    def _gate_logits(gate: Linear, h: torch.Tensor) -> torch.Tensor:
        """W h as float32 sums; the bias waits with them and is added by the kernel that takes the sigmoid."""
        g = torch.empty((h.shape[0], gate.out_features), dtype=torch.float32, device=h.device)
        matmul_backend.linear(h, gate.weight, None, g)
        return g

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        h = self.norm1.forward(stream, self.dtype)
        hm = h
        if self.taps:
            hm = torch.empty_like(h)
            st = cache.state if self.taps > 1 else None
            kernels.short_conv(h, self.conv_w, st.state if st is not None else None, self.state_off, ctx.token_request,
                               ctx.cu_tokens, ctx.state_slots, hm, ctx.num_requests, residual=True,
                               update_state=bool(st is not None and st.write))
        g = self._gate_logits(self.gate1, h)
        stream.push(self.mixer.forward(hm, ctx, self._mixer_cache(cache)), gate=g, gate_bias=self.gate1.bias)
        if self.feed_forward is not None:
            h = self.norm2.forward(stream, self.dtype)
            g = self._gate_logits(self.gate2, h)
            stream.push(self.feed_forward.forward(h, ctx), gate=g, gate_bias=self.gate2.bias)


@register_part("block", "pre_post_norm")
class PrePostNormBlock(Block):
    """A norm before and a norm after each branch:

        x += norm_out1(mixer(norm_in1(x)));   x += norm_out2(feed_forward(norm_in2(x)))   (a layer may have no feed-forward)

    A branch's output waits on the stream with its norm (and the bias its last product left out); the next norm's kernel
    norms it, adds it and norms the sum, one launch between two branches."""
    norm_roles = ("input", "mixer_out", "post_mixer", "feed_forward_out")

    def __init__(self, mixer: Mixer, feed_forward, norms: Dict[str, Norm]):
        need = self.norm_roles if feed_forward is not None else self.norm_roles[:2]
        missing = [r for r in need if r not in norms]
        if missing:
            raise ValueError(f"pre_post_norm block needs norms {need}, missing {missing}")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = [norms[r] for r in need]
        for n in self.norms[1::2]:
            if not hasattr(n, "as_post"):
                raise ValueError(f"pre_post_norm block: {type(n).__name__} cannot norm a branch's output")

    def parts(self):
        return self.norms + [p for p in (self.mixer, self.feed_forward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()]

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        for p in self.parts():
            p.bind(source, dtype, device)

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        h = self.norms[0].forward(stream, self.dtype)
        stream.push(self.mixer.forward(h, ctx, cache), post=self.norms[1].as_post())
        if self.feed_forward is None:
            return
        h = self.norms[2].forward(stream, self.dtype)
        ff, bias = self.feed_forward, None
        if hasattr(ff, "forward_without_bias"):
            delta, bias = ff.forward_without_bias(h, ctx)
        else:
            delta = ff.forward(h, ctx)
        stream.push(delta, post=self.norms[3].as_post(), bias=bias)


@register_part("block", "post_norm")
class PostNormBlock(Block):
    """A norm on each branch's output and none before it: the branches read the residual sum itself (rounded to the
    engine's dtype),

        x += norm_out1(mixer(x));   x += norm_out2(feed_forward(x))      (a layer may have no feed-forward)

    A branch's output waits on the stream with its norm; the launch that adds it also writes the rounded sum the next
    branch reads."""
    norm_roles = ("mixer_out", "feed_forward_out")

    def __init__(self, mixer: Mixer, feed_forward, norms: Dict[str, Norm]):
        need = self.norm_roles if feed_forward is not None else self.norm_roles[:1]
        missing = [r for r in need if r not in norms]
        if missing:
            raise ValueError(f"post_norm block needs norms {need}, missing {missing}")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = [norms[r] for r in need]
        for n in self.norms:
            if not hasattr(n, "as_post"):
                raise ValueError(f"post_norm block: {type(n).__name__} cannot norm a branch's output")

    def parts(self):
        return self.norms + [p for p in (self.mixer, self.feed_forward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()]

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        for p in self.parts():
            p.bind(source, dtype, device)

    def _sum(self, stream: ResidualStream) -> torch.Tensor:
        """The residual sum with what was pending, in the engine's dtype."""
        if self.dtype == torch.float32:
            stream.flush()
            return stream.x
        stream.settle(post_ok=True)
        if stream.delta_scale is not None:
            stream.flush()
        h = torch.empty(stream.x.shape, dtype=self.dtype, device=stream.x.device)
        kernels.group_add_norm(stream.x, stream.delta, stream.delta_post, stream.delta_bias, out=h)
        stream.clear()
        return h

    def forward(self, stream: ResidualStream, ctx, cache) -> None:
        stream.push(self.mixer.forward(self._sum(stream), ctx, cache), post=self.norms[0].as_post())
        if self.feed_forward is not None:
            stream.push(self.feed_forward.forward(self._sum(stream), ctx), post=self.norms[1].as_post())


@register_part("block", "loop_input")
class LoopInput(Block):
    """What stands before every pass of a loop of layers: the residual sum takes the embedding output x0 in again
    and a per-pass vector is added,

        x <- Win [x ; x0] + step[visit]          Win [size, 2 size] (x's half first), step [passes, size]

    It has no mixer, no feed-forward and no cache; the schedule names it once per pass and says which (``visit``).
    The product takes x and x0 rounded to the engine's dtype and leaves float32 sums, which become the new x."""
    takes_visit = True
    reads_embedding_output = True

    def __init__(self, mixer, feed_forward, norms, size: int, passes: int, prefix: str = "",
                 names=("loop.in", "loop.step")):
        if mixer is not None or feed_forward is not None or norms:
            raise ValueError("loop_input block takes no mixer, feed-forward or norm")
        self.mixer = self.feed_forward = None
        self.size, self.passes, self.prefix, self.names = size, int(passes), prefix, tuple(names)
        self.inp = Linear(2 * size, [(f"{prefix}{names[0]}", size)], bias=False, weight_suffix="")
        self.step = None

    def cache_need(self):
        return None

    def parts(self):
        return []

    def tensor_specs(self) -> List[TensorSpec]:
        return self.inp.tensor_specs() + [TensorSpec(f"{self.prefix}{self.names[1]}", (self.passes, self.size),
                                                     init="around_zero")]

    def bind(self, source: TensorSource, dtype: torch.dtype, device: torch.device) -> None:
        self.dtype = dtype
        self.inp.bind(source, dtype, device)
        self.step = source.get(f"{self.prefix}{self.names[1]}").to(device=device, dtype=torch.float32).contiguous()

    def forward(self, stream: ResidualStream, ctx, cache, visit: int = 0) -> None:
        if stream.origin is None:
            raise ValueError("loop_input block: the model did not keep the embedding output")
        if not (0 <= visit < self.passes):
            raise ValueError(f"loop_input block: pass {visit} of {self.passes}")
        stream.flush()
        T = stream.x.shape[0]
        both = torch.empty((T, 2 * self.size), dtype=self.dtype, device=stream.x.device)
        kernels.concat_round(stream.x, stream.origin, both)
        x = torch.empty((T, self.size), dtype=torch.float32, device=stream.x.device)
        matmul_backend.linear(both, self.inp.weight, self.step[visit], x)     # the pass's vector rides as the bias
        stream.x = x
