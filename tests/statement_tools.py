"""Expected logits from a design's plain statement, with what the statement allows at each place."""
import numpy as np
import torch

# A design that divides outputs by their own lengths multiplies rounding, at some tokens many times more than at others.  So a
# row may differ by a tolerance of the largest logit, or by ``ALLOW`` times what the statement itself moves there when every
# weight gets relative noise of the size of the dtype's rounding (a lost key, a wrong page or a lost state moves most rows by
# far more).
NOISE = {"float32": 2e-7, "bfloat16": 2e-3}
ALLOW = 4.0


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


def expected(forward, cfg, w, seqs, draws: int = 2, keep=None) -> Expected:
    """``forward(cfg, weights, tokens)``: the statement.  ``keep(name)``: tensors that get no noise (what no rounding reaches)."""
    want = Expected(forward(cfg, w, s).numpy() for s in seqs)
    gen = torch.Generator().manual_seed(1)
    want.allow = {}
    for dtype, eps in NOISE.items():
        rows = [np.zeros(len(s)) for s in seqs]
        for _ in range(draws):
            noisy = {k: v if keep is not None and keep(k) else
                     v.double() * (1 + eps * torch.randn(v.shape, generator=gen, dtype=torch.float64)) for k, v in w.items()}
            for r, s in enumerate(seqs):
                rows[r] = np.maximum(rows[r], np.abs(forward(cfg, noisy, s).numpy() - want[r]).max(axis=-1))
        want.allow[dtype] = [ALLOW * x for x in rows]
    return want
