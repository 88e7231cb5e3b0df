"""Small Gopevik configurations for the tests: every size and option differs between them and from layer to layer;
values that a model may happen to make equal or 1 are unequal or not 1 somewhere (and equal or 1 somewhere else)."""
import math

from fogurax_configs import make_folder, read_folder  # noqa: F401  (any registered architecture)


def _rot(dims, base, factor=None):
    r = {"base": base, "dims": dims}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    return r


def left(heads, kv_heads, dim, vdim, block, rot_dims=None, base=10000.0, factor=4.0, scale=None):
    """Attention over the query's own block of positions."""
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": block},
            "rot": _rot(rot_dims or dim - dim % 2, base, factor), "scale": scale if scale is not None else dim ** -0.5}


def decays(heads, lo=0.9, hi=0.999):
    """One decay per head, all different, from ``lo`` to ``hi``."""
    if heads == 1:
        return [hi]
    return [1.0 - math.exp(math.log(1.0 - lo) + (math.log(1.0 - hi) - math.log(1.0 - lo)) * i / (heads - 1)) for i in range(heads)]


def right(heads, dim, vdim, rot_dims=None, base=1e5, decay=None):
    """Retention."""
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads),
            "rot": _rot(rot_dims or dim - dim % 2, base)}


def par(l, r, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": l, "right": r, "left_scale": left_scale, "right_scale": right_scale}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, eps, groups, layers):
    return {"architecture": "Gopevik", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "layers": [dict(mix, mlp=mlp) for mix, mlp in layers]}


# grouped and single key/value heads, values larger and smaller than keys, part of a head unrotated, blocks shorter than a
# page, no multiple of one and longer than most prompts, two and five taps, several value heads per query/key head, a delta
# layer with a feed-forward and a parallel layer without one, parts of the norm that are no whole warps
GA = config(310, 96, 1e-6, 3, [
    (par(left(6, 3, 16, 24, 20, rot_dims=8, base=500.0, factor=2.5, scale=0.4), right(2, 24, 40, rot_dims=10), 0.8, 1.3), dense(40)),
    (delta(6, 2, 20, 24, 2), dense(56)),
    (par(left(4, 1, 24, 8, 7, base=77.0, factor=1.0), right(5, 8, 16, base=300.0), 1.0, 0.6), None),
    (delta(3, 3, 40, 8, 5), None),
    (par(left(2, 2, 32, 32, 150, base=1e6, factor=8.0, scale=0.3), right(1, 64, 12), 1.4, 1.0), dense(24)),
])
# one part in the norm, heads of 128 and head sizes that are no whole 16-byte pieces (the float32 kernel serves them in
# bfloat16 too), delta layers first and last, one tap, a block of one position, decays of 0, 0.5 and 1
GB = config(515, 128, 2e-5, 1, [
    (delta(4, 4, 64, 64, 4), dense(72)),
    (par(left(10, 1, 12, 20, 64, rot_dims=4, base=300.0, factor=3.0), right(3, 72, 20, rot_dims=36, decay=[0.0, 0.5, 1.0])), dense(96)),
    (par(left(2, 1, 128, 20, 1, factor=6.0, scale=0.1), right(4, 128, 8), 1.25, 0.9), None),
    (par(left(2, 2, 64, 128, 96, factor=None), right(2, 10, 136), 0.5, 1.1), dense(64)),
    (delta(2, 1, 100, 36, 1), None),
])
CONFIGS = {"A": GA, "B": GB}


def one_layer(mix, mlp, vocab=200, width=64, eps=3e-6, groups=4):
    return config(vocab, width, eps, groups, [(mix, mlp)])


def steady(tensors) -> None:
    """Recurrent heads whose first outputs are not short by cancellation.  A recurrent head's first output is (k . q) v
    divided by its own length: where random k and q are nearly orthogonal its sign hangs on the last digits, and the
    statement itself jumps.  Here the keys' matrices (and convolutions) lie near the queries'."""
    import torch
    for name in list(tensors):
        if name.endswith(".q") and ".left." not in name:
            key = name[:-1] + "k"
            for s in ("", ".conv"):
                if name + s in tensors:
                    tensors[key + s] = (0.8 * tensors[name + s].float() + 0.6 * tensors[key + s].float()).to(torch.bfloat16)


def drawn(seed: int) -> dict:
    """A model drawn at random: three to six layers of either kind in any order, sizes, taps, blocks, decays, constants
    and feed-forwards drawn anew for every layer (some sizes multiples of 8, some not)."""
    import random
    rng = random.Random(seed)
    groups = rng.choice([1, 2, 3, 4, 8])
    width = groups * rng.choice([16, 24, 20, 11])
    layers = []
    for _ in range(rng.randint(3, 6)):
        if rng.random() < 0.5:
            kv = rng.choice([1, 2, 3])
            mix = delta(kv * rng.choice([1, 2, 4]), kv, rng.choice([8, 12, 16, 33, 48, 64]), rng.choice([4, 8, 20, 32, 72]),
                        rng.choice([1, 2, 3, 4, 6]))
        else:
            kv = rng.choice([1, 2, 3])
            dim, rdim, rheads = rng.choice([8, 12, 16, 24, 40, 64]), rng.choice([8, 12, 16, 30, 64]), rng.choice([1, 2, 3, 5])
            mix = par(left(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([8, 12, 16, 20, 40]), rng.choice([1, 3, 16, 37, 64, 500]),
                           rot_dims=rng.choice([dim, dim // 2 - (dim // 2) % 2 or 2, 4]), base=rng.choice([50.0, 1000.0, 3e5]),
                           factor=rng.choice([None, 1.0, 2.0, 7.5]), scale=rng.choice([dim ** -0.5, 0.3, 0.5])),
                      right(rheads, rdim, rng.choice([8, 12, 24, 40]), rot_dims=rng.choice([rdim, 4]), base=rng.choice([50.0, 1e4]),
                            decay=[rng.choice([0.3, 0.9, 0.97, 0.995, 0.9995]) for _ in range(rheads)]),
                      left_scale=rng.choice([0.5, 1.0, 1.4]), right_scale=rng.choice([0.4, 1.0, 1.3]))
        layers.append((mix, rng.choice([None, dense(rng.choice([24, 40, 88, 50]))])))
    return config(rng.choice([150, 333]), width, rng.choice([1e-6, 1e-5, 1e-4]), groups, layers)
