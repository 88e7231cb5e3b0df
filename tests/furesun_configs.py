"""Small Furesun configurations for the tests: every size and option differs between them and from layer to layer;
values that a model may happen to make equal or 1 are unequal or not 1 somewhere (and equal or 1 somewhere else)."""
import torch

from fogurax_configs import make_folder, read_folder  # noqa: F401  (any registered architecture)


def ramp(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base=10000.0, scaling=(4.0, 64, 8.0, 1.0), scale=None):
    """Latent attention in a window; ``scaling`` None: rates as they are."""
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = ramp(*scaling)
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window}, "rot": rot,
        "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}}


def attn(heads, kv_heads, dim, vdim, window, rot_dims=None, base=10000.0, softcap=20.0, scale=None, kv_from=None):
    """Windowed attention with whole-projection norms, capped scores and one in the denominator."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "softcap": softcap,
         "rot": {"base": base, "dims": rot_dims or dim - dim % 2}, "scale": scale if scale is not None else dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def mlstm(heads, dim, vdim, cap=12.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=1.3, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def config(vocab, width, eps, layers, softcap=15.0):
    c = {"architecture": "Furesun", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [dict(mix, mlp=mlp) for mix, mlp in layers]}
    if softcap is not None:
        c["logit_softcap"] = softcap
    return c


# grouped and single key/value heads, values larger and smaller than keys, part of a head unrotated, windows shorter than a page,
# no multiple of one and longer than most prompts, a layer that reads another one's keys through a wider window than that
# layer's own and one through a narrower, experts with and without a shared one, layers without a feed-forward
FA = config(310, 96, 1e-5, [
    (attn(6, 3, 16, 24, 20, rot_dims=8, base=500.0, softcap=3.0, scale=0.6), moe(5, 2, 24, shared=40)),
    (mlstm(3, 20, 24, cap=7.0), dense(56)),
    (attn(3, 3, 16, 24, 37, rot_dims=8, base=500.0, softcap=9.0, scale=0.3, kv_from=0), None),
    (latent(4, 24, 8, 16, 40, 33, base=300.0), moe(7, 3, 16, scale=0.7)),
    (attn(6, 3, 16, 24, 5, rot_dims=8, base=500.0, softcap=30.0, scale=0.5, kv_from=0), dense(24)),
    (mlstm(2, 32, 12, cap=15.0), None),
])
# one key/value head, sizes that are no whole 16-byte pieces (the float32 kernels serve them in bfloat16 too), a recurrent
# layer first and last, a window of one position and one past every prompt, every expert chosen, no stretch of the rates
FB = config(515, 128, 2e-3, [
    (mlstm(4, 64, 64), moe(3, 3, 24, shared=16)),
    (latent(3, 20, 10, 12, 24, 64, base=77.0, scaling=None, scale=0.4), dense(72)),
    (attn(10, 1, 12, 20, 1, rot_dims=4, base=300.0, softcap=50.0), dense(40)),
    (latent(2, 32, 32, 64, 96, 500, scaling=(8.0, 32, 32.0, 1.0)), moe(9, 1, 32, scale=2.0)),
    (attn(4, 2, 64, 128, 96, softcap=5.0), None),
    (attn(4, 2, 64, 128, 64, softcap=5.0, kv_from=4), moe(4, 2, 40, scale=1.0, shared=24)),
    (mlstm(1, 100, 36, cap=5.0), dense(64)),
], softcap=None)
CONFIGS = {"A": FA, "B": FB}


def one_layer(mix, mlp, vocab=200, width=64, eps=3e-6, softcap=12.0):
    return config(vocab, width, eps, [(mix, mlp)], softcap)


def steady(tensors) -> None:
    """Recurrent heads whose first outputs are not short by cancellation: a head's first output is (k . q) v divided by its own
    length, and where random k and q are nearly orthogonal its sign hangs on the last digits.  Here the keys' matrices of the
    matrix memories lie near the queries'."""
    for name in list(tensors):
        if name.endswith(".mix.i"):
            p = name[:-1]
            tensors[p + "k"] = (0.8 * tensors[p + "q"].float() + 0.6 * tensors[p + "k"].float()).to(torch.bfloat16)


def steady_routing(tensors) -> None:
    """For runs in bfloat16: routers whose choice no rounding can flip.  Channel 0 of the residual sum is the embedding's alone
    (every norm's weight is 0 there), one of four exact numbers per token, two of them negative; a router reads channel 0
    only, with slopes that lie far apart.  So the choice and the weights depend on the token and on nothing that rounds.  With
    random routers a bfloat16 run meets, every few hundred tokens, two scores closer than its rounding and takes the other
    expert: the float32 runs keep the random routers and check the choice."""
    steady(tensors)
    if not any(n.endswith("mlp.router") for n in tensors):
        return
    v = tensors["embed"].shape[0]
    tensors["embed"][:, 0] = torch.tensor([1.0, -0.5, 0.75, -1.25])[torch.arange(v) % 4].to(torch.bfloat16)
    for name in list(tensors):
        if name.endswith((".norm1", ".norm2")):
            tensors[name][0] = 0.0
        if name.endswith("mlp.router"):
            n = tensors[name].shape[0]
            order = [n - 1 - j // 2 if j % 2 == 0 else j // 2 for j in range(n)]      # most preferred first
            r = torch.zeros_like(tensors[name])
            for j, e in enumerate(order):
                r[e, 0] = 4.0 * (j - (n - 1) / 2) / n
            tensors[name] = r


def drawn(seed: int) -> dict:
    """A model drawn at random: three to six layers of any kind in any order, sizes, windows, constants and feed-forwards
    drawn anew for every layer (some sizes multiples of 8, some not)."""
    import random
    rng = random.Random(seed)
    layers = []
    for i in range(rng.randint(3, 6)):
        kind = rng.choice(["latent", "attn", "attn", "mlstm"])
        owners = [n for n, (mix, _) in enumerate(layers) if mix["type"] == "attention" and "kv_from" not in mix["mixer"]]
        if kind == "mlstm":
            mix = mlstm(rng.choice([1, 2, 3, 5]), rng.choice([8, 12, 16, 33, 48, 64]), rng.choice([4, 8, 20, 32, 72]), rng.choice([3.0, 8.0, 15.0]))
        elif kind == "latent":
            rot = rng.choice([4, 8, 16, 10])
            mix = latent(rng.choice([1, 2, 3, 5]), rng.choice([8, 12, 16, 24]), rot, rng.choice([8, 12, 16, 40]), rng.choice([8, 20, 32, 48]),
                         rng.choice([1, 3, 16, 37, 64, 500]), base=rng.choice([50.0, 1000.0, 3e5]),
                         scaling=rng.choice([None, (4.0, 64, 8.0, 1.0), (2.5, 24, 2.0, 0.5)]), scale=rng.choice([0.2, 0.35]))
        elif owners and rng.random() < 0.6:
            j = rng.choice(owners)
            src = layers[j][0]["mixer"]
            mix = attn(src["kv_heads"] * rng.choice([1, 2, 4]), src["kv_heads"], src["dim"], src["vdim"], rng.choice([1, 5, 30, 90, 500]),
                       rot_dims=src["rot"]["dims"], base=src["rot"]["base"], softcap=rng.choice([2.0, 10.0, 50.0]),
                       scale=rng.choice([0.2, 0.4]), kv_from=j)
        else:
            kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 12, 16, 24, 40, 64])
            mix = attn(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([8, 12, 16, 20, 40]), rng.choice([1, 3, 16, 37, 64, 500]),
                       rot_dims=rng.choice([dim, dim // 2 - (dim // 2) % 2 or 2, 4]), base=rng.choice([50.0, 1000.0, 3e5]),
                       softcap=rng.choice([2.0, 10.0, 50.0]), scale=rng.choice([dim ** -0.5, 0.3]))
        experts = rng.choice([3, 6, 10])
        layers.append((mix, rng.choice([None, dense(rng.choice([24, 40, 88, 50])),
                                        moe(experts, rng.choice([1, 2, 3]), rng.choice([16, 24, 20]), rng.choice([0.6, 1.0, 2.5]),
                                            rng.choice([None, 16, 30]))])))
    return config(rng.choice([150, 333]), rng.choice([64, 96, 100, 88]), rng.choice([1e-6, 1e-4, 1e-2]), layers, rng.choice([None, 10.0, 30.0]))
