"""Small random Zasesun models for the tests: configuration builders and bf16-exact random tensors (folders: folizen_models.write)."""
import numpy as np

from folizen_models import bf16


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, mlp=None, scale=None, base=1e4, scaling=None):
    rot = dict(base=base, dims=rot_dim)
    if scaling is not None:
        rot["scaling"] = scaling
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                                                             scale=scale or (dim + rot_dim) ** -0.5, rot=rot))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared=None):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared is not None:
        m["shared"] = dict(ff=shared)
    return m


YARN = dict(factor=6.0, original=96, fast=9.0, slow=1.5)


def make(width, vocab, layers, eps=1e-6, mult=0.5, cap=20.0, seed=0):
    rng = np.random.default_rng(seed)
    t = {}

    def lin(name, out, inp, gain=1.0):
        t[name] = bf16(rng.standard_normal((out, inp)) * gain / np.sqrt(inp))

    def vec(name, n, mean=1.0, dev=0.2):
        t[name] = bf16(mean + dev * rng.standard_normal(n))

    t["embed"] = bf16(rng.standard_normal((vocab, width)))
    for i, layer in enumerate(layers):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        x, f = p + "mix.", p + "mlp."
        H, d, dr, dv, qr, kr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        vec(p + "norm1", width); vec(p + "norm1b", width)
        lin(x + "dq", qr, width); vec(x + "dq.norm", qr); lin(x + "uq", H * (d + dr), qr, 1.7)
        lin(x + "dkv", kr + dr, width); vec(x + "dkv.norm", kr)
        lin(x + "uk", H * d, kr); lin(x + "uv", H * dv, kr); lin(x + "o", width, H * dv)
        if mlp is None:
            continue
        vec(p + "norm2", width); vec(p + "norm2b", width)
        if mlp["kind"] == "dense":
            lin(f + "gate", mlp["ff"], width); lin(f + "up", mlp["ff"], width); lin(f + "down", width, mlp["ff"])
        else:
            lin(f + "router", mlp["router"]["experts"], width, 1.5)
            for e in range(mlp["router"]["experts"]):
                lin(f"{f}e{e}.up", mlp["expert"]["ff"], width); lin(f"{f}e{e}.down", width, mlp["expert"]["ff"])
            if "shared" in mlp:
                lin(f + "shared.up", mlp["shared"]["ff"], width); lin(f + "shared.down", width, mlp["shared"]["ff"])
    vec("final.norm", width)
    return dict(config=dict(architecture="Zasesun", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, logit_softcap=cap, layers=layers), tensors=t)


def pointer(heads=4, dim=24, rot_dim=8, vdim=32, q_rank=40, kv_rank=48, strength=16.0, seed=9):
    """One attention layer where token 1's key and token 2's query point at each other: their unrotated score stands `strength` above
    the others', whatever the distance.  Draw the other tokens from 3 up."""
    width = 96
    model = make(width, 40, [latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scaling=YARN)], mult=2.0, seed=seed)
    t, m = model["tensors"], model["config"]["layers"][0]["mixer"]
    rng = np.random.default_rng(5)
    dirs = np.linalg.qr(rng.standard_normal((width, 2)))[0].T
    t["embed"][:] = bf16(t["embed"] - t["embed"] @ dirs.T @ dirs)          # the others have no part in the two directions
    t["embed"][1], t["embed"][2] = bf16(30 * dirs[0]), bf16(30 * dirs[1])
    for n in ("norm1", "mix.dq.norm", "mix.dkv.norm"):
        t["l0." + n][:] = 1.0
    a, b = np.sign(rng.standard_normal(q_rank)), np.sign(rng.standard_normal(kv_rank))
    t["l0.mix.dq"] = bf16(0.3 * t["l0.mix.dq"] + np.outer(a, dirs[1]))
    t["l0.mix.dkv"] = bf16(0.3 * t["l0.mix.dkv"] + np.outer(np.concatenate([b, np.zeros(rot_dim)]), dirs[0]))
    gain = np.sqrt(strength / (m["scale"] * dim))          # both latents are close to the signs a and b: q = k = gain u
    for h in range(heads):
        u = np.sign(rng.standard_normal(dim))
        q, k = h * (dim + rot_dim), h * dim
        t["l0.mix.uq"][q:q + dim] = bf16(0.3 * t["l0.mix.uq"][q:q + dim] + gain * np.outer(u, a) / q_rank)
        t["l0.mix.uk"][k:k + dim] = bf16(0.3 * t["l0.mix.uk"][k:k + dim] + gain * np.outer(u, b) / kv_rank)
    return model
