"""Plain restatement of the Zasesun design in numpy (float64): one function per mechanism, whole sequences without a cache, keys
and values expanded from the latent for every head, nothing shared with the library.  `forward` returns the logits and the
residual stream after every layer; `model` = {"config": the dictionary of config.json, "tensors": {name: array}}."""
import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def rotation(rot):
    """(frequency of every pair, factor of cos and sin)."""
    d, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / d) for i in range(d // 2)])
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def turns(t):          # the (fractional) pair index whose wave makes t turns within the original length
        return d * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), d - 1)
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = fi / s["factor"] * r + fi * (1.0 - r)
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T][..][rot_dim]: neighbours (2i, 2i + 1) turn by position * frequency i; dimensions from rot["dims"] on stay."""
    f, gain = rotation(rot)
    y = np.array(x, np.float64)
    for i in range(rot["dims"] // 2):
        a = (positions * f[i]).reshape((-1,) + (1,) * (x.ndim - 2))
        c, s = np.cos(a) * gain, np.sin(a) * gain
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def causal_softmax(s):
    """Rows of scores [T][T]: weights over the keys up to the row's own position."""
    T = s.shape[0]
    s = np.where(np.arange(T)[None] <= np.arange(T)[:, None], s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def latent_attention(h, p, m, eps):
    T = h.shape[0]
    H, d, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (rms_norm(h @ p["dq"].T, p["dq.norm"], eps) @ p["uq"].T).reshape(T, H, d + dr)
    low = h @ p["dkv"].T
    c = rms_norm(low[:, :rank], p["dkv.norm"], eps)
    k_rot = rotate(low[:, rank:], pos, m["rot"])
    q_rot = rotate(q[:, :, d:], pos, m["rot"])
    k = (c @ p["uk"].T).reshape(T, H, d)
    v = (c @ p["uv"].T).reshape(T, H, dv)
    out = np.empty((T, H, dv))
    for n in range(H):
        out[:, n] = causal_softmax((q[:, n, :d] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]) @ v[:, n]
    return out.reshape(T, H * dv) @ p["o"].T


def gated_mlp(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def squared_mlp(h, p):
    return relu_squared(h @ p["up"].T) @ p["down"].T


def route(z, top):
    """Logits [T][E] -> (chosen experts [T][top], their softmax scores over all experts)."""
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, -1)


def expert_mlp(h, p, m):
    def sub(name):
        return {k[len(name) + 1:]: v for k, v in p.items() if k.startswith(name + ".")}

    chosen, weight = route(h @ p["router"].T, m["router"]["top"])
    y = np.zeros((h.shape[0], h.shape[1]))
    for e in range(m["router"]["experts"]):
        t, slot = np.nonzero(chosen == e)
        if len(t):
            y[t] += weight[t, slot][:, None] * squared_mlp(h[t], sub(f"e{e}"))
    return y + squared_mlp(h, sub("shared")) if m.get("shared") else y


def feed_forward(h, p, m):
    return expert_mlp(h, p, m) if m["kind"] == "moe" else gated_mlp(h, p)


def margin(z, top):
    """Distance of the last chosen logit from the first that is not."""
    s = -np.sort(-z, axis=-1)
    return s[:, top - 1] - s[:, top] if top < z.shape[-1] else np.full(z.shape[0], np.inf)


def forward(model, tokens, margins=None):
    """`margins` (a list) receives one array per expert layer: every token's margin()."""
    cfg = model["config"]
    W = {k: np.asarray(v, np.float64) for k, v in model["tensors"].items()}
    eps, mult, cap = cfg["norm"]["eps"], cfg["residual_mult"], cfg["logit_softcap"]

    def part(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}

    x = W["embed"][np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        n = part(f"l{i}.")
        x = x + mult * rms_norm(latent_attention(rms_norm(x, n["norm1"], eps), part(f"l{i}.mix."), layer["mixer"], eps), n["norm1b"], eps)
        if layer["mlp"] is not None:
            h, p = rms_norm(x, n["norm2"], eps), part(f"l{i}.mlp.")
            if margins is not None and layer["mlp"]["kind"] == "moe":
                margins.append(margin(h @ p["router"].T, layer["mlp"]["router"]["top"]))
            x = x + mult * rms_norm(feed_forward(h, p, layer["mlp"]), n["norm2b"], eps)
        streams.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["embed"].T
    return cap * np.tanh(logits / cap), np.stack(streams)
