"""Plain restatement of the Folizen design in numpy (float64): one function per mechanism, token by token, no cache, nothing
shared with the library.  `forward` runs a whole sequence and returns the logits and the residual stream after every layer;
`model` = {"config": the dictionary of config.json, "tensors": {name: array}}."""
import math

import numpy as np


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def poly_norm(z, coef, eps):
    """Sum of the normalised first three powers of z, and a constant."""
    a, b, c, e = (float(v) for v in coef)
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def bias_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_attention(q, k, v, scale, temp, window):
    """q [T][H][d] against k [T][G][d], v [T][G][dv]: every query head h reads key head h // (H / G); the score of a key at
    distance n is (q . k) * scale * temp[h] - slope[h] * n, for 0 <= n < window."""
    T, H, _ = q.shape
    G = k.shape[1]
    slopes = bias_slopes(H)
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = max(0, i - window + 1)
        dist = i - np.arange(lo, i + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale * temp[h] - slopes[h] * dist
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, g]
    return out


def delta_coefficients(decay_logit, rate_logit, k):
    """(w, a, u) of one token and head: decay per key channel, removal rate per key channel, unit key."""
    w = np.exp(-math.exp(-0.5) * sigmoid(decay_logit))
    a = sigmoid(rate_logit)
    u = k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)
    return w, a, u


def general_delta(r, w, a, u, k, v, state=None):
    """All [T][dim] of one head: S <- diag(w) S - (a u)(u^T S) + k v^T (both terms of the old S), o = S^T r.  Returns (o, S)."""
    T, d = r.shape
    S = np.zeros((d, v.shape[1])) if state is None else state.copy()
    o = np.zeros((T, v.shape[1]))
    for t in range(T):
        S = w[t][:, None] * S - np.outer(a[t] * u[t], u[t] @ S) + np.outer(k[t], v[t])
        o[t] = S.T @ r[t]
    return o, S


def attention_mixer(h, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ p["q"].T).reshape(T, H, d), p["q.norm"], eps)
    k = rms_norm((h @ p["k"].T).reshape(T, G, d), p["k.norm"], eps)
    v = (h @ p["v"].T).reshape(T, G, dv)
    o = window_attention(q, k, v, m["scale"], p["temp"], m["mask"]["size"])
    return o.reshape(T, H * dv) @ p["o"].T


def delta_mixer(h, p, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    r, k, v = ((h @ p[n].T).reshape(T, H, d) for n in ("r", "k", "v"))
    decay = (np.tanh(h @ p["w1"].T) @ p["w2"].T + p["w0"]).reshape(T, H, d)
    rate = (h @ p["a"].T + p["a.b"]).reshape(T, H, d)
    o = np.zeros((T, H, d))
    for n in range(H):
        w, a, u = delta_coefficients(decay[:, n], rate[:, n], k[:, n])
        o[:, n], _ = general_delta(r[:, n], w, a, u, k[:, n], v[:, n])
    o = rms(o, eps).reshape(T, H * d) * p["norm"] * sigmoid(h @ p["g"].T)
    return o @ p["o"].T


def dense_mlp(h, p, eps):
    return poly_norm(h @ p["up"].T, p["act"], eps) @ p["down"].T


def token_side(x, e, p, eps):
    """The increment of the per-layer token input."""
    y = (gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T
    return rms_norm(y, p["norm"], eps)


MIXERS = {"attention": attention_mixer, "general_delta": delta_mixer}


def forward(model, tokens):
    cfg = model["config"]
    W = {k: np.asarray(v, np.float64) for k, v in model["tensors"].items()}
    eps, sd = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    tokens = np.asarray(tokens)

    def part(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}

    x = W["embed"][tokens]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = part(f"l{i}.")
        x = x + rms_norm(MIXERS[layer["type"]](x, part(f"l{i}.mix."), layer["mixer"], eps), p["norm1"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(dense_mlp(x, part(f"l{i}.mlp."), eps), p["norm2"], eps)
        x = x + token_side(x, W["side.embed"][tokens, i * sd:(i + 1) * sd], part(f"l{i}.side."), eps)
        streams.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(streams)
