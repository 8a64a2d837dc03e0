"""Small random Folizen models for the tests: configuration builders, bf16-exact random tensors, model folders."""
import json
import os

import numpy as np


def bf16(x):
    """Rounds fp32 values to bf16 (ties to even), kept as fp32."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def attention(heads, kv_heads, dim, vdim, window, scale=None, ff=None):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, mask=dict(size=window)),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def delta(heads, dim, ff=None, rank=7):
    return dict(type="general_delta", mixer=dict(heads=heads, dim=dim), mlp=None if ff is None else dict(kind="dense", ff=ff), _rank=rank)


def make(width, vocab, layers, side=8, eps=1e-6, seed=0):
    rng = np.random.default_rng(seed)
    t = {}

    def lin(name, out, inp, gain=1.0):
        t[name] = bf16(rng.standard_normal((out, inp)) * gain / np.sqrt(inp))

    def vec(name, n, mean=1.0, dev=0.2):
        t[name] = bf16(mean + dev * rng.standard_normal(n))

    t["embed"] = bf16(rng.standard_normal((vocab, width)))
    t["side.embed"] = bf16(rng.standard_normal((vocab, side * len(layers))))
    for i, layer in enumerate(layers):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        vec(p + "norm1", width)
        if layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            lin(x + "q", H * d, width); lin(x + "k", G * d, width); lin(x + "v", G * dv, width); lin(x + "o", width, H * dv)
            vec(x + "q.norm", d); vec(x + "k.norm", d)
            t[x + "temp"] = bf16(rng.uniform(0.5, 3.0, H))
        else:
            hd, rank = m["heads"] * m["dim"], layer["_rank"]
            for n in ("r", "k", "v", "g", "a"):
                lin(x + n, hd, width)
            lin(x + "w1", rank, width); lin(x + "w2", hd, rank); lin(x + "o", width, hd)
            vec(x + "a.b", hd, -1.0, 1.0); vec(x + "norm", hd)
            t[x + "w0"] = bf16(rng.uniform(-7.0, 1.0, hd))
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            vec(p + "norm2", width)
            lin(p + "mlp.up", ff, width); lin(p + "mlp.down", width, ff)
            t[p + "mlp.act"] = bf16(rng.uniform(-1.0, 1.0, 4))
        lin(p + "side.gate", side, width); lin(p + "side.proj", width, side)
        vec(p + "side.norm", width, 0.5)
    vec("final.norm", width)
    lin("head", vocab, width)
    config = dict(architecture="Folizen", vocab=vocab, width=width, norm=dict(eps=eps), token_side=dict(dim=side),
                  layers=[{k: v for k, v in ly.items() if not k.startswith("_")} for ly in layers])
    return dict(config=config, tensors=t)


def write(model, folder):
    """config.json and model.safetensors (bf16)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(model["config"], f)
    header, blobs, at = {}, [], 0
    for name, a in model["tensors"].items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = dict(dtype="BF16", shape=list(a.shape), data_offsets=[at, at + len(raw)])
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head + b"".join(blobs))
    return folder


def error(got, want):
    """Per position: rms over the vocabulary of the centred difference, in units of the reference's spread."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.std(want)
