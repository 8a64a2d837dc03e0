"""Model folders: config.json chooses the architecture, the architecture's reader turns config and weights into an engine spec
(the dictionary `Engine` takes).

    spec = load_spec(folder, dtype="bfloat16", max_seq=4096)
    engine = load_engine(ctx, folder)

Registered: `Folizen` (config.json + model.safetensors: blocks of sliding-window attention and generalized delta rule), `Zasesun`
(the same files: blocks of latent attention, dense or expert feed-forwards), and the compiled Llama / Qwen models (a Hugging Face config.json beside one .k2tb container)."""
import glob
import json
import mmap
import os

import numpy as np

from . import ffi

READERS = {}


def register(*names):
    def add(fn):
        for n in names:
            READERS[n] = fn
        return fn
    return add


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def architecture(config):
    """The registered name a config.json asks for (`architecture`, or the first known entry of `architectures`)."""
    names = [config["architecture"]] if "architecture" in config else config.get("architectures", [])
    for n in names:
        if n in READERS:
            return n
    raise ValueError(f"no reader for the architecture {names or 'of this config.json'}; known: {', '.join(sorted(READERS))}")


def load_spec(folder, dtype="bfloat16", max_seq=4096):
    if dtype not in ("bfloat16", "float32"):
        raise ValueError("dtype must be bfloat16 or float32")
    config = read_config(folder)
    return READERS[architecture(config)](folder, config, dtype, max_seq)


def load_engine(ctx, folder, dtype="bfloat16", max_seq=4096):
    return ffi.Engine(ctx, load_spec(folder, dtype, max_seq))


def generate(engine, prompt, n_steps):
    """Greedy continuation: the prompt in batches, then the device-side decode loop.  Returns the new token ids."""
    prompt = np.asarray(prompt, np.uint32)
    if len(prompt) > 1:
        engine.forward_token_ids(prompt[:-1])
    return engine.decode_greedy(int(prompt[-1]), len(prompt) - 1, n_steps)


# ---- safetensors: 8-byte little-endian header length, JSON {name: {dtype, shape, data_offsets}}, data
_SAFE_DTYPES = {"BF16": np.uint16, "F32": np.float32, "F16": np.float16, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class Tensors:
    """Tensors of a safetensors file, mapped; bf16 ones come as bit patterns (`bits`) or widened to fp32 (`f32`)."""

    def __init__(self, path):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        n = int.from_bytes(self._map[:8], "little")
        self._base = 8 + n
        self._info = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}

    def __contains__(self, name):
        return name in self._info

    def shape(self, name):
        return tuple(self._info[name]["shape"])

    def raw(self, name):
        t = self._info[name]
        lo, hi = t["data_offsets"]
        dt = np.dtype(_SAFE_DTYPES[t["dtype"]]).newbyteorder("<")
        return np.frombuffer(self._map, dt, (hi - lo) // dt.itemsize, self._base + lo).reshape(t["shape"])

    def f32(self, name):
        a = self.raw(name)
        if self._info[name]["dtype"] == "BF16":
            return (a.astype(np.uint32) << 16).view(np.float32)
        return a.astype(np.float32)

    def bits(self, name):
        return self.raw(name) if self._info[name]["dtype"] == "BF16" else ffi.bf16_bits(self.f32(name))


# ---- Folizen
DELTA_DECAY_SCALE = float(np.exp(-0.5))     # log-decay of a key channel = -exp(-1/2) sigmoid(.)
DELTA_UNIT_EPS = 1e-6


def alibi_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], np.float32)


@register("Folizen")
def folizen_spec(folder, config, dtype, max_seq):
    t = Tensors(os.path.join(folder, "model.safetensors"))
    mat = t.bits if dtype == "bfloat16" else t.f32

    def rows(*names):
        return np.concatenate([mat(n) for n in names])

    side = (config.get("token_side") or {}).get("dim", 0)
    blocks = []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        b = dict(heads=m["heads"], dim=m["dim"], norm1=t.f32(p + "norm1"), o_proj=mat(x + "o"))
        if layer["type"] == "attention":
            b.update(mixer=ffi.MIXER_WINDOW_ATTENTION, kv_heads=m["kv_heads"], vdim=m["vdim"], window=(m.get("mask") or {}).get("size", 0),
                     q_norm=t.f32(x + "q.norm"), k_norm=t.f32(x + "k.norm"), head_scale=np.float32(m["scale"]) * t.f32(x + "temp"),
                     head_slope=alibi_slopes(m["heads"]), in_proj=rows(x + "q", x + "k", x + "v"))
        elif layer["type"] == "general_delta":
            b.update(mixer=ffi.MIXER_GENERAL_DELTA, decay_rank=t.shape(x + "w1")[0], decay_scale=DELTA_DECAY_SCALE, unit_eps=DELTA_UNIT_EPS,
                     decay_bias=t.f32(x + "w0"), rate_bias=t.f32(x + "a.b"), out_norm=t.f32(x + "norm"), decay_proj=mat(x + "w2"),
                     in_proj=rows(x + "r", x + "k", x + "v", x + "g", x + "a", x + "w1"))
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        if layer.get("mlp") is not None:
            if layer["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {layer['mlp']['kind']!r}")
            b.update(ff=t.shape(p + "mlp.up")[0], norm2=t.f32(p + "norm2"), act_coef=t.f32(p + "mlp.act"), up_proj=mat(p + "mlp.up"), down_proj=mat(p + "mlp.down"))
        if side:
            b.update(side_norm=t.f32(p + "side.norm"), side_gate=mat(p + "side.gate"), side_proj=mat(p + "side.proj"))
        blocks.append(b)
    vocab, width = t.shape("embed")
    return dict(cfg=dict(hidden=width, vocab=vocab, max_seq=max_seq, eps=config["norm"]["eps"], side_dim=side, precision=16 if dtype == "bfloat16" else 32),
                blocks=blocks, final_norm=t.f32("final.norm"), head=mat("head"), embed=t.bits("embed"), side_embed=t.bits("side.embed") if side else None)


# ---- rotary positions
def yarn_frequencies(dims, base, scaling=None):
    """(frequency of every rotated pair, factor of cos and sin), float64.  scaling {factor, original, fast, slow}: pairs that turn more
    than `fast` times within `original` positions keep their frequency, those that turn less than `slow` times have it divided by
    `factor`, with a linear ramp over the pairs in between."""
    i = np.arange(dims // 2)
    freq = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return freq, 1.0
    pair = lambda turns: dims * np.log(scaling["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
    lo, hi = max(np.floor(pair(scaling["fast"])), 0), min(np.ceil(pair(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / scaling["factor"] * ramp + freq * (1.0 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotation_table(positions, width, dims, base, scaling=None):
    """[positions][width]: (cos, sin) of every neighbouring pair; pairs from `dims` on stay as they are."""
    freq, gain = yarn_frequencies(dims, base, scaling)
    angle = np.arange(positions)[:, None] * freq
    table = np.zeros((positions, width), np.float32)
    table[:, 0::2] = 1.0
    table[:, 0:dims:2], table[:, 1:dims:2] = np.cos(angle) * gain, np.sin(angle) * gain
    return table


# ---- Zasesun
@register("Zasesun")
def zasesun_spec(folder, config, dtype, max_seq):
    t = Tensors(os.path.join(folder, "model.safetensors"))
    mat = t.bits if dtype == "bfloat16" else t.f32
    tables = {}

    def rows(*names):
        return np.concatenate([mat(n) for n in names])

    blocks = []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        if layer["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        rot = m["rot"]
        key = json.dumps([m["rot_dim"], rot], sort_keys=True)
        if key not in tables:
            tables[key] = rotation_table(max_seq, m["rot_dim"], rot["dims"], rot["base"], rot.get("scaling"))
        b = dict(mixer=ffi.MIXER_LATENT_ATTENTION, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], rot_dim=m["rot_dim"], kv_rank=m["kv_rank"],
                 q_rank=t.shape(x + "dq")[0], score_scale=m["scale"], rot_cos_sin=tables[key], q_latent_norm=t.f32(x + "dq.norm"),
                 kv_latent_norm=t.f32(x + "dkv.norm"), pre_norm1=t.f32(p + "norm1"), norm1=t.f32(p + "norm1b"),
                 in_proj=rows(x + "dq", x + "dkv"), q_up=mat(x + "uq"), kv_up=rows(x + "uk", x + "uv"), o_proj=mat(x + "o"))
        mlp, f = layer.get("mlp"), p + "mlp."
        if mlp is not None:
            b.update(pre_norm2=t.f32(p + "norm2"), norm2=t.f32(p + "norm2b"))
            kind = mlp.get("kind", "dense")
            if kind == "dense":
                gate, up = mat(f + "gate"), mat(f + "up")
                b.update(act=ffi.ACT_GELU_GATED, ff=up.shape[0], up_proj=np.stack([gate, up], 1).reshape(-1, up.shape[1]), down_proj=mat(f + "down"))
            elif kind == "moe":
                n, shared = mlp["router"]["experts"], mlp.get("shared") is not None
                b.update(act=ffi.ACT_RELU_SQUARED, experts=n, experts_top=mlp["router"]["top"], ff=t.shape(f + "e0.up")[0],
                         up_proj=rows(*(f"{f}e{e}.up" for e in range(n))), down_proj=rows(*(f"{f}e{e}.down" for e in range(n))),
                         router=rows(f + "router", *([f + "shared.up"] if shared else [])))
                if shared:
                    b.update(shared_ff=t.shape(f + "shared.up")[0], shared_down=mat(f + "shared.down"))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {kind!r}")
        blocks.append(b)
    embed = mat("embed")
    return dict(cfg=dict(hidden=embed.shape[1], vocab=embed.shape[0], max_seq=max_seq, eps=config["norm"]["eps"], residual_mult=config.get("residual_mult", 1.0),
                         logit_softcap=config.get("logit_softcap") or 0.0, precision=16 if dtype == "bfloat16" else 32),
                blocks=blocks, final_norm=t.f32("final.norm"), head=embed, embed=t.bits("embed"))


# ---- compiled Llama / Qwen models
@register("LlamaForCausalLM", "Qwen2ForCausalLM", "Qwen3ForCausalLM")
def compiled_spec(folder, config, dtype, max_seq):
    """A .k2tb container with the model's Hugging Face config.json (the container holds no shapes)."""
    from . import synth
    if dtype != "bfloat16":
        raise ValueError("compiled models run in their quantized format")
    files = sorted(glob.glob(os.path.join(folder, "*.k2tb")))
    if len(files) != 1:
        raise ValueError(f"{folder}: one .k2tb container is needed, found {len(files)}")
    heads = config["num_attention_heads"]
    hd = config.get("head_dim") or config["hidden_size"] // heads
    cfg = dict(hidden=config["hidden_size"], n_q=heads, n_kv=config.get("num_key_value_heads", heads), head_dim=hd, inter=config["intermediate_size"],
               vocab=config["vocab_size"], max_seq=max_seq, eps=config.get("rms_norm_eps", 1e-5))
    return ffi.k2tb_load(files[0], cfg, synth.rope_table(max_seq, hd, config.get("rope_theta", 10000.0)))[0]
