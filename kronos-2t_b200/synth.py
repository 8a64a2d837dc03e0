"""Synthetic matrices in the reference's file formats, built without any quantizer: uniformly random
codes / indices and bf16 scales in [2^-15, 2^-7).  GEMV time does not depend on the code values;
files produced this way are valid inputs for kronos_cuda_matrix_upload (and for the oracle)."""
import numpy as np

NF4_DEFAULT = np.array([-127, -96, -75, -58, -44, -31, -18, -6, 6, 18, 31, 44, 58, 75, 96, 127], np.int8)
NF3_DEFAULT = np.array([-127, -79, -45, -14, 14, 45, 79, 127, 0, 0, 0, 0, 0, 0, 0, 0], np.int8)
_NF_CHUNK = {5: 640, 4: 512, 3: 384, 2: 256}


def _rng(seed):
    return np.random.Generator(np.random.PCG64(seed))


def random_bipolar_bytes(seed, rows, cols, planes):
    """(interleaved planes u8, bf16 scales u16) of a FusedBipolarLutMatrix with random codes."""
    ns, nc = (rows + 15) // 16, cols // 64
    rng = _rng(seed)
    data = rng.integers(0, 256, ns * (cols // 8) * planes * 16, dtype=np.uint8)
    scales = rng.integers(0x3800, 0x3C00, ns * nc * 16, dtype=np.uint16)
    return data, scales


def random_nf_bytes(seed, rows, cols, bits, sgc):
    """(pair_stream, tail_stream) of an NfSdotMatrix with random indices; rows % 32 == 0, (cols/64) % sgc == 0."""
    nc = cols // 64
    assert rows % 32 == 0 and nc % sgc == 0
    nsg, cb = nc // sgc, _NF_CHUNK[bits]
    rng = _rng(seed)
    blk = 64 + sgc * 2 * cb
    stream = rng.integers(0, 256, (rows // 32) * nsg * blk, dtype=np.uint8).reshape(rows // 32, nsg, blk)
    sc = rng.integers(0x3800, 0x3C00, (rows // 32, nsg, 32), dtype=np.uint16)
    stream[:, :, :64] = sc.view(np.uint8).reshape(rows // 32, nsg, 64)
    return stream.reshape(-1), np.zeros(0, np.uint8)


def file_bytes(kind, rows, cols, bits, sgc=1):
    """Bytes of a matrix in the reference file format (the algorithmic weight bytes of one GEMV)."""
    ns, nc = (rows + 15) // 16, cols // 64
    if kind == "bipolar":
        return ns * (cols // 8) * bits * 16 + ns * nc * 16 * 2
    nsg, cb = -(-nc // sgc), _NF_CHUNK[bits]
    return (ns // 2) * (nsg * 64 + nc * 2 * cb) + (ns & 1) * (nsg * 32 + nc * cb) + 16


class HostMatrix:
    """A matrix in the reference file format: the fields kronos_2t_b200.ffi.desc_of (and the oracle) read."""

    def __init__(self, **kw):
        self.__dict__.update(kw)

    def file_bytes(self):
        if self.kind == 0:
            return self.data.nbytes + self.scales.nbytes
        return self.pair.nbytes + self.tail.nbytes + 16


def random_matrix(seed, rows, cols, mode):
    """mode: b4 / b5 / b6 / nf4 / nf4g128 / nf3 / nf3g128."""
    if mode.startswith("b"):
        planes = int(mode[1])
        data, scales = random_bipolar_bytes(seed, rows, cols, planes)
        return HostMatrix(kind=0, rows=rows, cols=cols, planes=planes, data=data, scales=scales)
    bits, sgc = int(mode[2]), 2 if mode.endswith("g128") else 1
    if (cols // 64) % sgc:
        sgc = 1
    pair, tail = random_nf_bytes(seed, rows, cols, bits, sgc)
    return HostMatrix(kind=2, rows=rows, cols=cols, bits=bits, sgc=sgc, codebook=NF4_DEFAULT if bits == 4 else NF3_DEFAULT,
                      pair=pair, tail=tail)


def rope_table(max_seq, head_dim, theta):
    """build_rope_table (src/model/real_llm.rs:9212-9236): rows [cos(hd/2), sin(hd/2)], inv_freq in f64 -> f32."""
    half = head_dim // 2
    inv_freq = (1.0 / np.power(float(theta), (2.0 * np.arange(half)) / head_dim)).astype(np.float32)
    ang = (np.arange(max_seq, dtype=np.float32)[:, None] * inv_freq[None, :]).astype(np.float32)
    return np.concatenate([np.cos(ang), np.sin(ang)], axis=1).astype(np.float32)


SMOLLM2_135M = dict(hidden=576, layers=30, n_q=9, n_kv=3, head_dim=64, inter=1536, vocab=49152, max_seq=512, eps=1e-5, theta=1e5)


SMOLLM2_1_7B = dict(hidden=2048, layers=24, n_q=32, n_kv=32, head_dim=64, inter=8192, vocab=49152, max_seq=8192 + 64, eps=1e-5, theta=1.3e5)
QWEN2_7B = dict(hidden=3584, layers=28, n_q=28, n_kv=4, head_dim=128, inter=18944, vocab=152064, max_seq=4096 + 64, eps=1e-6, theta=1e6)
P55454 = dict(qkv="b5", o="b5", gate_up="b4", down="b5", head="b4")     # the reference's mixed-plane tier pQOGDH


def random_bf16(seed, n, lo=0x3800, hi=0x3C00):
    """n bf16 values of random sign with magnitudes in [2^-15, 2^-7)."""
    rng = _rng(seed)
    return (rng.integers(lo, hi, n, dtype=np.uint16) | (rng.integers(0, 2, n, dtype=np.uint16) << 15)).astype(np.uint16)


QWEN3_30B_A3B = dict(hidden=2048, layers=48, n_q=32, n_kv=4, head_dim=128, inter=768, vocab=151936, max_seq=6600 + 64, eps=1e-6, theta=1e6)


def random_moe(seed, hidden, n_experts, top_k, d_ff, bits, sgc, norm_topk=True):
    """One sparse-MoE FFN with random expert codes in the reference's .k2tm record form (nf_expert_byte_layout,
    src/model/moe_800b.rs): codebooks at bytes 0 / 16, the gate_up pair stream at 64, the down pair stream at the next
    multiple of 64, records padded to 16 KiB; router weights N(0, 0.02) (near-uniform routing)."""
    cb = _NF_CHUNK[bits]
    gu_chunks, dn_chunks = hidden // 64, d_ff // 64
    gu_bytes = (2 * d_ff // 32) * (-(-gu_chunks // sgc) * 64 + gu_chunks * 2 * cb)
    dn_bytes = (hidden // 32) * (-(-dn_chunks // sgc) * 64 + dn_chunks * 2 * cb)
    gu_off, dn_off = 64, (64 + gu_bytes + 63) // 64 * 64
    rec = (dn_off + dn_bytes + 16383) // 16384 * 16384
    shard = np.zeros(n_experts * rec, np.uint8)
    book = (NF4_DEFAULT if bits == 4 else NF3_DEFAULT).view(np.uint8)
    for e in range(n_experts):
        r = shard[e * rec:(e + 1) * rec]
        r[0:16] = book
        r[16:32] = book
        r[gu_off:gu_off + gu_bytes] = random_nf_bytes(seed * 1009 + 2 * e, 2 * d_ff, hidden, bits, sgc)[0]
        r[dn_off:dn_off + dn_bytes] = random_nf_bytes(seed * 1009 + 2 * e + 1, hidden, d_ff, bits, sgc)[0]
    router = (_rng(seed * 1009 + 7).standard_normal((n_experts, hidden)) * 0.02).astype(np.float32)
    return dict(router_w=router, router_bias=None, n_experts=n_experts, top_k=top_k, norm_topk=norm_topk, d_ff=d_ff, bits=bits, sgc=sgc,
                shard=shard, expert_bytes=rec, scoring=0)


def random_model(cfg, mode, seed=0, modes=None, qkv_bias=False, untied=False, tp=(1, 0), share_layers=False, moe=None, ep=(1, 0)):
    """Engine spec of a dense Llama-shaped model with random codes (decode time does not depend on the values).

    modes: per-matrix formats {qkv, o, gate_up, down, head} overriding `mode`.  tp = (size, rank): the rank-local
    spec of a tensor-parallel group, generated directly in the rank's shapes (what kronos_2t_b200.tp.shard_spec cuts
    out of a whole model); tensor-parallel specs use an untied embedding table.  share_layers: every layer points at
    layer 0's host arrays (each still becomes its own device copy), which keeps multi-billion-parameter specs quick to make.
    moe: dict(n_experts, top_k, d_ff, bits, sgc) - every layer gets a sparse-MoE FFN (random_moe) instead of the dense MLP;
    ep = (size, rank): expert-parallel rank (the whole spec; the engine keeps the experts e % size == rank)."""
    c = dict(cfg)
    tp_size, tp_rank = tp
    md = dict(qkv=mode, o=mode, gate_up=mode, down=mode, head=mode)
    md.update(modes or {})
    h, hd = c["hidden"], c["head_dim"]
    vocab_total = c["vocab"]
    if tp_size > 1:
        from .tp import head_plan
        assert c["inter"] % (64 * tp_size) == 0 and c["vocab"] % (32 * tp_size) == 0
        qh0, nq_l, _, nkv_l = head_plan(c["n_q"], c["n_kv"], tp_size, tp_rank)      # more ranks than kv heads: the kv head is replicated
        c.update(n_q=nq_l, n_kv=nkv_l, inter=c["inter"] // tp_size, vocab=c["vocab"] // tp_size)
        c.update(tp_size=tp_size, tp_rank=tp_rank, vocab_total=vocab_total, o_chunk0=qh0 * hd // 64,
                 down_chunk0=tp_rank * c["inter"] // 64)
        untied = True
    if ep[0] > 1:
        c.update(ep_size=ep[0], ep_rank=ep[1])
    inter = c["inter"]
    q_dim, kv_dim = c["n_q"] * hd, c["n_kv"] * hd
    layers = []
    for l in range(c["layers"]):
        if share_layers and l > 0:
            layers.append(dict(layers[0]))
            continue
        s = seed * 100003 + 10 * l + 1000003 * tp_rank
        bias = None
        if qkv_bias:
            bias = (_rng(s + 5).standard_normal(q_dim + 2 * kv_dim) * 0.02).astype(np.float32)
        ly = dict(input_norm=np.ones(h, np.float32), post_norm=np.ones(h, np.float32), qkv_bias=bias, q_norm=None, k_norm=None,
                  qkv=random_matrix(s + 1, q_dim + 2 * kv_dim, h, md["qkv"]), o=random_matrix(s + 2, h, q_dim, md["o"]))
        if moe:
            ly["moe"] = random_moe(s + 6, h, moe["n_experts"], moe["top_k"], moe["d_ff"], moe["bits"], moe["sgc"])
        else:
            ly.update(gate_up=random_matrix(s + 3, 2 * inter, h, md["gate_up"]), down=random_matrix(s + 4, h, inter, md["down"]))
        layers.append(ly)
    embed = None
    if untied:       # a 4096-row random block, repeated
        blk = random_bf16(seed * 100003 + 8, min(vocab_total, 4096) * h)
        embed = np.tile(blk, -(-vocab_total // 4096))[:vocab_total * h]
    return dict(cfg=c, layers=layers, final_norm=np.ones(h, np.float32),
                lm_head=random_matrix(seed * 100003 + 7 + 1000003 * tp_rank, c["vocab"], h, md["head"]),
                rope=rope_table(c["max_seq"], hd, c["theta"]), embed_bf16=embed)


# Block models (ffi.Engine specs with `blocks`) beside which a Llama shape of the same width, depth, heads and MLP makes sense
FOLIZEN_SHAPES = {
    "small": dict(hidden=1024, layers=12, heads=16, kv_heads=4, dim=64, window=1024, ff=4096, side_dim=32, rank=32, vocab=32768),
    "medium": dict(hidden=2048, layers=24, heads=16, kv_heads=4, dim=128, window=2048, ff=8192, side_dim=64, rank=64, vocab=49152),
    "large": dict(hidden=4096, layers=16, heads=32, kv_heads=8, dim=128, window=4096, ff=14336, side_dim=64, rank=96, vocab=131072),
}


def _block_matrix(rng):
    """mat(rows, cols): random bf16 bit patterns with magnitudes around 1 / sqrt(cols)."""
    def mat(rows, cols):
        base = int(np.float32(cols ** -0.5).view(np.uint32) >> 16) & 0x7F80
        blk = rng.integers(base - 0x80, base + 0x80, min(rows * cols, 1 << 22), dtype=np.uint16) | (rng.integers(0, 2, min(rows * cols, 1 << 22), dtype=np.uint16) << 15)
        return np.resize(blk, rows * cols).reshape(rows, cols)
    return mat


def random_folizen(shape, seed=0, max_seq=8192, layers=None):
    """Engine spec of a block model with random bf16 weights: attention with feed-forward and delta-rule blocks by turns, or attention
    blocks only, with feed-forward sizes by turns, where the shape has ff_turns.  Blocks of a kind point at the same host arrays
    (each still becomes its own device copy)."""
    c = dict(FOLIZEN_SHAPES[shape] if isinstance(shape, str) else shape)
    n = layers or c["layers"]
    h, H, G, d, side = c["hidden"], c["heads"], c["kv_heads"], c["dim"], c["side_dim"]
    mat = _block_matrix(_rng(seed))
    one = lambda k: np.ones(k, np.float32)
    tail = dict(norm1=one(h))
    if side:
        tail.update(side_norm=one(h) * 0.5, side_gate=mat(side, h), side_proj=mat(h, side))

    def attention(ff):
        return dict(tail, mixer=1, heads=H, kv_heads=G, dim=d, vdim=d, window=c["window"], ff=ff, q_norm=one(d), k_norm=one(d), head_scale=one(H) * d ** -0.5,
                    head_slope=(2.0 ** (-8.0 * (np.arange(H) + 1) / H)).astype(np.float32), in_proj=mat((H + 2 * G) * d, h), o_proj=mat(h, H * d), norm2=one(h),
                    act_coef=np.array([0.5, 0.3, 0.2, 0.0], np.float32), up_proj=mat(ff, h), down_proj=mat(h, ff))

    if "ff_turns" in c:
        turns = [attention(ff) for ff in c["ff_turns"]]
    else:
        turns = [attention(c["ff"]), dict(tail, mixer=2, heads=H, dim=d, decay_rank=c["rank"], decay_scale=0.6065307, unit_eps=1e-6, decay_bias=-2.0 * one(H * d),
                                          rate_bias=-1.0 * one(H * d), out_norm=one(H * d), in_proj=mat(5 * H * d + c["rank"], h), decay_proj=mat(H * d, c["rank"]),
                                          o_proj=mat(h, H * d))]
    return dict(cfg=dict(hidden=h, vocab=c["vocab"], max_seq=max_seq, eps=1e-6, side_dim=side, precision=16), blocks=[turns[i % len(turns)] for i in range(n)],
                final_norm=one(h), head=mat(c["vocab"], h), embed=mat(c["vocab"], h), side_embed=mat(c["vocab"], side * n) if side else None)


ZASESUN_SHAPES = {
    "small": dict(hidden=1024, layers=12, heads=16, dim=64, rot_dim=32, vdim=64, q_rank=512, kv_rank=256, ff=4096, experts=32, top=4, expert_ff=704, shared_ff=1408, vocab=32768),
    "medium": dict(hidden=2048, layers=24, heads=16, dim=128, rot_dim=64, vdim=128, q_rank=1024, kv_rank=512, ff=8192, experts=64, top=6, expert_ff=1408, shared_ff=2816, vocab=49152),
    "large": dict(hidden=4096, layers=16, heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512, ff=14336, experts=32, top=4, expert_ff=2048, shared_ff=4096, vocab=131072),
}


def random_zasesun(shape, seed=0, max_seq=8192, layers=None):
    """Engine spec with random bf16 weights: latent attention with a dense and an expert feed-forward by turns."""
    from . import models
    c = dict(ZASESUN_SHAPES[shape] if isinstance(shape, str) else shape)
    n, h, H, d, dr, dv = layers or c["layers"], c["hidden"], c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    mat = _block_matrix(_rng(seed))
    one = lambda k: np.ones(k, np.float32)
    attn = dict(mixer=3, heads=H, dim=d, vdim=dv, rot_dim=dr, kv_rank=c["kv_rank"], q_rank=c["q_rank"], score_scale=(d + dr) ** -0.5,
                rot_cos_sin=models.rotation_table(max_seq, dr, dr, 1e4, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)), q_latent_norm=one(c["q_rank"]),
                kv_latent_norm=one(c["kv_rank"]), pre_norm1=one(h), norm1=one(h), in_proj=mat(c["q_rank"] + c["kv_rank"] + dr, h), q_up=mat(H * (d + dr), c["q_rank"]),
                kv_up=mat(H * (d + dv), c["kv_rank"]), o_proj=mat(h, H * dv), pre_norm2=one(h), norm2=one(h))
    E, ff, sh = c["experts"], c["expert_ff"], c["shared_ff"]
    turns = [dict(attn, act=1, ff=c["ff"], up_proj=mat(2 * c["ff"], h), down_proj=mat(h, c["ff"])),
             dict(attn, act=2, ff=ff, experts=E, experts_top=c["top"], shared_ff=sh, up_proj=mat(E * ff, h), down_proj=mat(E * h, ff), router=mat(E + sh, h), shared_down=mat(h, sh))]
    table = mat(c["vocab"], h)
    return dict(cfg=dict(hidden=h, vocab=c["vocab"], max_seq=max_seq, eps=1e-6, residual_mult=0.5, logit_softcap=30.0, precision=16),
                blocks=[turns[i % 2] for i in range(n)], final_norm=one(h), head=table, embed=table)


def zasesun_like(shape):
    """The Folizen shape of equal width, depth, heads and active feed-forward sizes: attention over every position, as many
    key/value heads as give the nearest cache (one eighth of the query heads, at least one)."""
    c = dict(ZASESUN_SHAPES[shape] if isinstance(shape, str) else shape)
    return dict(hidden=c["hidden"], layers=c["layers"], heads=c["heads"], kv_heads=max(1, c["heads"] // 8), dim=c["dim"], window=0, side_dim=0, vocab=c["vocab"],
                ff_turns=[c["ff"] * 3 // 2, c["top"] * c["expert_ff"] + c["shared_ff"]])
