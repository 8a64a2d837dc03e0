"""The Zasesun design on the device against the plain restatement in zasesun_ref.py: every mechanism alone, whole models, prompts
against token-by-token decoding, portions, keys at tile edges and far away, reused caches, long decoding, snapshots, greedy generation.
Mistakes are planted in the restatement, to show that the comparisons would see them."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import folizen_models as fm
import folizen_ref
import zasesun_models as zm
import zasesun_ref as ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 3e-5, "bfloat16": 5e-2}


@pytest.fixture(scope="module")
def ctx():
    import kronos_2t_b200 as k2
    c = k2.Context(0)
    yield c
    c.close()


@pytest.fixture
def engine(ctx, tmp_path):
    """engine(model, dtype) from a model folder through the registry."""
    from kronos_2t_b200 import models
    made = []

    def make(model, dtype="float32", max_seq=1536):
        folder = fm.write(model, str(tmp_path / f"m{len(made)}"))
        made.append(models.load_engine(ctx, folder, dtype, max_seq))
        return made[-1]

    yield make
    for e in made:
        e.close()


CLOSE = 0.03          # rounding moves a router logit by about a hundredth


def router_margins(model, toks):
    margins = []
    ref.forward(model, toks, margins)
    return np.min(margins, axis=0) if margins else np.full(len(toks), np.inf)


def tokens_of(model, n, seed=1):
    """Random tokens none of whose expert choices is a close call: in bf16 such a token may take another expert."""
    rng = np.random.default_rng(seed)
    toks = rng.integers(0, model["config"]["vocab"], n)
    for _ in range(50):
        close = router_margins(model, toks) < CLOSE
        if not close.any():
            return toks
        toks[close] = rng.integers(0, model["config"]["vocab"], close.sum())
    raise AssertionError("no sequence without a close call found")


def portions(eng, toks, sizes):
    out, at = [], 0
    while at < len(toks):
        for s in sizes:
            n = min(s, len(toks) - at)
            if n == 0:
                break
            out.append(eng.forward_token_ids(toks[at:at + n], pos_start=at, want_all=True))
            at += n
    return np.concatenate(out)


def decoded(eng, toks, at=0):
    return np.stack([eng.forward_token_ids([t], pos_start=at + i) for i, t in enumerate(toks[at:])])


ALONE = {
    "attention": zm.latent(4, 32, 16, 24, 40, 48),
    "scaled rotation": zm.latent(3, 16, 12, 16, 30, 32, scaling=zm.YARN, base=700.0),
    "odd sizes": zm.latent(3, 21, 6, 37, 33, 70, scale=0.4),
    "one head": zm.latent(1, 64, 2, 64, 17, 24),
    "more heads than a tile has rows": zm.latent(40, 16, 8, 8, 24, 32),
    "long rows": zm.latent(2, 136, 64, 200, 90, 130),
    "head larger than a panel group": zm.latent(2, 300, 80, 256, 64, 200),
    "values too long for the prompt kernel": zm.latent(2, 40, 8, 300, 32, 64),
    "wide latent": zm.latent(5, 48, 32, 40, 64, 320),
    "wider latent": zm.latent(2, 32, 16, 32, 64, 700),
    "gated feed-forward": zm.latent(2, 16, 8, 16, 16, 16, zm.dense(300)),
    "odd feed-forward": zm.latent(2, 16, 8, 16, 16, 16, zm.dense(33)),
    "experts": zm.latent(2, 16, 8, 16, 16, 16, zm.moe(9, 3, 40, shared=52)),
    "experts, none shared": zm.latent(2, 16, 8, 16, 16, 16, zm.moe(20, 4, 33)),
    "every expert": zm.latent(2, 16, 8, 16, 16, 16, zm.moe(4, 4, 72, shared=8)),
    "a single expert": zm.latent(2, 16, 8, 16, 16, 16, zm.moe(1, 1, 24, shared=130)),
    "many experts, one taken": zm.latent(2, 16, 8, 16, 16, 16, zm.moe(150, 1, 16, shared=24)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALONE))
def test_one_block(engine, name, dtype):
    model = zm.make(168, 211, [ALONE[name]], seed=len(name))
    toks = tokens_of(model, 190)
    want, streams = ref.forward(model, toks)
    eng = engine(model, dtype)
    assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]
    assert np.abs(eng.read_hidden() - streams[-1][-1]).max() / np.std(streams[-1]) < 4 * TOL[dtype]
    assert fm.error(decoded(eng, toks[:70]), want[:70]).max() < TOL[dtype]
    assert fm.error(portions(eng, toks, [20, 11, 100]), want).max() < TOL[dtype]


MIXED = {
    # width, vocab, eps, residual factor, cap, layers: sizes that differ from layer to layer, none a multiple of the kernels' tiles
    "uneven": (200, 331, 1e-5, 0.7, 9.0, [zm.latent(6, 40, 12, 24, 56, 72, zm.moe(7, 2, 44, shared=36), scaling=zm.YARN), zm.latent(3, 24, 20, 48, 30, 40, zm.dense(264)),
                                          zm.latent(2, 72, 8, 72, 100, 36)]),
    "narrow": (68, 97, 1e-6, 1.0, 30.0, [zm.latent(1, 36, 4, 28, 10, 12, zm.dense(70)), zm.latent(3, 8, 8, 12, 20, 20, zm.moe(3, 1, 12))]),
    "wide": (640, 1000, 1e-6, 0.4, 25.0, [zm.latent(8, 64, 32, 64, 192, 128, zm.dense(1100)), zm.latent(16, 48, 16, 64, 160, 256, zm.moe(9, 2, 160, shared=200), base=3e4),
                                          zm.latent(8, 64, 32, 64, 192, 128, zm.moe(6, 2, 300, shared=100))]),
}


def mixed(name, seed=3):
    w, v, eps, mult, cap, layers = MIXED[name]
    return zm.make(w, v, copy.deepcopy(layers), eps=eps, mult=mult, cap=cap, seed=seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MIXED))
def test_whole_prompt_decoding_and_portions(engine, name, dtype):
    model = mixed(name)
    toks = tokens_of(model, 300)
    want, _ = ref.forward(model, toks)
    eng = engine(model, dtype)
    assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < TOL[dtype], "whole prompt"
    assert fm.error(decoded(eng, toks), want).max() < TOL[dtype], "token by token"
    for sizes in ([2], [2, 3, 1, 7], [16, 17, 5], [64, 1, 1, 33], [129, 2], [127, 65, 2]):
        assert fm.error(portions(eng, toks, sizes), want).max() < TOL[dtype], sizes


def test_portions_agree_closely_in_bf16(engine):
    """The cut of a prompt changes the rounding only, although prompts and short portions take different kernels."""
    model = mixed("wide")
    toks = tokens_of(model, 260)
    eng = engine(model, "bfloat16")
    whole = eng.forward_token_ids(toks, want_all=True).astype(np.float64)
    for sizes in ([2], [150, 1, 20]):
        assert fm.error(portions(eng, toks, sizes), whole).max() < 3e-2


# ---- one key stands out, placed at tile edges (64 and 128 positions), at the first tokens and far away
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portions"])
def test_a_far_key(engine, how, dtype):
    model = zm.pointer()
    eng = engine(model, dtype)
    n = 700
    base = np.random.default_rng(4).integers(3, 40, n)
    plain, _ = ref.forward(model, np.concatenate([base[:-1], [2]]))
    for at in (0, 1, 63, 64, 127, 128, 129, 383, 511, 512, 575, 576, 639, 640, 697, 698):
        toks = base.copy()
        toks[at], toks[-1] = 1, 2
        want, _ = ref.forward(model, toks)
        assert fm.error(plain, want)[-1] > 10 * TOL[dtype]          # without the key the last logits are far off
        if how == "prompt":
            got = eng.forward_token_ids(toks, want_all=True)
        elif how == "decoded":
            eng.forward_token_ids(toks[:690])
            got = np.concatenate([want[:690], decoded(eng, toks, 690)])
        else:
            got = portions(eng, toks, [at + 1, 2, 131] if at else [2, 131])
        assert fm.error(got, want)[-1] < TOL[dtype], at


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_seen_from_a_prompt_batch_behind_it(engine, dtype):
    """The query in the middle of a portion of 100 that starts far behind the key; and the key in the portion itself."""
    model = zm.pointer(heads=3, dim=40, vdim=24, kv_rank=80)
    eng = engine(model, dtype)
    for at in (5, 300, 330):
        toks = np.random.default_rng(at).integers(3, 40, 400)
        toks[at], toks[350] = 1, 2
        want, _ = ref.forward(model, toks)
        eng.forward_token_ids(toks[:300])
        e = fm.error(eng.forward_token_ids(toks[300:], pos_start=300, want_all=True), want[300:])
        assert e[50] < TOL[dtype] and e.max() < 2 * TOL[dtype]          # most weight of a noise token is its attention's, normed and doubled


@pytest.mark.parametrize("heads", [4, 70])
def test_long_context_by_both_ways(engine, heads):
    """Nine thousand positions: splits of several tiles, prompt batches that follow one another.  A prompt's last tokens (keys and
    values expanded) against the same tokens decoded (in latent space); the key far back is what the last one looks at."""
    model = zm.pointer(heads=heads)
    eng = engine(model, "bfloat16", max_seq=9100)
    toks = np.random.default_rng(1).integers(3, 40, 9000)
    toks[[5, -1]] = 1, 2
    eng.forward_token_ids(toks[:8900])
    tail = eng.forward_token_ids(toks[8900:], pos_start=8900, want_all=True)
    eng.forward_token_ids(toks[:8996])
    assert fm.error(decoded(eng, toks, 8996), tail[96:]).max() < 3e-2
    toks[5] = 9
    eng.forward_token_ids(toks[:8999])
    assert fm.error(decoded(eng, toks, 8999), tail[99:]).max() > 0.2


def planted(model, change):
    """Error that a restatement with `change` applied to its configuration or tensors would show."""
    other = copy.deepcopy(model)
    change(other)
    return other


def test_constants_show(engine):
    """Rotation, scales, residual factor, cap and epsilon: the device agrees, a restatement with any of them changed does not."""
    model = zm.make(96, 120, [zm.latent(4, 16, 16, 24, 40, 32, zm.moe(6, 2, 40, shared=24), scaling=zm.YARN), zm.latent(2, 24, 8, 16, 20, 28, zm.dense(64))], eps=1e-2, mult=0.6, cap=8.0, seed=5)
    toks = tokens_of(model, 200)
    want, _ = ref.forward(model, toks)
    for dtype in ("float32", "bfloat16"):
        assert fm.error(engine(model, dtype).forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]

    def rot(**kw):
        return lambda o: o["config"]["layers"][0]["mixer"]["rot"].update(**kw)

    def scaling(**kw):
        return lambda o: o["config"]["layers"][0]["mixer"]["rot"]["scaling"].update(**kw)

    def config(**kw):
        return lambda o: o["config"].update(**kw)

    def swap(a, b):
        return lambda o: o["tensors"].update({a: o["tensors"][b], b: o["tensors"][a]})

    for change in (rot(base=9e3), rot(scaling=None), scaling(factor=5.0), scaling(original=960), scaling(fast=3.0), scaling(slow=0.2), config(residual_mult=0.62),
                   config(logit_softcap=8.2), config(norm=dict(eps=5e-3)), lambda o: o["config"]["layers"][0]["mixer"].update(scale=0.17),
                   lambda o: o["config"]["layers"][0]["mlp"]["router"].update(top=1), swap("l0.norm1", "l0.norm1b"), swap("l0.norm2", "l0.norm2b"),
                   swap("l1.mlp.gate", "l1.mlp.up"), swap("l0.mlp.e0.up", "l0.mlp.e1.up")):
        assert fm.error(ref.forward(planted(model, change), toks)[0], want).max() > 20 * TOL["float32"]


def test_mechanisms_show(engine):
    """The same with a mechanism replaced in the restatement."""
    model = zm.make(96, 120, [zm.latent(4, 16, 16, 24, 40, 32, zm.moe(6, 2, 40, shared=24), scaling=zm.YARN)], seed=6)
    toks = tokens_of(model, 150)
    want, _ = ref.forward(model, toks)
    assert fm.error(engine(model).forward_token_ids(toks, want_all=True), want).max() < TOL["float32"]
    kept = {n: getattr(ref, n) for n in ("rotate", "rotation", "route", "relu_squared", "rms_norm")}

    def halves(x, positions, rot):          # pairs (i, i + dims / 2) instead of neighbours
        order = np.concatenate([np.arange(0, rot["dims"], 2), np.arange(1, rot["dims"], 2)])
        back = np.argsort(order)
        return kept["rotate"](x[..., back], positions, rot)[..., order]

    def renormalized(z, top):
        c, w = kept["route"](z, top)
        return c, w / w.sum(-1, keepdims=True)

    wrong = dict(rotate=halves, rotation=lambda rot: (kept["rotation"](rot)[0], 1.0), route=renormalized, relu_squared=lambda z: np.maximum(z, 0.0),
                 rms_norm=lambda x, w, eps: x / (np.sqrt(np.mean(x * x, -1, keepdims=True)) + 1e-2) * w)
    for name, fn in wrong.items():
        try:
            setattr(ref, name, fn)
            assert fm.error(ref.forward(model, toks)[0], want).max() > 20 * TOL["float32"], name
        finally:
            setattr(ref, name, kept[name])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [16, 48, 128])
def test_prompt_batches(engine, monkeypatch, batch, dtype):
    """A prompt cut into batches by the engine itself: later batches attend to the cache that the earlier ones left."""
    monkeypatch.setenv("KRONOS_CUDA_PROMPT_BATCH", str(batch))
    model = mixed("uneven")
    toks = tokens_of(model, 333)
    want, _ = ref.forward(model, toks)
    eng = engine(model, dtype, max_seq=340)
    assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]
    assert fm.error(portions(eng, toks, [batch + 1, 2, 3 * batch]), want).max() < TOL[dtype]


def test_sequences_follow_one_another(engine):
    """A new sequence starts from nothing, whatever ran before; the same sequence gives the same bits again; an earlier position can be
    continued from."""
    import kronos_2t_b200 as k2
    model = mixed("uneven")
    eng = engine(model, "bfloat16")
    a, b = tokens_of(model, 240, 1), tokens_of(model, 90, 2)
    first = eng.forward_token_ids(a, want_all=True)
    alone = eng.forward_token_ids(b, want_all=True)
    eng.decode_greedy(3, 90, 50)
    assert np.array_equal(eng.forward_token_ids(a, want_all=True), first)
    assert eng.can_truncate_kv_to(240, 240) and eng.can_truncate_kv_to(240, 12) and not eng.can_truncate_kv_to(240, 241)
    tail = eng.forward_token_ids(b[30:], pos_start=30, want_all=True)          # the first 30 of a, then b
    both = np.concatenate([a[:30], b[30:]])
    calm = router_margins(model, both)[30:] > CLOSE
    assert fm.error(tail, ref.forward(model, both)[0][30:])[calm].max() < 2 * TOL["bfloat16"]
    with pytest.raises(k2.KronosCudaError, match="position 90"):
        eng.forward_token_ids([1, 2], pos_start=91)
    assert np.array_equal(eng.forward_token_ids(b, want_all=True), alone)


def test_repeats_bit_for_bit(engine):
    """The kernels' order of additions is fixed: thirty repeats of a prompt in two portions, and of a few decoded tokens."""
    model = mixed("wide")
    eng = engine(model, "bfloat16")
    toks = tokens_of(model, 260)

    def run():
        a = eng.forward_token_ids(toks[:150], want_all=True)
        b = eng.forward_token_ids(toks[150:250], pos_start=150, want_all=True)
        return np.concatenate([a, b, decoded(eng, toks, 250)])

    first = run()
    for _ in range(30):
        assert np.array_equal(run(), first)


def test_first_tokens(engine):
    model = mixed("uneven")
    for n in (1, 2, 3, 17, 64, 65):
        toks = tokens_of(model, n, seed=n)
        want, _ = ref.forward(model, toks)
        for dtype in ("float32", "bfloat16"):
            assert fm.error(engine(model, dtype).forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]


def test_full_cache(engine):
    """The last position of the cache, by prompt and by decoding."""
    model = mixed("narrow")
    toks = tokens_of(model, 200)
    want, _ = ref.forward(model, toks)
    for dtype in ("float32", "bfloat16"):
        eng = engine(model, dtype, max_seq=200)
        assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]
        eng.forward_token_ids(toks[:190])
        assert fm.error(decoded(eng, toks, 190), want[190:]).max() < TOL[dtype]


def test_snapshot(engine):
    model = mixed("uneven")
    eng = engine(model, "bfloat16")
    toks = tokens_of(model, 220)
    eng.forward_token_ids(toks[:130])
    blob = eng.save_kv_prefix(130, 130)
    rest = eng.forward_token_ids(toks[130:], pos_start=130, want_all=True)
    eng.forward_token_ids(toks[::-1].copy())
    eng.restore_kv_prefix(blob)
    assert np.array_equal(eng.forward_token_ids(toks[130:], pos_start=130, want_all=True), rest)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation(engine, dtype):
    """generate() against the restatement: every chosen token has the reference's largest logit, up to rounding."""
    from kronos_2t_b200 import models
    model = mixed("uneven")
    eng = engine(model, dtype)
    prompt = tokens_of(model, 80)
    new = models.generate(eng, prompt, 150)
    seq = np.concatenate([prompt, new])
    want, _ = ref.forward(model, seq)
    calm = router_margins(model, seq) > CLOSE
    for i, tok in enumerate(new):
        row = want[len(prompt) - 1 + i]
        if dtype == "float32" or calm[len(prompt) - 1 + i]:
            assert row.max() - row[tok] < 6 * TOL[dtype] * row.std(), i
    # the captured step and the profile of one leave the sequence as it was
    table = eng.profile_step(int(new[-1]), len(seq) - 1, 2)
    assert "latent norms" in table and "experts down" in table
    more = eng.forward_token_ids([int(new[-1])], pos_start=len(seq) - 1)
    assert fm.error(more[None], want[-1:]).max() < 2 * TOL[dtype] or (dtype == "bfloat16" and not calm[-1])


def test_long_decoding(engine):
    model = mixed("narrow")
    eng = engine(model, "float32")
    new = eng.decode_greedy(5, 0, 700)
    seq = np.concatenate([[5], new[:-1]])
    want, _ = ref.forward(model, seq)
    assert fm.error(eng.forward_token_ids(seq, want_all=True), want).max() < 1e-4
    picked = np.take_along_axis(want, new[:, None].astype(int), 1)[:, 0]
    assert ((want.max(1) - picked) / want.std(1)).max() < 2e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mechanisms_mix_with_other_blocks(ctx, dtype):
    """Window attention and latent attention, a polynomial feed-forward, gated and squared experts in one model of no named design."""
    import kronos_2t_b200 as k2
    from kronos_2t_b200 import ffi, models
    width, eps, mult = 72, 1e-5, 0.8
    layers = [zm.latent(3, 16, 8, 20, 24, 28, zm.moe(5, 2, 24, shared=16)), zm.latent(2, 16, 8, 16, 16, 20, zm.dense(40))]
    z = zm.make(width, 90, layers, eps=eps, mult=mult, seed=2)
    f = fm.make(width, 90, [fm.attention(4, 2, 16, 24, 19, ff=56)], side=4, eps=eps, seed=3)
    W = {k: np.asarray(v, np.float64) for k, v in z["tensors"].items()}
    V = {k: np.asarray(v, np.float64) for k, v in f["tensors"].items()}
    rng = np.random.default_rng(0)
    gates = fm.bf16(rng.standard_normal((5 * 24 + 16, width)) / np.sqrt(width))          # makes the experts of layer 0 gated ones

    def part(T, prefix):
        return {k[len(prefix):]: v for k, v in T.items() if k.startswith(prefix)}

    toks = np.random.default_rng(1).integers(0, 90, 160)
    x = W["embed"][toks]
    n = part(W, "l0.")
    x = x + mult * ref.rms_norm(ref.latent_attention(ref.rms_norm(x, n["norm1"], eps), part(W, "l0.mix."), layers[0]["mixer"], eps), n["norm1b"], eps)
    h = ref.rms_norm(x, n["norm2"], eps)
    z_router = h @ n["mlp.router"].T
    chosen, weight = ref.route(z_router, 2)
    seen = slice(None) if dtype == "float32" else ref.margin(z_router, 2) > CLOSE
    y = (ref.gelu_tanh(h @ gates[120:].T) * (h @ n["mlp.shared.up"].T)) @ n["mlp.shared.down"].T
    for t in range(160):
        for e, w in zip(chosen[t], weight[t]):
            y[t] += w * ((ref.gelu_tanh(gates[24 * e:24 * e + 24] @ h[t]) * (n[f"mlp.e{e}.up"] @ h[t])) @ n[f"mlp.e{e}.down"].T)
    x = x + mult * ref.rms_norm(y, n["norm2b"], eps)
    x = x + mult * ref.rms_norm(folizen_ref.attention_mixer(x, part(V, "l0.mix."), f["config"]["layers"][0]["mixer"], eps), V["l0.norm1"], eps)      # no norm in front
    x = x + mult * ref.rms_norm(folizen_ref.dense_mlp(x, part(V, "l0.mlp."), eps), V["l0.norm2"], eps)
    want = ref.rms_norm(x, W["final.norm"], eps) @ W["embed"].T

    mat = ffi.bf16_bits if dtype == "bfloat16" else (lambda a: np.asarray(a, np.float32))
    t, u, m, g = z["tensors"], f["tensors"], layers[0]["mixer"], f["config"]["layers"][0]["mixer"]
    pairs = lambda gate, up: np.stack([gate, up], 1).reshape(-1, width)
    first = dict(mixer=ffi.MIXER_LATENT_ATTENTION, heads=3, dim=16, rot_dim=8, vdim=20, q_rank=24, kv_rank=28, score_scale=m["scale"], rot_cos_sin=models.rotation_table(256, 8, 8, 1e4),
                 q_latent_norm=t["l0.mix.dq.norm"], kv_latent_norm=t["l0.mix.dkv.norm"], pre_norm1=t["l0.norm1"], norm1=t["l0.norm1b"], pre_norm2=t["l0.norm2"], norm2=t["l0.norm2b"],
                 in_proj=mat(np.concatenate([t["l0.mix.dq"], t["l0.mix.dkv"]])), q_up=mat(t["l0.mix.uq"]), kv_up=mat(np.concatenate([t["l0.mix.uk"], t["l0.mix.uv"]])),
                 o_proj=mat(t["l0.mix.o"]), act=ffi.ACT_GELU_GATED, experts=5, experts_top=2, ff=24, shared_ff=16,
                 up_proj=mat(np.concatenate([pairs(gates[24 * e:24 * e + 24], t[f"l0.mlp.e{e}.up"]) for e in range(5)])),
                 down_proj=mat(np.concatenate([t[f"l0.mlp.e{e}.down"] for e in range(5)])), shared_down=mat(t["l0.mlp.shared.down"]),
                 router=mat(np.concatenate([t["l0.mlp.router"], pairs(gates[120:], t["l0.mlp.shared.up"])])))
    second = dict(mixer=ffi.MIXER_WINDOW_ATTENTION, heads=4, kv_heads=2, dim=16, vdim=24, window=19, ff=56, act=ffi.ACT_POLYNORM, norm1=u["l0.norm1"], norm2=u["l0.norm2"],
                  q_norm=u["l0.mix.q.norm"], k_norm=u["l0.mix.k.norm"], head_scale=np.float32(g["scale"]) * u["l0.mix.temp"], head_slope=models.alibi_slopes(4), act_coef=u["l0.mlp.act"],
                  in_proj=mat(np.concatenate([u["l0.mix.q"], u["l0.mix.k"], u["l0.mix.v"]])), o_proj=mat(u["l0.mix.o"]), up_proj=mat(u["l0.mlp.up"]), down_proj=mat(u["l0.mlp.down"]))
    eng = k2.Engine(ctx, dict(cfg=dict(hidden=width, vocab=90, max_seq=256, eps=eps, residual_mult=mult, precision=16 if dtype == "bfloat16" else 32), blocks=[first, second],
                              final_norm=t["final.norm"], head=mat(t["embed"]), embed=ffi.bf16_bits(t["embed"])))
    try:
        for got in (eng.forward_token_ids(toks, want_all=True), decoded(eng, toks), portions(eng, toks, [50, 3])):
            assert fm.error(got, want)[seen].max() < TOL[dtype]
    finally:
        eng.close()


def test_creation_refuses_bad_descriptions(ctx, tmp_path):
    import kronos_2t_b200 as k2
    from kronos_2t_b200 import models
    folder = fm.write(zm.make(40, 50, [zm.latent(2, 16, 8, 16, 16, 20, zm.moe(4, 2, 8, shared=8))]), str(tmp_path / "m"))
    for change, why in ((dict(experts_top=5), "experts"), (dict(score_scale=0.0), "score_scale"), (dict(rot_dim=7), "odd"), (dict(act=0), "experts take"), (dict(kv_rank=1100), "kv_rank")):
        spec = models.load_spec(folder, "bfloat16", 64)
        spec["blocks"][0].update(change)
        with pytest.raises(k2.KronosCudaError, match=why):
            k2.Engine(ctx, spec)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    model = mixed("narrow")
    folder = fm.write(model, str(tmp_path / "model"))
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens_of(model, 30, 1), tokens_of(model, 9, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:20].tolist(), want=[0, 19])], end=[]), dict(step=1, entries=[dict(id="a", tokens=[int(a[20])], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[21:].tolist(), want=[8])], end=["a"]), dict(step=3, entries=[dict(id="b", tokens=b.tolist(), want=[8, 3])], end=["b"])]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    wa, wb = ref.forward(model, a)[0], ref.forward(model, b)[0]
    for n, want in ((0, wa[[0, 19]]), (2, wa[[29]]), (3, wb[[8, 3]])):
        got = np.fromfile(out / f"{n}.f32", "<f4").reshape(want.shape)
        assert fm.error(got, want).max() < TOL[dtype]
    assert not (out / "1.f32").exists()


def test_command_line(tmp_path):
    model = mixed("narrow")
    folder = fm.write(model, str(tmp_path / "model"))
    p = subprocess.run([sys.executable, os.path.join(ROOT, "kronos_2t_b200.py"), "generate", "--model", folder, "--tokens", "5,6,7", "--steps", "6", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    new = [int(t) for t in p.stdout.strip().splitlines()[-1].split(",")]
    want, _ = ref.forward(model, [5, 6, 7] + new[:-1])
    assert new == [int(np.argmax(r)) for r in want[2:]]
