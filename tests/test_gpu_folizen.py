"""The Folizen design on the device (kronos_cuda_engine_create_blocks) against the plain restatement in folizen_ref.py: every
mechanism alone, whole models, prompts against token-by-token decoding, portions, window edges, reused state, long decoding,
snapshots and greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import folizen_models as fm
import folizen_ref as ref

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

    def make(model, dtype="float32", max_seq=2048):
        folder = fm.write(model, str(tmp_path / f"m{len(made)}"))
        made.append(models.load_engine(ctx, folder, dtype, max_seq))
        return made[-1]

    yield make
    for e in made:
        e.close()


def tokens_of(model, n, seed=1):
    return np.random.default_rng(seed).integers(0, model["config"]["vocab"], n)


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


ALONE = {
    "attention": [fm.attention(4, 2, 32, 32, 20)],
    "attention, one kv head, value size apart": [fm.attention(6, 1, 48, 80, 33)],
    "attention, as many kv heads, long rows": [fm.attention(3, 3, 136, 200, 70, scale=0.05)],
    "attention, large group": [fm.attention(20, 1, 16, 24, 50)],
    "attention, itself only": [fm.attention(2, 1, 16, 16, 1)],
    "delta": [fm.delta(3, 32)],
    "delta, odd sizes": [fm.delta(2, 44, rank=70)],
    "delta, large head": [fm.delta(2, 128, rank=16)],
    "delta, larger head": [fm.delta(1, 200, rank=3)],
    "polynomial feed-forward": [fm.delta(1, 16, ff=300)],
    "long feed-forward": [fm.attention(1, 1, 16, 16, 8, ff=9000)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALONE))
def test_one_block(engine, name, dtype):
    model = fm.make(160, 211, ALONE[name], side=12, seed=len(name))
    toks = tokens_of(model, 150)
    want, streams = ref.forward(model, toks)
    eng = engine(model, dtype)
    got = eng.forward_token_ids(toks, want_all=True)
    assert fm.error(got, want).max() < TOL[dtype]
    x = eng.read_hidden()
    assert np.abs(x - streams[-1][-1]).max() / np.std(streams[-1]) < 4 * TOL[dtype]
    one = np.stack([eng.forward_token_ids([t], pos_start=i) for i, t in enumerate(toks[:60])])
    assert fm.error(one, want[:60]).max() < TOL[dtype]


MIXED = {
    # width, vocab, side, eps, layers: sizes that differ from layer to layer, none a multiple of the kernels' tiles
    "uneven": (200, 331, 12, 1e-5, [fm.attention(6, 2, 40, 24, 37, ff=264), fm.delta(3, 48), fm.delta(2, 20, ff=96), fm.attention(2, 2, 72, 72, 90)]),
    "narrow": (68, 97, 5, 1e-6, [fm.delta(1, 36, ff=70, rank=3), fm.attention(3, 1, 28, 36, 5)]),
    "wide": (640, 1000, 40, 1e-6, [fm.attention(8, 4, 64, 64, 128, ff=1100), fm.delta(4, 96, rank=33), fm.attention(4, 1, 128, 128, 64, ff=512)]),
}


def mixed(name, seed=3):
    w, v, side, eps, layers = MIXED[name]
    return fm.make(w, v, layers, side=side, eps=eps, seed=seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MIXED))
def test_whole_prompt_decoding_and_portions(engine, name, dtype):
    model = mixed(name)
    toks = tokens_of(model, 230)
    want, _ = ref.forward(model, toks)
    eng = engine(model, dtype)
    whole = eng.forward_token_ids(toks, want_all=True)
    assert fm.error(whole, want).max() < TOL[dtype], "whole prompt"
    one = np.stack([eng.forward_token_ids([t], pos_start=i) for i, t in enumerate(toks)])
    assert fm.error(one, want).max() < TOL[dtype], "token by token"
    for sizes in ([2], [2, 3, 1, 7], [16, 17, 5], [64, 1, 1, 33], [100, 2]):
        assert fm.error(portions(eng, toks, sizes), want).max() < TOL[dtype], sizes


def test_portions_agree_closely_in_bf16(engine):
    """The cut of a prompt changes the rounding only; both cuts read the same rows and state."""
    model = mixed("wide")
    toks = tokens_of(model, 200)
    eng = engine(model, "bfloat16")
    whole = eng.forward_token_ids(toks, want_all=True).astype(np.float64)
    for sizes in ([2], [50, 1, 20]):
        assert fm.error(portions(eng, toks, sizes), whole).max() < 3e-2


# ---- window edges: one key stands out, placed by distance
def pointer_model(window, dtype_seed=0):
    """Token 1 carries a value and the key that token 2's query looks for; all other tokens are noise.  With the score scaled up
    a visible token 1 takes most of the weight whatever its distance."""
    model = fm.make(96, 40, [fm.attention(4, 2, 32, 32, window, scale=1.0)], side=4, seed=9 + dtype_seed)
    t = model["tensors"]
    rng = np.random.default_rng(5)
    dirs = np.linalg.qr(rng.standard_normal((96, 3)))[0].T
    t["embed"][:] = fm.bf16(t["embed"] - t["embed"] @ dirs[:2].T @ dirs[:2])          # the others have no part in the two directions
    t["embed"][1], t["embed"][2] = fm.bf16(30 * dirs[0]), fm.bf16(30 * dirs[1])
    for h in range(4):          # the same unit direction for the query of token 2 and the key of token 1
        u = np.sign(rng.standard_normal(32)) if h % 2 == 0 else u
        t["l0.mix.q"][h * 32:(h + 1) * 32] = fm.bf16(0.3 * t["l0.mix.q"][h * 32:(h + 1) * 32] + np.outer(u, dirs[1]))
        if h % 2 == 0:
            g = h // 2
            t["l0.mix.k"][g * 32:(g + 1) * 32] = fm.bf16(0.3 * t["l0.mix.k"][g * 32:(g + 1) * 32] + np.outer(u, dirs[0]))
    t["l0.mix.q.norm"][:] = t["l0.mix.k.norm"][:] = 1.0
    t["l0.mix.temp"][:] = [3.0, 3.0, 2.0, 2.0]
    return model


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [2, 16, 63, 64, 65, 130])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portions"])
def test_window_edge(engine, window, how, dtype):
    model = pointer_model(window)
    n = window + 60
    eng = engine(model, dtype)
    for dist in sorted({1, window // 2, window - 1, window, window + 1}):
        toks = tokens_of(model, n, seed=dist) % 37 + 3
        at = n - 1 - dist
        toks[at], toks[-1] = 1, 2
        want, _ = ref.forward(model, toks)
        if how == "prompt":
            got = eng.forward_token_ids(toks, want_all=True)
        elif how == "decoded":
            head = eng.forward_token_ids(toks[:at + 1], want_all=True)
            got = np.concatenate([head] + [eng.forward_token_ids([t], pos_start=at + 1 + i)[None] for i, t in enumerate(toks[at + 1:])])
        else:
            got = portions(eng, toks, [window - 1, 2, 19] if window > 2 else [2, 3])
        assert fm.error(got, want)[-1] < TOL[dtype], (dist, "seen" if dist < window else "not seen")
        # the planted neighbours of the rule do not pass: one position more, one less
        for wrong in (window - 1, window + 1):
            if (dist < window) == (dist < wrong):
                continue
            other = json.loads(json.dumps(model["config"]))
            other["layers"][0]["mixer"]["mask"]["size"] = wrong
            bad, _ = ref.forward(dict(config=other, tensors=model["tensors"]), toks)
            assert fm.error(bad, want)[-1] > 3 * TOL[dtype]


def test_bias_and_temperature_show(engine):
    """Slopes and temperatures belong to their heads: a restatement with them permuted or left out is far away."""
    model = fm.make(96, 50, [fm.attention(4, 2, 32, 32, 40)], side=4, seed=2)
    model["tensors"]["l0.mix.temp"][:] = [0.5, 1.0, 2.0, 4.0]
    toks = tokens_of(model, 80)
    want, _ = ref.forward(model, toks)
    assert fm.error(engine(model).forward_token_ids(toks, want_all=True), want).max() < TOL["float32"]
    wrong = dict(config=model["config"], tensors=dict(model["tensors"]))
    wrong["tensors"]["l0.mix.temp"] = model["tensors"]["l0.mix.temp"][::-1].copy()
    assert fm.error(ref.forward(wrong, toks)[0], want).max() > 1e-2
    slopes = ref.bias_slopes
    try:
        ref.bias_slopes = lambda h: slopes(h)[::-1]
        assert fm.error(ref.forward(model, toks)[0], want).max() > 1e-2
    finally:
        ref.bias_slopes = slopes


def test_state_far_back(engine):
    """A channel that hardly decays carries a token's value over a thousand tokens, through prompts and decoding."""
    model = fm.make(64, 30, [fm.delta(2, 32, rank=4)], side=4, seed=4)
    t = model["tensors"]
    t["l0.mix.w0"][:] = -12.0
    t["l0.mix.a.b"][:] = -9.0
    t["l0.mix.v"][:] = fm.bf16(0.02 * t["l0.mix.v"])
    t["embed"][1] = fm.bf16(50 * t["embed"][1])
    toks = tokens_of(model, 1200, seed=6) % 28 + 2
    plain, _ = ref.forward(model, toks)
    toks[3] = 1
    want, _ = ref.forward(model, toks)
    assert fm.error(plain, want)[1000:].max() > 1e-1          # the early token is visible at the end
    eng = engine(model)
    assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < 2e-4
    got = portions(eng, toks, [700, 2, 1, 1])
    assert fm.error(got, want).max() < 2e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ring_is_used_again(engine, monkeypatch, dtype):
    """Short rings (prompt batches of 16): hundreds of tokens through a ring of 64 rows, in batches, odd portions and decoding."""
    monkeypatch.setenv("KRONOS_CUDA_PROMPT_BATCH", "16")
    model = fm.make(96, 60, [fm.attention(4, 2, 32, 32, 21), fm.attention(2, 1, 24, 24, 48, ff=80), fm.delta(2, 24)], side=4, seed=8)
    toks = tokens_of(model, 420)
    want, _ = ref.forward(model, toks)
    eng = engine(model, dtype, max_seq=512)
    assert eng.kv_rows == 64
    assert fm.error(eng.forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]
    assert fm.error(portions(eng, toks, [7, 16, 1, 33]), want).max() < TOL[dtype]
    got = np.concatenate([eng.forward_token_ids(toks[:5], want_all=True)] + [eng.forward_token_ids([t], pos_start=5 + i)[None] for i, t in enumerate(toks[5:])])
    assert fm.error(got, want).max() < TOL[dtype]


def test_sequences_follow_one_another(engine):
    """A new sequence starts from nothing, whatever ran before; the same sequence gives the same bits again."""
    import kronos_2t_b200 as k2
    model = mixed("uneven")
    eng = engine(model, "bfloat16")
    a, b = tokens_of(model, 140, 1), tokens_of(model, 40, 2)
    first = eng.forward_token_ids(a, want_all=True)
    alone = eng.forward_token_ids(b, want_all=True)
    eng.decode_greedy(3, 40, 50)
    assert np.array_equal(eng.forward_token_ids(a, want_all=True), first)
    assert np.array_equal(eng.forward_token_ids(b, want_all=True), alone)
    assert eng.can_truncate_kv_to(40, 40) and not eng.can_truncate_kv_to(40, 12)
    with pytest.raises(k2.KronosCudaError, match="position 40"):
        eng.forward_token_ids([1, 2], pos_start=12)
    with pytest.raises(k2.KronosCudaError):
        eng.reconfigure_kv(8)
    assert np.array_equal(eng.forward_token_ids(b, want_all=True), alone)


def test_first_tokens(engine):
    model = mixed("uneven")
    for n in (1, 2, 3, 17):
        toks = tokens_of(model, n, seed=n)
        want, _ = ref.forward(model, toks)
        for dtype in ("float32", "bfloat16"):
            assert fm.error(engine(model, dtype).forward_token_ids(toks, want_all=True), want).max() < TOL[dtype]


def test_snapshot(engine):
    model = mixed("uneven")
    eng = engine(model, "bfloat16")
    toks = tokens_of(model, 120)
    eng.forward_token_ids(toks[:70])
    blob = eng.save_kv_prefix(70, 70)
    rest = eng.forward_token_ids(toks[70:], pos_start=70, want_all=True)
    eng.forward_token_ids(toks[::-1].copy())
    eng.restore_kv_prefix(blob)
    assert np.array_equal(eng.forward_token_ids(toks[70:], pos_start=70, want_all=True), rest)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation(engine, dtype):
    """generate() against the restatement: every chosen token has the reference's largest logit, up to rounding."""
    from kronos_2t_b200 import models
    model = mixed("uneven")
    eng = engine(model, dtype)
    prompt = tokens_of(model, 21)
    new = models.generate(eng, prompt, 150)
    seq = np.concatenate([prompt, new])
    want, _ = ref.forward(model, seq)
    for i, tok in enumerate(new):
        row = want[len(prompt) - 1 + i]
        assert row.max() - row[tok] < 6 * TOL[dtype] * row.std(), i
    # the captured step and the profile of one leave the sequence as it was
    table = eng.profile_step(int(new[-1]), len(seq) - 1, 2)
    assert "recurrence" in table and "attention" in table
    more = eng.forward_token_ids([int(new[-1])], pos_start=len(seq) - 1)
    assert fm.error(more[None], want[-1:]).max() < TOL[dtype]


def test_long_decoding(engine):
    model = mixed("narrow")
    eng = engine(model, "float32")
    new = eng.decode_greedy(5, 0, 700)
    seq = np.concatenate([[5], new[:-1]])
    want, _ = ref.forward(model, seq)
    got = eng.forward_token_ids(seq, want_all=True)
    assert fm.error(got, want).max() < 3e-4
    picked = np.take_along_axis(want, new[:, None].astype(int), 1)[:, 0]
    assert ((want.max(1) - picked) / want.std(1)).max() < 2e-3


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
