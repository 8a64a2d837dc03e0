"""Host side of the block engine, no GPU: dense matrix images, the model registry and the Folizen reader, and the plain
restatement the device tests compare with (checked here against a second, differently organised evaluation)."""
import json

import numpy as np
import pytest

import folizen_models as fm
import folizen_ref as ref
from kronos_2t_b200 import ffi, models


@pytest.mark.parametrize("rows,cols", [(1, 1), (7, 64), (130, 200), (256, 129)])
def test_dense_bf16_image(rows, cols):
    """Panels of 64 columns, rows padded to 128, 16-byte chunk c of row r at position c ^ (r % 8), zeros behind the last column."""
    w = np.random.default_rng(rows).integers(1, 65536, (rows, cols)).astype(np.uint16)
    img = ffi.matrix_image(ffi.dense_desc(w, 16)).view(np.uint16)
    pad, panels = -(-rows // 128) * 128, -(-cols // 64)
    img = img.reshape(panels, pad, 8, 8)
    want = np.zeros((panels, pad, 8, 8), np.uint16)
    full = np.zeros((rows, panels * 64), np.uint16)
    full[:, :cols] = w
    for r in range(rows):
        for p in range(panels):
            for c in range(8):
                want[p, r, c ^ (r % 8)] = full[r, p * 64 + c * 8:p * 64 + c * 8 + 8]
    assert np.array_equal(img, want)


def test_dense_fp32_image():
    w = np.random.default_rng(1).standard_normal((5, 7)).astype(np.float32)
    img = ffi.matrix_image(ffi.dense_desc(w, 32)).view(np.float32).reshape(5, 8)
    assert np.array_equal(img[:, :7], w) and not img[:, 7].any()


def test_bf16_rounding():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.14159, 0.0], np.float32)
    assert np.array_equal((ffi.bf16_bits(x).astype(np.uint32) << 16).view(np.float32), fm.bf16(x))


LAYERS = [fm.attention(6, 2, 24, 40, 11, scale=0.3, ff=72), fm.delta(3, 20, rank=5), fm.attention(2, 2, 16, 16, 4), fm.delta(1, 28, ff=33)]


def test_reader_fills_the_spec(tmp_path):
    model = fm.make(52, 61, LAYERS, side=6, eps=3e-5)
    folder = fm.write(model, str(tmp_path))
    t = model["tensors"]
    for dtype, precision in (("bfloat16", 16), ("float32", 32)):
        spec = models.load_spec(folder, dtype, 100)
        assert spec["cfg"] == dict(hidden=52, vocab=61, max_seq=100, eps=3e-5, side_dim=6, precision=precision)
        widen = (lambda a: (a.astype(np.uint32) << 16).view(np.float32)) if precision == 16 else (lambda a: a)
        a, d, _, last = spec["blocks"]
        assert (a["mixer"], a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["window"], a["ff"]) == (ffi.MIXER_WINDOW_ATTENTION, 6, 2, 24, 40, 11, 72)
        assert np.array_equal(widen(a["in_proj"]), np.concatenate([t["l0.mix.q"], t["l0.mix.k"], t["l0.mix.v"]]))
        assert np.allclose(a["head_scale"], 0.3 * t["l0.mix.temp"]) and np.allclose(a["head_slope"], ref.bias_slopes(6))
        assert (d["mixer"], d["heads"], d["dim"], d["decay_rank"], d.get("ff", 0)) == (ffi.MIXER_GENERAL_DELTA, 3, 20, 5, 0)
        assert np.array_equal(widen(d["in_proj"]), np.concatenate([t["l1.mix." + n] for n in ("r", "k", "v", "g", "a", "w1")]))
        assert last["ff"] == 33 and np.array_equal(last["act_coef"], t["l3.mlp.act"])
        assert np.array_equal(widen(spec["head"]), t["head"])


def test_registry_refuses_what_it_does_not_know(tmp_path):
    model = fm.make(16, 20, [fm.attention(1, 1, 8, 8, 4)], side=2)
    model["config"]["architecture"] = "Nothing"
    with pytest.raises(ValueError, match="Nothing"):
        models.load_spec(fm.write(model, str(tmp_path)))
    assert models.architecture(dict(architectures=["X", "Qwen2ForCausalLM"])) == "Qwen2ForCausalLM"
    model["config"].update(architecture="Folizen")
    model["config"]["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="other"):
        models.load_spec(fm.write(model, str(tmp_path)))


def test_compiled_models_go_through_the_registry(tmp_path):
    from kronos_2t_b200 import synth
    cfg = dict(hidden=128, layers=1, n_q=2, n_kv=1, head_dim=64, inter=128, vocab=64, max_seq=32, eps=1e-5, theta=1e4)
    ffi.k2tb_save(str(tmp_path / "m.k2tb"), synth.random_model(cfg, "b4", seed=2, untied=True), [0] * 6)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(dict(architectures=["LlamaForCausalLM"], hidden_size=128, num_attention_heads=2, num_key_value_heads=1, intermediate_size=128, vocab_size=64,
                       rms_norm_eps=1e-5, rope_theta=1e4), f)
    spec = models.load_spec(str(tmp_path), max_seq=32)
    assert spec["cfg"]["layers"] == 1 and spec["cfg"]["head_dim"] == 64 and spec["layers"][0]["qkv"].rows == 256


# ---- the restatement itself
def test_attention_of_the_restatement_matches_a_matrix_form():
    rng = np.random.default_rng(0)
    T, H, G, d, dv, window, scale = 30, 4, 2, 8, 6, 7, 0.4
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, G, d)), rng.standard_normal((T, G, dv))
    temp = rng.uniform(0.5, 2, H)
    got = ref.window_attention(q, k, v, scale, temp, window)
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    for h in range(H):
        s = q[:, h] @ k[:, h // 2].T * scale * temp[h] - 2.0 ** (-8 * (h + 1) / H) * (i - j)
        s = np.where((j <= i) & (i - j <= window - 1), s, -np.inf)
        p = np.exp(s) / np.exp(s).sum(1, keepdims=True)
        assert np.allclose(got[:, h], p @ v[:, h // 2])


def test_delta_of_the_restatement_matches_transition_matrices():
    rng = np.random.default_rng(1)
    T, d = 12, 5
    r, k, v = (rng.standard_normal((T, d)) for _ in range(3))
    w, a, u = ref.delta_coefficients(rng.standard_normal((T, d)), rng.standard_normal((T, d)), k)
    o, S = ref.general_delta(r, w, a, u, k, v)
    want = np.zeros((d, d))
    for t in range(T):
        want = (np.diag(w[t]) - np.outer(a[t] * u[t], u[t])) @ want + np.outer(k[t], v[t])
        assert np.allclose(o[t], want.T @ r[t])
    assert np.allclose(S, want)
    half, mid = ref.general_delta(r[:5], w[:5], a[:5], u[:5], k[:5], v[:5])
    rest, _ = ref.general_delta(r[5:], w[5:], a[5:], u[5:], k[5:], v[5:], mid)
    assert np.allclose(np.concatenate([half, rest]), o)


def test_restatement_is_causal_and_cut_free():
    model = fm.make(52, 61, LAYERS, side=6)
    toks = np.random.default_rng(3).integers(0, 61, 40)
    whole, streams = ref.forward(model, toks)
    part, _ = ref.forward(model, toks[:25])
    assert np.allclose(whole[:25], part) and streams.shape == (4, 40, 52)
