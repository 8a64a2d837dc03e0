"""Host side of the Zasesun design, no GPU: reader, rotation tables, and the plain restatement the device tests compare with (checked
against second, differently organised evaluations)."""
import json

import numpy as np
import pytest

import folizen_models as fm
import zasesun_models as zm
import zasesun_ref as ref
from kronos_2t_b200 import ffi, models

LAYERS = [zm.latent(3, 20, 6, 14, 22, 26, zm.dense(30), scale=0.3), zm.latent(2, 12, 8, 10, 9, 18, zm.moe(5, 2, 12, shared=17), scaling=zm.YARN),
          zm.latent(1, 8, 4, 8, 8, 8), zm.latent(2, 12, 8, 10, 9, 18, zm.moe(3, 3, 7), scaling=zm.YARN)]


def widen(a):
    return (a.astype(np.uint32) << 16).view(np.float32) if a.dtype == np.uint16 else a


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_reader_fills_the_spec(tmp_path, dtype):
    model = zm.make(44, 57, LAYERS, eps=2e-5, mult=0.7, cap=11.0)
    t = model["tensors"]
    spec = models.load_spec(fm.write(model, str(tmp_path)), dtype, 60)
    assert spec["cfg"] == dict(hidden=44, vocab=57, max_seq=60, eps=2e-5, residual_mult=0.7, logit_softcap=11.0, precision=16 if dtype == "bfloat16" else 32)
    a, b, c, d = spec["blocks"]
    assert [x["mixer"] for x in spec["blocks"]] == [ffi.MIXER_LATENT_ATTENTION] * 4
    assert (a["heads"], a["dim"], a["rot_dim"], a["vdim"], a["q_rank"], a["kv_rank"], a["score_scale"]) == (3, 20, 6, 14, 22, 26, 0.3)
    assert np.array_equal(widen(a["in_proj"]), np.concatenate([t["l0.mix.dq"], t["l0.mix.dkv"]]))
    assert np.array_equal(widen(a["kv_up"]), np.concatenate([t["l0.mix.uk"], t["l0.mix.uv"]])) and np.array_equal(widen(a["q_up"]), t["l0.mix.uq"])
    assert np.array_equal(a["pre_norm1"], t["l0.norm1"]) and np.array_equal(a["norm1"], t["l0.norm1b"])
    assert np.array_equal(a["pre_norm2"], t["l0.norm2"]) and np.array_equal(a["norm2"], t["l0.norm2b"])
    assert a["act"] == ffi.ACT_GELU_GATED and a["ff"] == 30
    assert np.array_equal(widen(a["up_proj"])[0::2], t["l0.mlp.gate"]) and np.array_equal(widen(a["up_proj"])[1::2], t["l0.mlp.up"])
    assert (b["act"], b["experts"], b["experts_top"], b["ff"], b["shared_ff"]) == (ffi.ACT_RELU_SQUARED, 5, 2, 12, 17)
    assert np.array_equal(widen(b["router"]), np.concatenate([t["l1.mlp.router"], t["l1.mlp.shared.up"]]))
    assert np.array_equal(widen(b["up_proj"])[12:24], t["l1.mlp.e1.up"]) and np.array_equal(widen(b["down_proj"])[44:88], t["l1.mlp.e1.down"])
    assert "ff" not in c and "norm2" not in c
    assert "shared_ff" not in d and d["experts_top"] == 3 and d["rot_cos_sin"] is b["rot_cos_sin"] and a["rot_cos_sin"] is not b["rot_cos_sin"]
    assert np.array_equal(widen(spec["head"]), t["embed"])


def test_reader_refuses_what_it_does_not_know(tmp_path):
    model = zm.make(16, 20, [zm.latent(1, 8, 4, 8, 8, 8, zm.dense(8))])
    model["config"]["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="sparse"):
        models.load_spec(fm.write(model, str(tmp_path)))
    model["config"]["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="other"):
        models.load_spec(fm.write(model, str(tmp_path)))


ROTATIONS = [dict(base=1e4, dims=16), dict(base=500.0, dims=6, scaling=zm.YARN), dict(base=5e5, dims=64, scaling=dict(factor=40.0, original=4096, fast=32, slow=1)),
             dict(base=100.0, dims=10, scaling=dict(factor=2.0, original=50, fast=2.0, slow=2.0)), dict(base=1e4, dims=32, scaling=dict(factor=1.0, original=256, fast=8, slow=1)),
             dict(base=20.0, dims=8, scaling=dict(factor=4.0, original=100000, fast=4, slow=0.001))]


@pytest.mark.parametrize("rot", ROTATIONS, ids=str)
def test_rotation_table(rot):
    """The engine's table turns a vector as the restatement does; dimensions behind rot dims stay."""
    width = rot["dims"] + 4
    table = models.rotation_table(50, width, rot["dims"], rot["base"], rot.get("scaling")).astype(np.float64)
    x = np.random.default_rng(0).standard_normal((50, width))
    y = np.empty_like(x)
    y[:, 0::2] = x[:, 0::2] * table[:, 0::2] - x[:, 1::2] * table[:, 1::2]
    y[:, 1::2] = x[:, 1::2] * table[:, 0::2] + x[:, 0::2] * table[:, 1::2]
    assert np.allclose(y, ref.rotate(x, np.arange(50), rot), atol=1e-6)
    assert np.array_equal(y[:, rot["dims"]:], x[:, rot["dims"]:])


def test_ramp_of_the_frequencies():
    """Fast pairs keep their frequency, slow ones are divided, and the ramp lies in between."""
    f, gain = models.yarn_frequencies(64, 1e4, dict(factor=8.0, original=2048, fast=32.0, slow=1.0))
    plain = 1e4 ** (-np.arange(32) / 32.0)
    turns = 2048 * plain / (2 * np.pi)
    ratio = plain / f
    assert np.allclose(ratio[turns > 40], 1) and np.allclose(ratio[turns < 0.9], 8) and np.all(np.diff(ratio) > -1e-12)
    assert np.any((ratio > 1.1) & (ratio < 7.9)) and abs(gain - (0.1 * np.log(8) + 1)) < 1e-12


# ---- the restatement itself
def test_attention_of_the_restatement_in_latent_space():
    """Scores as (W_uk^T q) . c and values as W_uv (sum of p c): the form that needs no keys and values per head."""
    rng = np.random.default_rng(1)
    m = zm.latent(3, 10, 6, 8, 12, 14, scaling=zm.YARN)["mixer"]
    T, W = 25, 20
    p = {"dq": rng.standard_normal((12, W)), "dq.norm": rng.uniform(0.5, 2, 12), "uq": rng.standard_normal((48, 12)), "dkv": rng.standard_normal((20, W)),
         "dkv.norm": rng.uniform(0.5, 2, 14), "uk": rng.standard_normal((30, 14)), "uv": rng.standard_normal((24, 14)), "o": rng.standard_normal((W, 24))}
    h = rng.standard_normal((T, W))
    got = ref.latent_attention(h, p, m, 1e-6)
    c = ref.rms_norm((h @ p["dkv"].T)[:, :14], p["dkv.norm"], 1e-6)
    f, gain = ref.rotation(m["rot"])

    def turn(v, t):
        z = (v[0::2] + 1j * v[1::2]) * np.exp(1j * t * f) * gain
        return np.stack([z.real, z.imag], 1).reshape(-1)

    for i in range(T):
        q = (p["uq"] @ ref.rms_norm(p["dq"] @ h[i], p["dq.norm"], 1e-6)).reshape(3, 16)
        out = []
        for n in range(3):
            lat = p["uk"][n * 10:n * 10 + 10].T @ q[n, :10]
            s = np.array([(lat @ c[j] + turn(q[n, 10:], i) @ turn((p["dkv"] @ h[j])[14:], j)) * m["scale"] for j in range(i + 1)])
            w = np.exp(s - s.max())
            out.append(p["uv"][n * 8:n * 8 + 8] @ (w / w.sum() @ c[:i + 1]))
        assert np.allclose(got[i], p["o"] @ np.concatenate(out))


def test_router_of_the_restatement():
    z = np.array([[0.0, 2.0, -1.0, 1.0], [3.0, 3.5, 0.0, 0.1]])
    chosen, w = ref.route(z, 2)
    s = np.exp(z) / np.exp(z).sum(1, keepdims=True)
    assert chosen.tolist() == [[1, 3], [1, 0]] and np.allclose(w, [[s[0, 1], s[0, 3]], [s[1, 1], s[1, 0]]]) and np.all(w.sum(1) < 1)


def test_margin_of_the_restatement():
    z = np.array([[0.0, 2.0, -1.0, 1.0], [3.0, 3.5, 0.0, 0.1]])
    assert np.allclose(ref.margin(z, 2), [1.0, 2.9]) and np.all(np.isinf(ref.margin(z, 4)))


def test_restatement_is_causal_and_cut_free():
    model = zm.make(44, 57, LAYERS)
    toks = np.random.default_rng(3).integers(0, 57, 40)
    whole, streams = ref.forward(model, toks)
    part, _ = ref.forward(model, toks[:25])
    assert np.allclose(whole[:25], part) and streams.shape == (4, 40, 44) and np.abs(whole).max() < 20.0


def test_pointer_model_points():
    model = zm.pointer()
    toks = np.random.default_rng(0).integers(3, 40, 300)
    toks[[7, -1]] = 1, 2
    want, _ = ref.forward(model, toks)
    toks[7] = 5
    assert fm.error(ref.forward(model, toks)[0], want)[-1] > 0.5


def test_architecture_is_registered(tmp_path):
    with open(tmp_path / "config.json", "w") as f:
        json.dump(dict(architecture="Zasesun"), f)
    assert models.architecture(models.read_config(str(tmp_path))) == "Zasesun"
