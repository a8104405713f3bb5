"""Layer-stack models without a GPU: the configuration reader refuses what it cannot run, before any device work, and the plain
restatement that the GPU tests compare with agrees with independent forms of its own mechanisms."""
from __future__ import annotations

import copy
import json

import numpy as np
import pytest

import puzevik_model as pm
import puzevik_oracle as po
import sipadra_model as sm
import sipadra_oracle as so


def _open_error(pkg, folder) -> str:
    lib = pkg.load_lib()
    pkg.model_api.bind_model_api(lib)
    lib.ckb200_clear_error()
    assert not lib.ckb200_model_open(str(folder).encode(), 1)
    msg = lib.ckb200_last_error_message().decode()
    lib.ckb200_clear_error()
    return msg


GOOD = pm.config([pm.layer("retention", pm.retention(), 48), pm.layer("latent_attention", pm.latent()), pm.layer("channel_delta", pm.delta(), 50)])


@pytest.mark.parametrize("change, expect", [
    (lambda c: c.update(architecture="Nothing"), "no design"),
    (lambda c: c.pop("width"), "'width'"),
    (lambda c: c.update(vocab=0), "'vocab'"),
    (lambda c: c["norm"].pop("eps"), "'eps'"),
    (lambda c: c["embedding"].pop("scale"), "'scale'"),
    (lambda c: c.update(layers=[]), "no layers"),
    (lambda c: c["layers"][0].update(type="windmill"), "windmill"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=64), "rotation"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rotates"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "key heads"),
    (lambda c: c["layers"][2]["mixer"].update(dim=300), "head size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="router"), "router"),
])
def test_config_is_refused_with_a_reason(pkg, tmp_path, change, expect):
    cfg = copy.deepcopy(GOOD)
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert expect in _open_error(pkg, tmp_path)


GOOD_SIPADRA = sm.config([sm.layer("wkv", sm.wkv(), 40), sm.layer("parallel", sm.parallel())])


@pytest.mark.parametrize("change, expect", [
    (lambda c: c.pop("logit_softcap"), "'logit_softcap'"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c["layers"][0].update(type="retention"), "retention"),
    (lambda c: c["layers"][0]["mixer"].update(dim=257), "head size"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "'left_scale'"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "key heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(dim=300), "head size"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("mask"), "'size'"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "'scale'"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26), "rotation"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "'slow'"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "scaling"),
])
def test_sipadra_config_is_refused_with_a_reason(pkg, tmp_path, change, expect):
    cfg = copy.deepcopy(GOOD_SIPADRA)
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert expect in _open_error(pkg, tmp_path)


def test_a_missing_decay_matrix_is_refused(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(GOOD_SIPADRA))
    w = sm.weights(GOOD_SIPADRA, 1)
    del w["l0.mix.w1"]
    pm.write_safetensors(tmp_path / "model.safetensors", w)
    assert "l0.mix.w1" in _open_error(pkg, tmp_path)


def test_missing_and_broken_weight_files_are_refused(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(GOOD))
    assert "cannot open" in _open_error(pkg, tmp_path)
    (tmp_path / "model.safetensors").write_bytes(b"\xff" * 64)
    assert "safetensors" in _open_error(pkg, tmp_path)
    w = pm.weights(GOOD, 1)
    del w["l2.mix.a1"]
    pm.write_safetensors(tmp_path / "model.safetensors", w)
    assert "l2.mix.a1" in _open_error(pkg, tmp_path)


def test_retention_recurrence_equals_its_attention_form():
    mix, eps, T = pm.retention(), 1e-5, 19
    cfg = pm.config([pm.layer("retention", mix)])
    w = po.sub({k: v.astype(np.float64) for k, v in pm.weights(cfg, 3).items()}, "l0.mix.")
    h = np.random.default_rng(0).normal(size=(T, cfg["width"]))
    H, d, dv, rot = mix["heads"], mix["dim"], mix["vdim"], mix["rot"]
    pos = np.arange(T)
    q = po.rotate((h @ w["q"].T).reshape(T, H, d), pos, rot["dims"], rot["base"])
    k = po.rotate((h @ w["k"].T).reshape(T, H, d), pos, rot["dims"], rot["base"]) / np.sqrt(d)
    v = (h @ w["v"].T).reshape(T, H, dv)
    o = np.empty((T, H, dv))
    for n in range(H):
        lag = pos[:, None] - pos[None, :]
        o[:, n] = (np.where(lag >= 0, float(mix["decay"][n]) ** np.maximum(lag, 0), 0) * (q[:, n] @ k[:, n].T)) @ v[:, n]
    want = (po.rms(o, eps).reshape(T, -1) * po.silu(h @ w["g"].T)) @ w["o"].T
    assert np.allclose(po.retention(h, w, mix, eps), want, atol=1e-10)


def test_delta_rule_without_decay_overwrites_a_repeated_key():
    """beta = 1 and no decay: after writing v1 then v2 under one key, reading that key gives v2."""
    S = np.zeros((4, 3))
    k = po.unit(np.array([[0.3, -1.0, 2.0, 0.5]]))[0]
    for v in (np.array([1.0, 2.0, 3.0]), np.array([-4.0, 0.5, 9.0])):
        S = S + np.outer(k, v - S.T @ k)
    assert np.allclose(S.T @ k, [-4.0, 0.5, 9.0], atol=1e-4)


def test_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.normal(size=(1, 1, 20)), rng.normal(size=(1, 1, 20))
    dot = [float(np.sum(po.rotate(q, np.array([p + 5]), 12, 1e3) * po.rotate(k, np.array([p]), 12, 1e3))) for p in (0, 17, 900)]
    assert np.allclose(dot, dot[0], atol=1e-9)
    assert np.array_equal(po.rotate(q, np.array([9]), 12, 1e3)[..., 12:], q[..., 12:])


def test_causal_conv_reads_zeros_before_the_start():
    x, w = np.arange(1.0, 6.0)[:, None], np.array([[100.0, 10.0, 1.0]])
    assert po.causal_conv(x, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]


# ---- Sipadra's own mechanisms

def _sipadra(layer, T, seed=3):
    cfg = sm.config([layer])
    w = so.sub({k: v.astype(np.float64) for k, v in sm.weights(cfg, seed).items()}, "l0.mix.")
    return w, np.random.default_rng(seed).normal(size=(T, cfg["width"]))


def test_windowed_attention_equals_its_masked_form():
    mix, eps, T = sm.left(size=7), 1e-4, 30
    w, h = _sipadra(sm.layer("parallel", sm.parallel(mix)), T)
    w = so.sub(w, "left.")
    H, G, d, dv, rot = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"], mix["rot"]
    q = so.rms(so.rotate((h @ w["q"].T).reshape(T, H, d), rot["dims"], rot["base"], rot["scaling"]), eps)
    k = so.rms(so.rotate((h @ w["k"].T).reshape(T, G, d), rot["dims"], rot["base"], rot["scaling"]), eps).repeat(H // G, axis=1)
    v = (h @ w["v"].T).reshape(T, G, dv).repeat(H // G, axis=1)
    lag = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where((lag >= 0) & (lag < 7), np.einsum("thd,shd->hts", q, k) * mix["scale"], -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    o = np.einsum("hts,shd->thd", p / p.sum(-1, keepdims=True), v)
    assert np.allclose(so.windowed_attention(h, w, mix, eps), o.reshape(T, -1) @ w["o"].T, atol=1e-10)


def test_lightning_recurrence_equals_its_attention_form():
    mix, eps, T = sm.right(), 1e-4, 25
    w, h = _sipadra(sm.layer("parallel", sm.parallel(right_arm=mix)), T)
    w = so.sub(w, "right.")
    q, k, v = (so.silu(h @ w[n].T).reshape(T, mix["heads"], -1) for n in "qkv")
    lag = np.arange(T)[:, None] - np.arange(T)[None, :]
    a = np.where(lag >= 0, np.power(np.array(mix["decay"])[:, None, None], np.maximum(lag, 0)), 0.0)
    o = np.einsum("hts,shd->thd", a * np.einsum("thd,shd->hts", q, k), v).reshape(T, -1)
    want = (so.rms(o, eps) * w["norm"] * so.sigmoid(h @ w["g"].T)) @ w["o"].T
    assert np.allclose(so.lightning_attention(h, w, mix, eps), want, atol=1e-10)


def test_wkv_recurrence_equals_its_sum_over_the_past():
    mix, eps, T = sm.wkv(heads=2, dim=6), 1e-4, 14
    w, h = _sipadra(sm.layer("wkv", mix), T)
    r, k, v = ((so.token_shift(h, w["mu." + n]) @ w[n].T).reshape(T, 2, 6) for n in "rkv")
    log = -np.exp(np.tanh(so.token_shift(h, w["mu.w"]) @ w["w1"].T) @ w["w2"].T + w["w0"]).reshape(T, 2, 6)
    o = np.zeros((T, 2, 6))
    for t in range(T):
        for s in range(t + 1):
            weight = w["u"] if s == t else np.exp(log[s + 1:t].sum(0))
            o[t] += (r[t] * weight * k[s]).sum(-1, keepdims=True) * v[s]
    gate = so.silu(so.token_shift(h, w["mu.g"]) @ w["g"].T)
    assert np.allclose(so.wkv(h, w, mix, eps), (so.rms(o, eps).reshape(T, -1) * w["norm"] * gate) @ w["o"].T, atol=1e-10)


def test_scaled_rotation_between_its_limits():
    plain, one = so.yarn_frequencies(16, 500.0)
    assert one == 1.0
    f, mul = so.yarn_frequencies(16, 500.0, sm.yarn(factor=4.0, original=64, fast=8.0, slow=1.0))
    assert mul == 0.1 * np.log(4.0) + 1.0 and f[0] == plain[0] and np.isclose(f[-1], plain[-1] / 4)
    assert np.all(f <= plain) and np.all(f >= plain / 4 * (1 - 1e-12)) and np.any((f < plain * 0.99) & (f > plain / 4 * 1.01))


def test_the_first_token_mixes_with_zeros():
    h, mu = np.array([[2.0, 4.0], [6.0, 8.0]]), np.array([0.25, 1.0])
    assert so.token_shift(h, mu).tolist() == [[1.5, 0.0], [5.0, 4.0]]
