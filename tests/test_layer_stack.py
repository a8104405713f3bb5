"""Layer-stack models without a GPU: the configuration reader refuses what it cannot run, before any device work, and the plain
restatement that the GPU tests compare with agrees with independent forms of its own mechanisms."""
from __future__ import annotations

import copy
import json

import numpy as np
import pytest

import puzevik_model as pm
import puzevik_oracle as po


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
