"""What the GPU tests of the layer-stack designs share: a model on disk with its oracle, and running a sequence through a session cut into
portions."""
from __future__ import annotations

import numpy as np

import puzevik_model
import puzevik_oracle
import sipadra_model
import sipadra_oracle

DESIGNS = {"Puzevik": (puzevik_model, puzevik_oracle), "Sipadra": (sipadra_model, sipadra_oracle)}

# worst position relative to the spread of the logits; bfloat16: products with rounded inputs over a few layers, sharp softmaxes among them
TOL = {True: 2e-5, False: 6e-2}


def error(got, want):
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(axis=-1)).max() / want.std())


class Case:
    """A model on disk, its oracle logits for one token sequence, and sessions on it."""

    def __init__(self, pkg, lib, tmp_path, cfg, tokens=70, seed=5, **kw):
        model, self.reference = DESIGNS[cfg["architecture"]]
        self.pkg, self.lib, self.cfg = pkg, lib, cfg
        self.w = model.weights(cfg, seed, **kw)
        self.dir = puzevik_model.write(tmp_path / "model", cfg, self.w)
        self.w64 = {k: v.astype(np.float64) for k, v in self.w.items()}
        self.ids = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], tokens)
        self.want = self.oracle(self.ids)

    def oracle(self, ids, layers_out=None, cfg=None):
        return self.reference.forward(cfg or self.cfg, self.w64, ids, layers_out)

    def session(self, float32, max_tokens=256):
        return self.pkg.model_api.Session(self.lib, self.dir, max_tokens, float32)


def run(session, ids, cuts):
    """Logits of every position, the sequence cut into portions of the sizes `cuts` (the last one repeats)."""
    out, t, i = [], 0, 0
    while t < len(ids):
        n = min(cuts[min(i, len(cuts) - 1)], len(ids) - t)
        out.append(session.extend(ids[t:t + n], range(n)))
        t, i = t + n, i + 1
    return np.concatenate(out)


SCHEDULES = {"whole": [10 ** 6], "decode": [1], "twos": [2], "mixed": [9, 2, 1, 16, 3, 1, 1, 7, 20, 2], "prompt then decode": [41, 1], "tens": [10]}


def check_all(case, float32, schedules=SCHEDULES, max_tokens=256):
    s = case.session(float32, max_tokens)
    try:
        for name, cuts in schedules.items():
            err = error(run(s, case.ids, cuts), case.want)
            assert err < TOL[float32], (name, err)
            s.reset()
    finally:
        s.close()


def batch_logits(pkg, lib, case, ids, portions, float32, max_tokens):
    """Logits [T, batch, vocab] of sequences side by side (ids [T, batch]), in the given portions."""
    T, batch = ids.shape
    V, api = case.cfg["vocab"], pkg.model_api
    api.bind_model_api(lib)
    lib.ckb200_tune_set(b"model_f32", int(float32))
    lib.ckb200_tune_set(b"model_max_seq", max_tokens)
    m = lib.ckb200_model_open(case.dir.encode(), batch)
    try:
        assert m, lib.ckb200_last_error_message()
        got = np.zeros((T, batch, V), np.float32)
        t = 0
        for n in portions:
            part, places = np.ascontiguousarray(ids[t:t + n], dtype=np.int32), np.arange(n, dtype=np.int32)
            out = np.zeros((n, batch, V), np.float32)
            assert lib.ckb200_model_extend(m, api.vptr(part), n, api.vptr(places), n, api.vptr(out)) == 0, lib.ckb200_last_error_message()
            got[t:t + n] = out
            t += n
        assert t == T
        return got
    finally:
        lib.ckb200_model_free(m)
        lib.ckb200_tune_set(b"model_f32", 0)


def greedy(case, prompt, steps):
    """The oracle's greedy continuation, and the smallest margin between the first and second choice."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = case.oracle(ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, float(top[1] - top[0]) / case.want.std())
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin


def greedy_through_the_model_abi(pkg, lib, case, steps, max_tokens=64):
    """ck_model_init on the folder, ck_model_embed_tokens for the prompt, ck_model_decode per token - how a chat front end drives a model.
    Two continuations, the second after the context has been given back."""
    import ctypes as C

    lib.ckb200_tune_set(b"model_f32", 1)
    lib.ckb200_tune_set(b"model_max_seq", max_tokens)
    v7 = C.CDLL(pkg.find_lib("libckb200_model_v7.so"))
    runs = []
    try:
        assert v7.ck_model_init(case.dir.encode()) == 0
        V = v7.ck_model_get_vocab_size()
        assert V == case.cfg["vocab"] and v7.ck_model_get_context_window() == max_tokens
        for _ in range(2):
            ids = np.ascontiguousarray(case.ids, dtype=np.int32)
            logits = np.zeros(V, np.float32)
            assert v7.ck_model_embed_tokens(ids.ctypes.data_as(C.c_void_p), len(ids)) == 0
            assert v7.ck_model_forward(logits.ctypes.data_as(C.c_void_p)) == 0
            got = []
            for _ in range(steps):
                got.append(int(logits.argmax()))
                assert v7.ck_model_decode(C.c_int32(got[-1]), logits.ctypes.data_as(C.c_void_p)) == 0
            runs.append(got)
            v7.ck_model_kv_cache_reset()
    finally:
        v7.ck_model_free()
        lib.ckb200_tune_set(b"model_f32", 0)
    return runs


def trace(root, case, steps, dtype, out, max_tokens=64):
    """bin/trace_run over (step, expected logits or None) pairs; compares what it writes."""
    import json
    import os
    import subprocess

    out.mkdir()
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", case.dir, "--dtype", dtype, "--out", str(out), "--max-tokens", str(max_tokens)],
                       input="".join(json.dumps(s) + "\n" for s, _ in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {s['step']}" for s, _ in steps]
    for s, want in steps:
        path = out / f"{s['step']}.f32"
        assert path.exists() == (want is not None)
        if want is not None:
            assert error(np.fromfile(path, "<f4").reshape(want.shape), want) < TOL[dtype == "float32"]
