"""Layer-stack models on the GPU against the plain numpy restatement: every mixer alone and together, whole prompts, portions, decoding,
batches, state that is given back and used again, sizes that fit no tile."""
from __future__ import annotations

import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

import puzevik_model as pm
import puzevik_oracle as po

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

# worst position relative to the spread of the logits; bfloat16: products with rounded inputs over a few layers, sharp softmaxes among them
TOL = {True: 2e-5, False: 6e-2}


def error(got, want):
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(axis=-1)).max() / want.std())


class Case:
    """A model on disk, its oracle logits for one token sequence, and sessions on it."""

    def __init__(self, pkg, lib, tmp_path, cfg, tokens=70, seed=5, **kw):
        self.pkg, self.lib, self.cfg = pkg, lib, cfg
        self.w = pm.weights(cfg, seed, **kw)
        self.dir = pm.write(tmp_path / "model", cfg, self.w)
        self.w64 = {k: v.astype(np.float64) for k, v in self.w.items()}
        self.ids = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], tokens)
        self.want = self.oracle(self.ids)

    def oracle(self, ids):
        return po.forward(self.cfg, self.w64, ids)

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


def check_all(case, float32, schedules=SCHEDULES):
    s = case.session(float32)
    try:
        for name, cuts in schedules.items():
            err = error(run(s, case.ids, cuts), case.want)
            assert err < TOL[float32], (name, err)
            s.reset()
    finally:
        s.close()


SINGLE = {
    "retention": pm.layer("retention", pm.retention()),
    "retention, all dimensions rotated, one head": pm.layer("retention", pm.retention(heads=1, dim=32, vdim=64, dims=32, base=1e2, decay=[0.9997])),
    "retention, wide": pm.layer("retention", pm.retention(heads=2, dim=200, vdim=140, dims=6, decay=[1.0, 0.25])),
    "latent": pm.layer("latent_attention", pm.latent()),
    "latent, odd sizes": pm.layer("latent_attention", pm.latent(heads=5, dim=10, rot_dim=6, vdim=13, q_rank=21, kv_rank=35, scale=0.9)),
    "latent, many heads": pm.layer("latent_attention", pm.latent(heads=18, dim=16, rot_dim=8, vdim=16, q_rank=40, kv_rank=136, scale=0.5)),
    "delta": pm.layer("channel_delta", pm.delta()),
    "delta, equal heads, four taps": pm.layer("channel_delta", pm.delta(heads=3, kv_heads=3, dim=64, vdim=64, conv=4)),
    "delta, one tap, one key head, wide values": pm.layer("channel_delta", pm.delta(heads=2, kv_heads=1, dim=17, vdim=70, conv=1)),
    "delta, wide keys": pm.layer("channel_delta", pm.delta(heads=2, kv_heads=2, dim=130, vdim=9, conv=5)),
}


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_one_mixer(pkg, ck, tmp_path, name, float32):
    check_all(Case(pkg, ck, tmp_path, pm.config([SINGLE[name]])), float32)


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
@pytest.mark.parametrize("ff", [16, 50, 200])
def test_feed_forward_beside_a_mixer(pkg, ck, tmp_path, ff, float32):
    check_all(Case(pkg, ck, tmp_path, pm.config([pm.layer("retention", pm.retention(), ff)], width=72)), float32, {"whole": [10 ** 6], "decode": [1], "fives": [5]})


def stack_config(**kw):
    return pm.config([pm.layer("latent_attention", pm.latent(), 120), pm.layer("channel_delta", pm.delta()), pm.layer("retention", pm.retention(), 72),
                      pm.layer("channel_delta", pm.delta(heads=3, kv_heads=1, dim=24, vdim=32, conv=2), 96), pm.layer("latent_attention", pm.latent(heads=2, dim=8, rot_dim=24, vdim=16))], **kw)


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
def test_stack_in_all_schedules(pkg, ck, tmp_path, float32):
    check_all(Case(pkg, ck, tmp_path, stack_config()), float32)


def test_large_eps_and_small_embeddings(pkg, ck, tmp_path):
    """eps of the size of the mean square: it must stand inside the root, in every norm."""
    check_all(Case(pkg, ck, tmp_path, stack_config(eps=0.3, scale=0.6)), True, {"whole": [10 ** 6], "decode": [1]})


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
def test_many_tiles(pkg, ck, tmp_path, float32):
    """More rows, columns and keys than one tile of any kernel has."""
    cfg = pm.config([pm.layer("latent_attention", pm.latent(heads=2, kv_rank=192, q_rank=130), 300), pm.layer("channel_delta", pm.delta(heads=2, kv_heads=2, dim=32, vdim=48), 90)],
                    width=328, vocab=413)
    case = Case(pkg, ck, tmp_path, cfg, tokens=290)
    s = case.session(float32, 300)
    for cuts in ([10 ** 6], [129, 1, 31, 64], [257, 2]):
        assert error(run(s, case.ids, cuts), case.want) < TOL[float32], cuts
        s.reset()
    s.close()


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
def test_a_far_key_decides(pkg, ck, tmp_path, float32):
    """Scores so sharp that most queries take their value from one key alone, some of them from one of the first positions."""
    case = Case(pkg, ck, tmp_path, pm.config([pm.layer("latent_attention", pm.latent(scale=2.5))]), tokens=200)
    shows = 0.0
    for place in range(12):
        other = case.ids.copy()
        other[place] = (other[place] + 1) % case.cfg["vocab"]
        shows = max(shows, float(np.abs(case.oracle(other)[150:] - case.want[150:]).max()) / case.want.std())
    assert shows > 0.5, "no far key decides: choose another seed"
    check_all(case, float32, {"whole": [10 ** 6], "decode": [1], "at 64s": [64], "prompt then decode": [130, 1]})


def test_state_remembers_far_back(pkg, ck, tmp_path):
    """Slow decays: the first tokens still show after 200 steps, in both recurrent mixers, however the steps are cut."""
    cfg = pm.config([pm.layer("retention", pm.retention(decay=[0.9995, 0.999, 1.0])), pm.layer("channel_delta", pm.delta(conv=2))])
    case = Case(pkg, ck, tmp_path, cfg, tokens=230, a_log=(-9.0, -7.0))
    other = case.ids.copy()
    other[:4] = (other[:4] + 1) % cfg["vocab"]
    assert np.abs(case.oracle(other)[-1] - case.want[-1]).max() / case.want.std() > 50 * TOL[True]
    check_all(case, True, {"whole": [10 ** 6], "decode": [1], "mixed": [17, 1, 40, 2, 8]})


def test_strong_decay_forgets(pkg, ck, tmp_path):
    """Decays that underflow to zero within a token: no overflow, no stale state."""
    check_all(Case(pkg, ck, tmp_path, pm.config([pm.layer("channel_delta", pm.delta())]), a_log=(3.0, 6.0)), True, {"whole": [10 ** 6], "decode": [1], "threes": [3]})


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
def test_first_tokens(pkg, ck, tmp_path, float32):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=9)
    s = case.session(float32)
    for n in (1, 2, 3, 9):
        assert error(run(s, case.ids[:n], [n]), case.want[:n]) < TOL[float32], n
        s.reset()
    s.close()


def test_a_session_used_again_starts_fresh(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config())
    s = case.session(True)
    first = run(s, case.ids, [30, 1])
    s.reset()
    run(s, case.ids[::-1][:50], [50])                        # another sequence leaves its state and cache rows behind
    s.reset()
    again = run(s, case.ids, [30, 1])
    assert np.array_equal(first, again)
    assert s.lib.ckb200_model_get_pos(s.handle) == len(case.ids)
    assert s.lib.ckb200_model_set_pos(s.handle, 5) != 0      # a recurrent state cannot move back
    s.lib.ckb200_clear_error()
    s.close()


def test_context_end_and_bad_arguments_are_errors(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=20)
    s = case.session(True, 16)
    assert error(s.extend(case.ids[:16], range(16)), case.want[:16]) < TOL[True]
    for tokens, want in ((case.ids[16:17], [0]), (case.ids[16:18], [1])):
        with pytest.raises(RuntimeError):
            s.extend(tokens, want)
        s.lib.ckb200_clear_error()
    s.reset()
    with pytest.raises(RuntimeError):
        s.extend(case.ids[:4], [4])
    s.lib.ckb200_clear_error()
    assert error(s.extend(case.ids[:16], range(16)), case.want[:16]) < TOL[True]
    s.close()


@pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [3, 11])
def test_batch_of_sequences(pkg, ck, tmp_path, batch, float32):
    """`batch` sequences side by side (prompt portions, then steps) against each alone."""
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=4)
    T, V = 26, case.cfg["vocab"]
    ids = np.random.default_rng(9).integers(0, V, (T, batch)).astype(np.int32)
    want = np.stack([case.oracle(ids[:, b]) for b in range(batch)], axis=1)
    lib, api = ck, pkg.model_api
    api.bind_model_api(lib)
    lib.ckb200_tune_set(b"model_f32", int(float32))
    lib.ckb200_tune_set(b"model_max_seq", 40)
    m = lib.ckb200_model_open(case.dir.encode(), batch)
    try:
        assert m, lib.ckb200_last_error_message()
        got = np.zeros((T, batch, V), np.float32)
        t = 0
        for n in (2, 13, 1, 1, 5, 1, 1, 1, 1):
            part, places = np.ascontiguousarray(ids[t:t + n]), np.arange(n, dtype=np.int32)
            out = np.zeros((n, batch, V), np.float32)
            assert lib.ckb200_model_extend(m, api.vptr(part), n, api.vptr(places), n, api.vptr(out)) == 0, lib.ckb200_last_error_message()
            got[t:t + n] = out
            t += n
        assert t == T
        assert error(got.reshape(-1, V), want.reshape(-1, V)) < TOL[float32]
    finally:
        lib.ckb200_model_free(m)
        lib.ckb200_tune_set(b"model_f32", 0)


def test_long_decoding(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=330)
    s = case.session(True, 400)
    assert error(run(s, case.ids, [5, 1]), case.want) < TOL[True]
    s.close()
    s = case.session(False, 400)
    assert error(run(s, case.ids, [5, 1]), case.want) < TOL[False]
    s.close()


@pytest.mark.parametrize("tune", ["stack_fused_step", "latent_mma", "model_graph", "pdl", "stack_portion"])
def test_variants_agree(pkg, ck, tmp_path, tune):
    """The unfused step, the CUDA-core attention, eager steps, plain launches, prompts cut inside: the same logits."""
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=60)
    before = ck.ckb200_tune_get(tune.encode(), {"stack_portion": 2048}.get(tune, 1))
    ck.ckb200_tune_set(tune.encode(), 24 if tune == "stack_portion" else 0)
    try:
        for float32 in (True, False):
            check_all(case, float32, {"whole": [10 ** 6], "prompt then decode": [33, 1]})
    finally:
        ck.ckb200_tune_set(tune.encode(), before)


def test_residual_probe(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=21)
    layers = []
    po.forward(case.cfg, case.w64, case.ids, layers)
    s = case.session(True)
    rows = np.zeros((len(layers), 21, case.cfg["width"]), np.float32)
    assert s.lib.ckb200_model_probe_residual(s.handle, pkg.model_api.vptr(rows), 21) == 0
    s.extend(case.ids[:12])
    s.extend(case.ids[12:])
    for i, want in enumerate(layers):
        assert np.abs(rows[i] - want).max() < 1e-4 * np.abs(want).max(), i
    s.close()


def greedy(case, prompt, steps):
    """The oracle's greedy continuation, and the smallest margin between the first and second choice."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = case.oracle(ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, float(top[1] - top[0]) / case.want.std())
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin


def test_greedy_generation_through_the_model_abi(pkg, ck, tmp_path):
    """ck_model_init on the folder, ck_model_embed_tokens for the prompt, ck_model_decode per token - how a chat front end drives a model."""
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=24)
    want, margin = greedy(case, case.ids, 24)
    assert margin > 10 * TOL[True], "ties: choose another seed"
    ck.ckb200_tune_set(b"model_f32", 1)
    ck.ckb200_tune_set(b"model_max_seq", 64)
    v7 = C.CDLL(pkg.find_lib("libckb200_model_v7.so"))
    try:
        assert v7.ck_model_init(case.dir.encode()) == 0
        V = v7.ck_model_get_vocab_size()
        assert V == case.cfg["vocab"] and v7.ck_model_get_context_window() == 64
        for _ in range(2):
            ids = np.ascontiguousarray(case.ids, dtype=np.int32)
            logits = np.zeros(V, np.float32)
            assert v7.ck_model_embed_tokens(ids.ctypes.data_as(C.c_void_p), len(ids)) == 0
            assert v7.ck_model_forward(logits.ctypes.data_as(C.c_void_p)) == 0
            got = []
            for _ in want:
                got.append(int(logits.argmax()))
                assert v7.ck_model_decode(C.c_int32(got[-1]), logits.ctypes.data_as(C.c_void_p)) == 0
            assert got == want
            v7.ck_model_kv_cache_reset()
    finally:
        v7.ck_model_free()
        ck.ckb200_tune_set(b"model_f32", 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(pkg, ck, tmp_path, dtype):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=40)
    out = tmp_path / "out"
    out.mkdir()
    ids = [int(x) for x in case.ids]
    other = case.oracle(ids[::-1][:12])
    steps = [({"step": 0, "entries": [{"id": "a", "tokens": ids[:30], "want": [0, 29]}], "end": []}, case.want[[0, 29]]),
             ({"step": 1, "entries": [{"id": "a", "tokens": ids[30:33], "want": []}], "end": []}, None),
             ({"step": 2, "entries": [{"id": "a", "tokens": ids[33:34], "want": [0]}], "end": ["a"]}, case.want[[33]]),
             ({"step": 3, "entries": [{"id": "b", "tokens": ids[::-1][:12], "want": [3, 11]}], "end": ["b"]}, other[[3, 11]])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", case.dir, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s, _ in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    for s, want in steps:
        path = out / f"{s['step']}.f32"
        assert path.exists() == (want is not None)
        if want is not None:
            assert error(np.fromfile(path, "<f4").reshape(want.shape), want) < TOL[dtype == "float32"]


# ---- the products alone

class LinMat(C.Structure):
    _fields_ = [("w", C.c_void_p), ("rows", C.c_int), ("cols", C.c_int), ("tmap", C.c_uint64 * 16)]


class LinSeg(C.Structure):
    _fields_ = [("row0", C.c_int), ("count", C.c_int), ("kind", C.c_int), ("ld", C.c_int), ("dst", C.c_void_p), ("x0", C.c_int), ("cap", C.c_float),
                ("vec", C.c_void_p)]


class LinSegs(C.Structure):
    _fields_ = [("n", C.c_int), ("act_f32", C.c_int), ("s", LinSeg * 8)]


@pytest.mark.parametrize("tokens", [1, 2, 5, 8, 9, 33, 100, 300])
@pytest.mark.parametrize("path", ["gemv", "f32", "tc"])
def test_product_and_its_segments(ck, path, tokens):
    """One stacked matrix with all four kinds of outputs: fp32 rows, activation rows, SwiGLU units, sums into the residual."""
    import torch

    if path == "gemv" and tokens > 8:
        pytest.skip("the streaming product takes up to eight rows")
    K, counts = 192, (45, 70, 41, 130)                        # outputs of the segments; 41 SwiGLU units are 82 rows
    row0, rows = [], 0
    for kind, n in enumerate(counts):
        row0.append(rows)
        rows += (n + 15) // 16 * 32 if kind == 2 else (n + 31) // 32 * 32
    g = torch.Generator(device="cuda").manual_seed(tokens)
    w = torch.zeros(rows, K, device="cuda")
    for kind, n in enumerate(counts):
        if kind == 2:
            for u in range(n):
                for half in range(2):
                    w[row0[2] + u // 16 * 32 + u % 16 + 16 * half] = torch.randn(K, generator=g, device="cuda") * 0.1
        else:
            w[row0[kind]:row0[kind] + n] = torch.randn(n, K, generator=g, device="cuda") * 0.1
    w16 = w.to(torch.bfloat16)
    act = torch.bfloat16 if path == "tc" else torch.float32
    x = torch.randn(tokens, K + 8, generator=g, device="cuda").to(act)
    x64, w64 = x[:, :K].double(), w16.double()
    full = x64 @ w64.T
    outs = [torch.full((tokens, n + 3), 7.0, dtype=torch.float32 if kind in (0, 3) else act, device="cuda") for kind, n in enumerate(counts)]
    torch.cuda.synchronize()
    mat = LinMat(w16.data_ptr(), rows, K)
    ck.ckb_linear_encode.argtypes = [C.c_void_p]
    assert ck.ckb_linear_encode(C.byref(mat)) == 0
    sg = LinSegs(4, int(act == torch.float32))
    for i, n in enumerate(counts):
        sg.s[i] = LinSeg(row0[i], n, i, n + 3, outs[i].data_ptr())
    P, I = C.c_void_p, C.c_int
    if path == "gemv":
        ck.ckb_launch_linear_gemv.argtypes = [P, P, I, I, P, I, C.c_float, P, P]
        rc = ck.ckb_launch_linear_gemv(C.byref(mat), x.data_ptr(), K + 8, tokens, None, 0, 0.0, C.byref(sg), None)
    else:
        f = getattr(ck, "ckb_launch_linear_" + path)
        f.argtypes = [P, P, I, I, P, P]
        rc = f(C.byref(mat), x.data_ptr(), K + 8, tokens, C.byref(sg), None)
    assert rc == 0 and ck.ckb200_synchronize() == 0
    tol = 1e-5 if path != "tc" else 1e-2
    for i, n in enumerate(counts):
        if i == 2:
            idx = torch.tensor([row0[2] + u // 16 * 32 + u % 16 for u in range(n)], device="cuda")
            gate, up = full[:, idx], full[:, idx + 16]
            want = gate * torch.sigmoid(gate) * up
        else:
            want = full[:, row0[i]:row0[i] + n] + (7.0 if i == 3 else 0.0)
        assert (outs[i][:, :n].double() - want).abs().max() < (tol if i in (1, 2) else 2e-5) * want.abs().max(), (path, i)
        assert (outs[i][:, n:] == 7.0).all(), "a store past the segment's outputs"
