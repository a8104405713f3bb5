"""Layer-stack models on the GPU against the plain numpy restatement: every mixer alone and together, whole prompts, portions, decoding,
batches, state that is given back and used again, sizes that fit no tile."""
from __future__ import annotations

import ctypes as C
import os

import numpy as np
import pytest

import puzevik_model as pm
from stack_cases import TOL, Case, batch_logits, check_all, error, greedy, greedy_through_the_model_abi, run, trace

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

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
    got = batch_logits(pkg, ck, case, ids, (2, 13, 1, 1, 5, 1, 1, 1, 1), float32, 40)
    assert error(got.reshape(-1, V), want.reshape(-1, V)) < TOL[float32]


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
    case.oracle(case.ids, layers)
    s = case.session(True)
    rows = np.zeros((len(layers), 21, case.cfg["width"]), np.float32)
    assert s.lib.ckb200_model_probe_residual(s.handle, pkg.model_api.vptr(rows), 21) == 0
    s.extend(case.ids[:12])
    s.extend(case.ids[12:])
    for i, want in enumerate(layers):
        assert np.abs(rows[i] - want).max() < 1e-4 * np.abs(want).max(), i
    s.close()


def test_greedy_generation_through_the_model_abi(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=24)
    want, margin = greedy(case, case.ids, 24)
    assert margin > 10 * TOL[True], "ties: choose another seed"
    assert greedy_through_the_model_abi(pkg, ck, case, 24) == [want, want]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(pkg, ck, tmp_path, dtype):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=40)
    ids = [int(x) for x in case.ids]
    other = case.oracle(ids[::-1][:12])
    steps = [({"step": 0, "entries": [{"id": "a", "tokens": ids[:30], "want": [0, 29]}], "end": []}, case.want[[0, 29]]),
             ({"step": 1, "entries": [{"id": "a", "tokens": ids[30:33], "want": []}], "end": []}, None),
             ({"step": 2, "entries": [{"id": "a", "tokens": ids[33:34], "want": [0]}], "end": ["a"]}, case.want[[33]]),
             ({"step": 3, "entries": [{"id": "b", "tokens": ids[::-1][:12], "want": [3, 11]}], "end": ["b"]}, other[[3, 11]])]
    trace(ROOT, case, steps, dtype, tmp_path / "out")


# ---- the products alone

class LinMat(C.Structure):
    _fields_ = [("w", C.c_void_p), ("rows", C.c_int), ("cols", C.c_int), ("tmap", C.c_uint64 * 16)]


class LinSeg(C.Structure):
    _fields_ = [("row0", C.c_int), ("count", C.c_int), ("kind", C.c_int), ("ld", C.c_int), ("dst", C.c_void_p), ("x0", C.c_int), ("cap", C.c_float),
                ("vec", C.c_void_p)]


class LinSegs(C.Structure):
    _fields_ = [("n", C.c_int), ("act", C.c_int), ("s", LinSeg * 8)]


F32, ACT, SWIGLU, ADD, SILU, TANH, DECAY, CAP = range(8)


def launch_product(ck, path, mat, x, ldx, tokens, sg):
    P, I = C.c_void_p, C.c_int
    if path == "gemv":
        ck.ckb_launch_linear_gemv.argtypes = [P, P, I, I, P, I, C.c_float, P, P]
        return ck.ckb_launch_linear_gemv(C.byref(mat), x.data_ptr(), ldx, tokens, None, 0, 0.0, C.byref(sg), None)
    f = getattr(ck, "ckb_launch_linear_" + path)
    f.argtypes = [P, P, I, I, P, P]
    return f(C.byref(mat), x.data_ptr(), ldx, tokens, C.byref(sg), None)


@pytest.mark.parametrize("inputs", [1, 3])
@pytest.mark.parametrize("tokens", [1, 2, 5, 8, 9, 33, 100, 300])
@pytest.mark.parametrize("path", ["gemv", "f32", "tc"])
def test_product_and_its_segments(ck, path, tokens, inputs):
    """One stacked matrix with all kinds of outputs, over one input or with segments that read different parts of the rows."""
    import torch

    if path == "gemv" and tokens > 8:
        pytest.skip("the streaming product takes up to eight rows")
    # (kind, outputs, input); 41 SwiGLU units are 82 rows
    parts = [(F32, 45, 0), (ACT, 70, 0), (SWIGLU, 41, 0), (ADD, 130, 1), (SILU, 33, 1), (TANH, 20, 2), (DECAY, 64, 2), (CAP, 31, 2)]
    K, row0, rows, last = 192, [], 0, 0
    for kind, n, src in parts:
        src = min(src, inputs - 1)
        if src != last:
            rows, last = (rows + 127) // 128 * 128, src
        row0.append(rows)
        rows += (n + 15) // 16 * 32 if kind == SWIGLU else (n + 31) // 32 * 32
    g = torch.Generator(device="cuda").manual_seed(tokens)
    w = torch.zeros(rows, K, device="cuda")
    for r0, (kind, n, _) in zip(row0, parts):
        if kind == SWIGLU:
            for u in range(n):
                for half in range(2):
                    w[r0 + u // 16 * 32 + u % 16 + 16 * half] = torch.randn(K, generator=g, device="cuda") * 0.1
        else:
            w[r0:r0 + n] = torch.randn(n, K, generator=g, device="cuda") * 0.1
    w16 = w.to(torch.bfloat16)
    act, ldx = torch.bfloat16 if path == "tc" else torch.float32, K * inputs + 8
    x = torch.randn(tokens, ldx, generator=g, device="cuda").to(act)
    w64, bias = w16.double(), torch.randn(64, generator=g, device="cuda")
    is_act = (ACT, SWIGLU, TANH)
    outs = [torch.full((tokens, n + 3), 7.0, dtype=act if kind in is_act else torch.float32, device="cuda") for kind, n, _ in parts]
    torch.cuda.synchronize()
    mat = LinMat(w16.data_ptr(), rows, K)
    ck.ckb_linear_encode.argtypes = [C.c_void_p]
    assert ck.ckb_linear_encode(C.byref(mat)) == 0
    sg = LinSegs(len(parts), int(act == torch.float32))
    for i, (kind, n, src) in enumerate(parts):
        sg.s[i] = LinSeg(row0[i], n, kind, n + 3, outs[i].data_ptr(), min(src, inputs - 1) * K, 1.5, bias.data_ptr())
    assert launch_product(ck, path, mat, x, ldx, tokens, sg) == 0 and ck.ckb200_synchronize() == 0
    tol = 1e-5 if path != "tc" else 1e-2
    for r0, (kind, n, src), out in zip(row0, parts, outs):
        src = min(src, inputs - 1)
        full = x[:, src * K:src * K + K].double() @ w64.T
        if kind == SWIGLU:
            idx = torch.tensor([r0 + u // 16 * 32 + u % 16 for u in range(n)], device="cuda")
            want = torch.nn.functional.silu(full[:, idx]) * full[:, idx + 16]
        else:
            z = full[:, r0:r0 + n]
            want = {F32: lambda: z, ACT: lambda: z, ADD: lambda: z + 7.0, SILU: lambda: z * torch.sigmoid(z), TANH: lambda: torch.tanh(z),
                    DECAY: lambda: torch.exp(-torch.exp(z + bias.double()[:n])), CAP: lambda: 1.5 * torch.tanh(z / 1.5)}[kind]()
        assert (out[:, :n].double() - want).abs().max() < (tol if kind in is_act else 2e-5) * want.abs().max(), (path, kind)
        assert (out[:, n:] == 7.0).all(), "a store past the segment's outputs"


def with_lead(x, lead):
    """bfloat16 rows with the first `lead` of them as two pieces each: every eight take sixteen places."""
    import torch

    hi = x.to(torch.bfloat16)
    lo = (x - hi.float()).to(torch.bfloat16)
    blocks = [torch.cat([hi[i:i + 8], lo[i:i + 8]]) for i in range(0, lead, 8)]
    return torch.cat(blocks + [hi[lead:]]).contiguous()


@pytest.mark.parametrize("tokens, lead", [(8, 8), (9, 8), (21, 16), (40, 8), (130, 8), (300, 24)])
def test_product_of_rows_with_a_lead(ck, tokens, lead):
    """Lead rows come out as from fp32 inputs, into fp32 rows, sums, and activation rows with a lead of their own."""
    import torch

    K, parts = 320, [(F32, 100), (ADD, 40), (ACT, 37), (SWIGLU, 41), (SILU, 30), (TANH, 64)]
    row0, rows = [], 0
    for kind, n in parts:
        row0.append(rows)
        rows += (n + 15) // 16 * 32 if kind == SWIGLU else (n + 31) // 32 * 32
    g = torch.Generator(device="cuda").manual_seed(tokens)
    w16 = (torch.randn(rows, K, generator=g, device="cuda") * 0.1).to(torch.bfloat16)
    x = torch.randn(tokens, K, generator=g, device="cuda")
    packed = with_lead(x, lead)
    acts = (ACT, SWIGLU, TANH)
    outs = [torch.full((tokens + lead if kind in acts else tokens, n), 7.0, dtype=torch.bfloat16 if kind in acts else torch.float32, device="cuda") for kind, n in parts]
    torch.cuda.synchronize()
    mat = LinMat(w16.data_ptr(), rows, K)
    ck.ckb_linear_encode.argtypes = [C.c_void_p]
    assert ck.ckb_linear_encode(C.byref(mat)) == 0
    sg = LinSegs(len(parts), -lead)
    for i, (kind, n) in enumerate(parts):
        sg.s[i] = LinSeg(row0[i], n, kind, n, outs[i].data_ptr())
    assert launch_product(ck, "tc", mat, packed, K, tokens, sg) == 0 and ck.ckb200_synchronize() == 0
    exact = torch.cat([x[:lead].double(), x[lead:].to(torch.bfloat16).double()]) @ w16.double().T
    for r0, (kind, n), out in zip(row0, parts, outs):
        z = exact[:, r0:r0 + n]
        if kind == SWIGLU:
            idx = torch.tensor([r0 + u // 16 * 32 + u % 16 for u in range(n)], device="cuda")
            z = torch.nn.functional.silu(exact[:, idx]) * exact[:, idx + 16]
        want = {SILU: torch.nn.functional.silu, TANH: torch.tanh, ADD: lambda v: v + 7.0}.get(kind, lambda v: v)(z)
        out, scale = out.double(), want.abs().max()
        if kind in acts:
            first = torch.cat([out[i:i + 8] + out[i + 8:i + 16] for i in range(0, 2 * lead, 16)])
            if tokens > lead:
                assert (out[2 * lead:] - want[lead:]).abs().max() < 5e-3 * scale, kind
        else:
            first = out[:lead]
            assert (out - want).abs().max() < 5e-5 * scale, kind
        assert (first - want[:lead]).abs().max() < 5e-5 * scale, kind


class LinInput(C.Structure):
    _fields_ = [("x", C.c_void_p), ("ldx", C.c_int), ("n", C.c_int), ("eps", C.c_float), ("y", C.c_void_p), ("y_w", C.c_void_p), ("ldy", C.c_int), ("x_out", C.c_void_p),
                ("mu", C.c_void_p), ("before", C.c_void_p), ("ld_before", C.c_int), ("norm_w", C.c_void_p), ("part", C.c_void_p), ("part_n", C.c_int), ("part_col", C.c_int),
                ("part_width", C.c_int)]


class StreamRows(C.Structure):
    _fields_ = [("x", C.c_void_p), ("y", C.c_void_p), ("y_w", C.c_void_p), ("ldx", C.c_int), ("ldy", C.c_int), ("idx", C.c_void_p), ("x_out", C.c_void_p), ("norm_w", C.c_void_p),
                ("mu", C.c_void_p), ("before", C.c_void_p), ("n_mu", C.c_int), ("ld_mu", C.c_int), ("ld_before", C.c_int), ("dst", C.c_void_p), ("ldd", C.c_int),
                ("act", C.c_int), ("n", C.c_int), ("width", C.c_int), ("eps", C.c_float)]


class Stream:
    """Random residual rows, a sublayer's output that is to join them, mixing vectors and previous rows, padded with zeros."""

    def __init__(self, rows, n, ld, batch, inputs=3):
        import torch

        g = torch.Generator(device="cuda").manual_seed(rows * 1000 + n)

        def padded(*shape):
            t = torch.zeros(*shape, ld, device="cuda")
            t[..., :n] = torch.randn(*shape, n, generator=g, device="cuda")
            return t

        self.n, self.x, self.y, self.before, self.mu = n, padded(rows), 3.0 * padded(rows), padded(batch), padded(inputs)
        self.y_w, self.norm_w, self.x_out = padded(), padded(), torch.full((rows, ld), 7.0, device="cuda")
        self.eps = 0.05

    def rms(self, v):
        return v / (v[..., :self.n].double().pow(2).mean(-1, keepdim=True) + self.eps).sqrt()

    def joined(self, join):
        return self.x.double() + (self.rms(self.y.double()) * self.y_w if join else 0.0)

    def mixed(self, v, batch):
        import torch

        last = torch.cat([self.before.double(), v])[:len(v)] if batch else None
        return torch.stack([v + (last - v) * m.double() for m in self.mu], 1)


@pytest.mark.parametrize("mix", [False, True])
@pytest.mark.parametrize("join", [False, True])
@pytest.mark.parametrize("norm", [False, True])
@pytest.mark.parametrize("rows", [1, 3, 8])
def test_streaming_product_makes_its_input(ck, rows, norm, join, mix):
    """The residual joined by a normed output, mixed with the previous token's row, normed, on the way into the product."""
    import torch

    n, ld, counts = 150, 192, (40, 64, 9)
    st = Stream(rows, n, ld, rows)
    w = (torch.randn(128 * 3, ld, device="cuda") * 0.1).to(torch.bfloat16)
    outs = [torch.full((rows, c), 7.0, device="cuda") for c in counts]
    torch.cuda.synchronize()
    mat = LinMat(w.data_ptr(), w.shape[0], ld)
    assert ck.ckb_linear_encode(C.byref(mat)) == 0
    sg = LinSegs(3, 1)
    for i, c in enumerate(counts):
        sg.s[i] = LinSeg(128 * i, c, F32, c, outs[i].data_ptr(), i * ld if mix else 0)
    a = LinInput(x=st.x.data_ptr(), ldx=ld, n=n, eps=st.eps)
    if join:
        a.y, a.y_w, a.ldy, a.x_out = st.y.data_ptr(), st.y_w.data_ptr(), ld, st.x_out.data_ptr()
    if mix:
        a.mu, a.before, a.ld_before = st.mu.data_ptr(), st.before.data_ptr(), ld
    if norm:
        a.norm_w = st.norm_w.data_ptr()
    ck.ckb_launch_linear_gemv_in.argtypes = [C.c_void_p, C.c_void_p, C.c_int, C.c_void_p, C.c_void_p]
    assert ck.ckb_launch_linear_gemv_in(C.byref(mat), C.byref(a), rows, C.byref(sg), None) == 0 and ck.ckb200_synchronize() == 0
    v = st.joined(join)
    if join:
        assert (st.x_out.double() - v).abs().max() < 1e-5
    for i, out in enumerate(outs):
        h = v + (st.before.double() - v) * st.mu[i].double() if mix else v
        if norm:
            h = st.rms(h) * st.norm_w
        want = h @ w[128 * i:128 * i + counts[i]].double().T
        assert (out.double() - want).abs().max() < 2e-5 * want.abs().max(), i


@pytest.mark.parametrize("rows", [1, 2, 7])
def test_streaming_product_scales_a_part_of_its_input(ck, rows):
    import torch

    K, col, parts, width = 256, 128, 37, 90
    x, w = torch.randn(rows, K, device="cuda"), (torch.randn(64, K, device="cuda") * 0.1).to(torch.bfloat16)
    ss, out = torch.rand(rows, parts, device="cuda"), torch.zeros(rows, 64, device="cuda")
    torch.cuda.synchronize()
    mat = LinMat(w.data_ptr(), 64, K)
    assert ck.ckb_linear_encode(C.byref(mat)) == 0
    sg = LinSegs(1, 1)
    sg.s[0] = LinSeg(0, 64, F32, 64, out.data_ptr())
    a = LinInput(x=x.data_ptr(), ldx=K, eps=0.1, part=ss.data_ptr(), part_n=parts, part_col=col, part_width=width)
    ck.ckb_launch_linear_gemv_in.argtypes = [C.c_void_p, C.c_void_p, C.c_int, C.c_void_p, C.c_void_p]
    assert ck.ckb_launch_linear_gemv_in(C.byref(mat), C.byref(a), rows, C.byref(sg), None) == 0 and ck.ckb200_synchronize() == 0
    h = x.double()
    h[:, col:] /= (ss.double().sum(1, keepdim=True) / width + 0.1).sqrt()
    want = h @ w.double().T
    assert (out.double() - want).abs().max() < 2e-5 * want.abs().max()


@pytest.mark.parametrize("mode", ["plain", "norm", "some rows", "mix"])
@pytest.mark.parametrize("join", [False, True])
@pytest.mark.parametrize("n, ld, tokens, batch", [(150, 192, 21, 1), (150, 192, 9, 3), (1500, 1536, 17, 2), (5000, 5056, 3, 1), (9000, 9024, 10, 1)])
def test_stream_rows(ck, n, ld, tokens, batch, join, mode):
    import torch

    rows = tokens * batch
    st = Stream(rows, n, ld, batch)
    idx = torch.tensor([2, 0, rows - 1], dtype=torch.int32, device="cuda")
    count = 3 if mode == "some rows" else rows
    ldd = 3 * ld if mode == "mix" else ld
    out = torch.full((count, ldd), 7.0, device="cuda")
    torch.cuda.synchronize()
    a = StreamRows(x=st.x.data_ptr(), ldx=ld, dst=out.data_ptr(), ldd=ldd, act=1, n=n, width=ld, eps=st.eps)
    if join:
        a.y, a.y_w, a.ldy, a.x_out = st.y.data_ptr(), st.y_w.data_ptr(), ld, st.x_out.data_ptr()
    if mode in ("norm", "some rows"):
        a.norm_w = st.norm_w.data_ptr()
    if mode == "some rows":
        a.idx, a.x_out = idx.data_ptr(), None
    if mode == "mix":
        a.mu, a.before, a.n_mu, a.ld_mu, a.ld_before = st.mu.data_ptr(), st.before.data_ptr(), 3, ld, ld
    ck.ckb_launch_stream_rows.argtypes = [C.c_void_p, C.c_int, C.c_int, C.c_void_p]
    assert ck.ckb_launch_stream_rows(C.byref(a), count, 1 if mode == "some rows" else batch, None) == 0 and ck.ckb200_synchronize() == 0
    v = st.joined(join)
    want = v
    if mode in ("norm", "some rows"):
        want = st.rms(v) * st.norm_w
    if mode == "some rows":
        want = want[idx.long()]
    if mode == "mix":
        want = st.mixed(v, batch).reshape(rows, -1)
    if join and mode != "some rows":
        assert (st.x_out.double() - v).abs().max() < 1e-5
    assert (out.double() - want).abs().max() < 2e-5
