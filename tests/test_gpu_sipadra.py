"""Sipadra on the GPU against the plain numpy restatement: every mixer and each of its halves alone and together, whole prompts, portions,
decoding, batches, window edges, slots that are used again, states that remember far back, sizes that fit no tile."""
from __future__ import annotations

import copy
import os

import numpy as np
import pytest

import sipadra_model as sm
from stack_cases import TOL, Case, batch_logits, check_all, error, greedy, greedy_through_the_model_abi, run, trace

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("float32", [True, False], ids=["float32", "bfloat16"])


def only_left(**kw):
    return sm.layer("parallel", sm.parallel(sm.left(**kw), right_scale=0.0))


def only_right(**kw):
    return sm.layer("parallel", sm.parallel(right_arm=sm.right(**kw), left_scale=0.0))


SINGLE = {
    "both halves": sm.layer("parallel", sm.parallel()),
    "attention": only_left(),
    "attention, no scaling of the rotation": only_left(scaling=None),
    "attention, all dimensions rotated, stretched": only_left(dim=32, dims=32, scaling=sm.yarn(factor=8.0, original=100, fast=3.0, slow=0.2), base=60.0),
    "attention, ramp without width": only_left(scaling=sm.yarn(factor=2.0, original=9, fast=1.0, slow=1.0)),
    "attention, ramp past the last pair": only_left(dim=16, dims=8, scaling=sm.yarn(factor=5.0, original=5000, fast=2.0, slow=0.001), base=7.0),
    "attention, two rotated dimensions, one head": only_left(heads=1, kv_heads=1, dim=9, vdim=7, dims=2),
    "attention, key heads as many as heads": only_left(heads=3, kv_heads=3, dim=32, vdim=64),
    "attention, six heads of one key head": only_left(heads=6, kv_heads=1, dim=64, vdim=32),
    "attention, wide keys": only_left(heads=2, kv_heads=1, dim=200, vdim=72, dims=36),
    "attention, wide values": only_left(heads=2, kv_heads=2, dim=72, vdim=203, size=70),
    "attention, only itself": only_left(size=1),
    "attention, itself and one": only_left(size=2),
    "attention, window of a tile": only_left(size=64),
    "attention, window past the prompt": only_left(size=500),
    "lightning": only_right(),
    "lightning, one head, no decay": only_right(heads=1, dim=32, vdim=64, decay=[1.0]),
    "lightning, wide values": only_right(heads=2, dim=7, vdim=300),
    "lightning, wide keys": only_right(heads=2, dim=200, vdim=33, decay=[0.3, 0.99]),
    "halves of unlike sizes": sm.layer("parallel", sm.parallel(sm.left(heads=5, kv_heads=1, dim=16, vdim=13, dims=6), sm.right(heads=7, dim=12, vdim=9), 1.0, -0.4)),
    "wkv": sm.layer("wkv", sm.wkv()),
    "wkv, one head": sm.layer("wkv", sm.wkv(heads=1, dim=32)),
    "wkv, odd heads": sm.layer("wkv", sm.wkv(heads=7, dim=13)),
    "wkv, heads of 64": sm.layer("wkv", sm.wkv(heads=2, dim=64)),
    "wkv, wide heads": sm.layer("wkv", sm.wkv(heads=2, dim=150)),
}


@BOTH
@pytest.mark.parametrize("name", list(SINGLE))
def test_one_mixer(pkg, ck, tmp_path, name, float32):
    check_all(Case(pkg, ck, tmp_path, sm.config([SINGLE[name]])), float32)


@BOTH
@pytest.mark.parametrize("ff", [16, 50, 200])
def test_feed_forward_after_a_mixer(pkg, ck, tmp_path, ff, float32):
    cfg = sm.config([sm.layer("wkv", sm.wkv(), ff), sm.layer("parallel", sm.parallel(), ff)], width=72)
    check_all(Case(pkg, ck, tmp_path, cfg), float32, {"whole": [10 ** 6], "decode": [1], "fives": [5]})


@pytest.mark.parametrize("rank", [1, 64, 70])
def test_ranks_of_the_decay(pkg, ck, tmp_path, rank):
    check_all(Case(pkg, ck, tmp_path, sm.config([sm.layer("wkv", sm.wkv(), 32)]), rank=rank), True, {"whole": [10 ** 6], "decode": [1], "threes": [3]})


def stack_config(**kw):
    return sm.config([sm.layer("wkv", sm.wkv(), 120), sm.layer("parallel", sm.parallel(), 72), sm.layer("wkv", sm.wkv(heads=5, dim=16)),
                      sm.layer("parallel", sm.parallel(sm.left(heads=2, kv_heads=2, dim=8, vdim=16, dims=8, size=9), sm.right(heads=2, dim=32, vdim=24))),
                      sm.layer("wkv", sm.wkv(heads=2, dim=40), 96)], **kw)


@BOTH
def test_stack_in_all_schedules(pkg, ck, tmp_path, float32):
    check_all(Case(pkg, ck, tmp_path, stack_config()), float32)


@pytest.mark.parametrize("first", [0, 1])
def test_a_stack_may_begin_with_any_layer(pkg, ck, tmp_path, first):
    cfg = stack_config()
    cfg["layers"] = cfg["layers"][first:first + 2]
    check_all(Case(pkg, ck, tmp_path, cfg), True, {"whole": [10 ** 6], "decode": [1], "sevens": [7]})


def test_large_eps_and_a_low_cap(pkg, ck, tmp_path):
    """eps of the size of the mean square: it must stand inside the root, in every norm.  Most logits lie on the cap's flat part."""
    check_all(Case(pkg, ck, tmp_path, stack_config(eps=0.3, cap=0.8)), True, {"whole": [10 ** 6], "decode": [1], "nines": [9]})


@BOTH
def test_many_tiles(pkg, ck, tmp_path, float32):
    """More rows, columns and keys than one tile of any kernel has."""
    cfg = sm.config([sm.layer("wkv", sm.wkv(heads=3, dim=64), 300), sm.layer("parallel", sm.parallel(sm.left(heads=4, kv_heads=2, dim=128, vdim=128, dims=64, size=150, scale=0.1),
                                                                                                   sm.right(heads=3, dim=64, vdim=128)), 90)], width=328, vocab=413)
    case = Case(pkg, ck, tmp_path, cfg, tokens=290)
    check_all(case, float32, {"whole": [10 ** 6], "cut": [129, 1, 31, 64], "two tokens last": [257, 2], "decode": [200, 1]}, 300)


# ---- window edges

SHARP = 1.5                                                  # attention scale with which most queries take their value from one key or two


def edge_case(pkg, ck, tmp_path, size, **kw):
    return Case(pkg, ck, tmp_path, sm.config([sm.layer("parallel", sm.parallel(sm.left(size=size, scale=SHARP, **kw), right_scale=0.0))]), tokens=210, seed=11)


@BOTH
@pytest.mark.parametrize("size", [5, 33, 63, 64, 65, 128, 130])
def test_window_edges(pkg, ck, tmp_path, size, float32):
    """The key just inside the window decides some queries, and the one just outside would."""
    case = edge_case(pkg, ck, tmp_path, size)
    for off in (-1, 1):                                      # a window one key off shows far above the tolerance
        cfg = copy.deepcopy(case.cfg)
        cfg["layers"][0]["mixer"]["left"]["mask"]["size"] = size + off
        assert error(case.oracle(case.ids, cfg=cfg), case.want) > 4 * TOL[False]
    check_all(case, float32, {"whole": [10 ** 6], "decode": [1], "at 64s": [64], "at 37s": [37], "prompt then decode": [140, 1]})


@pytest.mark.parametrize("size", [33, 64])
def test_a_key_outside_every_window_leaves_no_trace(pkg, ck, tmp_path, size):
    case = edge_case(pkg, ck, tmp_path, size)
    for place in range(40, 120):
        other = case.ids.copy()
        other[place] = (other[place] + 1) % case.cfg["vocab"]
        if np.abs(case.oracle(other) - case.want)[place + size - 1].max() > 0.1 * case.want.std():
            break                                            # a query that takes much of its value from the last key of its window
    else:
        pytest.fail("the edge does not show: choose another seed")
    for cuts in ([10 ** 6], [1], [50, 20, 1]):
        s = case.session(True)
        a = run(s, case.ids, cuts)
        s.reset()
        b = run(s, other, cuts)
        s.close()
        assert np.array_equal(a[:place], b[:place]) and np.array_equal(a[place + size:], b[place + size:])
        assert np.abs(a - b)[place + size - 1].max() > 0.09 * case.want.std()


@BOTH
@pytest.mark.parametrize("portion", [1, 24, 60])
def test_slots_are_used_again(pkg, ck, tmp_path, portion, float32):
    """Short passes, so that the window's ring of slots is as short as it can be and goes round several times, in prompts and decoding."""
    case = edge_case(pkg, ck, tmp_path, 41, heads=4, kv_heads=4, dim=12, vdim=10, dims=4)
    before = ck.ckb200_tune_get(b"stack_portion", 2048)
    ck.ckb200_tune_set(b"stack_portion", portion)
    try:
        check_all(case, float32, {"whole": [10 ** 6], "decode": [1], "mixed": [60, 1, 1, 23, 2], "prompt then decode": [100, 1]})
    finally:
        ck.ckb200_tune_set(b"stack_portion", before)


@BOTH
def test_scores_of_unlike_size(pkg, ck, tmp_path, float32):
    """Queries and keys of very different lengths: the unit mean square takes the length out, whatever it is, and eps counts for tiny ones."""
    case = Case(pkg, ck, tmp_path, sm.config([only_left(scale=0.6)], eps=1e-4), tokens=90)
    w = dict(case.w)
    w["l0.mix.left.q"] = sm.bf16_round(w["l0.mix.left.q"] * np.float32(64.0))
    w["l0.mix.left.k"] = sm.bf16_round(w["l0.mix.left.k"] * np.float32(0.01))
    import puzevik_model
    puzevik_model.write(tmp_path / "model", case.cfg, w)
    case.w64 = {k: v.astype(np.float64) for k, v in w.items()}
    case.want = case.oracle(case.ids)
    check_all(case, float32, {"whole": [10 ** 6], "decode": [1], "tens": [10]})


# ---- recurrent state

@pytest.mark.parametrize("kind", ["wkv", "lightning"])
def test_state_remembers_far_back(pkg, ck, tmp_path, kind):
    """Slow decays: the first tokens still show after 200 steps, however the steps are cut."""
    layer = sm.layer("wkv", sm.wkv()) if kind == "wkv" else only_right(decay=[0.9995, 0.999, 1.0])
    case = Case(pkg, ck, tmp_path, sm.config([layer]), tokens=230, w0=(-9.0, -7.0))
    other = case.ids.copy()
    other[:4] = (other[:4] + 1) % case.cfg["vocab"]
    assert np.abs(case.oracle(other)[-1] - case.want[-1]).max() / case.want.std() > 50 * TOL[True]
    check_all(case, True, {"whole": [10 ** 6], "decode": [1], "mixed": [17, 1, 40, 2, 8]})


def test_strong_decay_forgets(pkg, ck, tmp_path):
    """Decays that underflow to zero within a token: no overflow, no stale state."""
    cfg = sm.config([sm.layer("wkv", sm.wkv()), only_right(decay=[0.0, 1e-30, 1e-6])])
    check_all(Case(pkg, ck, tmp_path, cfg, w0=(2.0, 5.0)), True, {"whole": [10 ** 6], "decode": [1], "threes": [3]})


def test_the_previous_token_is_carried_over_every_cut(pkg, ck, tmp_path):
    """All inputs of wkv lean on the previous token alone: a lost or stale row shows at once."""
    case = Case(pkg, ck, tmp_path, sm.config([sm.layer("wkv", sm.wkv(), 40), sm.layer("wkv", sm.wkv())]), tokens=40)
    import puzevik_model
    w = {k: np.ones_like(v) if ".mu." in k else v for k, v in case.w.items()}
    puzevik_model.write(tmp_path / "model", case.cfg, w)
    case.w64 = {k: v.astype(np.float64) for k, v in w.items()}
    case.want = case.oracle(case.ids)
    for float32 in (True, False):
        check_all(case, float32, {"whole": [10 ** 6], "decode": [1], "twos": [2], "mixed": [1, 2, 11, 1, 1, 9, 3]})


# ---- sequences, sessions, batches

@BOTH
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


@pytest.mark.parametrize("batch", [1, 3])
def test_first_tokens_of_a_prompt_keep_their_signs(pkg, ck, tmp_path, batch):
    """At the start of a sequence a head's read-out is one value times r (u * k), and the head norm leaves only the sign of that number.
    Sequences chosen so that it is all but zero for some head: inputs rounded to bfloat16 would turn the head's output around."""
    cfg = sm.config([sm.layer("wkv", sm.wkv(heads=6, dim=16), 64), sm.layer("wkv", sm.wkv(heads=6, dim=16))], vocab=1201)
    case = Case(pkg, ck, tmp_path, cfg, tokens=4)
    w = {k: v.astype(np.float64) for k, v in case.w.items()}
    h = w["embed"]
    r, k = (((1 - w["l0.mix.mu." + n]) * h) @ w["l0.mix." + n].T for n in "rk")
    terms = (r * k).reshape(-1, 6, 16) * w["l0.mix.u"]
    share = np.abs(terms.sum(-1)) / np.abs(terms).sum(-1)
    first = np.argsort(share.min(1))[:6]
    assert share.min(1)[first].max() < 2e-3
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], (30, 6))
    ids[0] = first
    for lo in range(0, 6, batch):
        part = ids[:, lo:lo + batch]
        want = np.stack([case.oracle(part[:, b]) for b in range(batch)], axis=1)
        for portions in ((30,), (2, 28), (12, 18)):
            got = batch_logits(pkg, ck, case, part, portions, False, 40)
            assert error(got.reshape(-1, cfg["vocab"]), want.reshape(-1, cfg["vocab"])) < TOL[False], (lo, portions)


def test_context_end_is_an_error(pkg, ck, tmp_path):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=20)
    s = case.session(True, 16)
    assert error(s.extend(case.ids[:16], range(16)), case.want[:16]) < TOL[True]
    with pytest.raises(RuntimeError):
        s.extend(case.ids[16:17], [0])
    s.lib.ckb200_clear_error()
    s.close()


@BOTH
@pytest.mark.parametrize("batch", [2, 3, 11])
def test_batch_of_sequences(pkg, ck, tmp_path, batch, float32):
    """`batch` sequences side by side (prompt portions, then steps) against each alone."""
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=4)
    V = case.cfg["vocab"]
    ids = np.random.default_rng(9).integers(0, V, (28, batch))
    want = np.stack([case.oracle(ids[:, b]) for b in range(batch)], axis=1)
    got = batch_logits(pkg, ck, case, ids, (2, 13, 1, 1, 5, 2, 1, 1, 1, 1), float32, 40)
    assert error(got.reshape(-1, V), want.reshape(-1, V)) < TOL[float32]


@BOTH
def test_long_decoding(pkg, ck, tmp_path, float32):
    case = Case(pkg, ck, tmp_path, stack_config(), tokens=330)
    s = case.session(float32, 400)
    assert error(run(s, case.ids, [5, 1]), case.want) < TOL[float32]
    s.close()


@pytest.mark.parametrize("tune", ["stack_fused_step", "model_graph", "pdl", "stack_portion"])
def test_variants_agree(pkg, ck, tmp_path, tune):
    """The unfused step, eager steps, plain launches, prompts cut inside: the same logits."""
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
