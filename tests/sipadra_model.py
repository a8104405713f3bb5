"""Small Sipadra models for the tests: the configurations the cases use and random weights for them."""
from __future__ import annotations

import numpy as np

from puzevik_model import bf16_round, layer  # noqa: F401  (layer: type, mixer, feed-forward units)


def yarn(factor=3.0, original=48, fast=6.0, slow=0.5):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def left(heads=6, kv_heads=2, dim=24, vdim=20, dims=16, base=900.0, scaling="yarn", size=23, scale=0.3):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = yarn() if scaling == "yarn" else scaling
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rot, "scale": scale}


def right(heads=3, dim=20, vdim=28, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.6, 0.93, 0.999][:heads] + [0.97] * (heads - 3)}


def parallel(left_arm=None, right_arm=None, left_scale=0.7, right_scale=1.3):
    return {"left": left_arm or left(), "right": right_arm or right(), "left_scale": left_scale, "right_scale": right_scale}


def wkv(heads=3, dim=20):
    return {"heads": heads, "dim": dim}


def config(layers, width=104, vocab=149, eps=3e-4, cap=6.0):
    return {"architecture": "Sipadra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


def weights(cfg, seed, rank=12, w0=(-4.0, 0.5)):
    """Random tensors; w0 is the range of the log rates of wkv's decays (low: the state remembers far back)."""
    rng = np.random.default_rng(seed)
    D, w = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.normal(0, gain / np.sqrt(cols), (rows, cols))

    def vec(name, n):
        w[name] = 1.0 + 0.3 * rng.normal(size=n)

    w["embed"] = rng.normal(0, 1.0, (cfg["vocab"], D))
    vec("final.norm", D)
    w["final.norm"] *= 3.0 / np.sqrt(D)                     # logits of a few units: inside the cap's bend, not flat on it
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        vec(f"l{i}.norm1", D)
        if L["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                w[p + "mu." + s] = rng.uniform(0, 1, D)
            for s in "rkvg":
                mat(p + s, n, D)
            mat(p + "w1", rank, D)
            mat(p + "w2", n, rank)
            w[p + "w0"] = rng.uniform(*w0, n)
            w[p + "u"] = rng.normal(0, 1.0, (m["heads"], m["dim"]))
            vec(p + "norm", n)
            mat(p + "o", D, n)
        else:
            a, b = m["left"], m["right"]
            mat(p + "left.q", a["heads"] * a["dim"], D)
            mat(p + "left.k", a["kv_heads"] * a["dim"], D)
            mat(p + "left.v", a["kv_heads"] * a["vdim"], D)
            mat(p + "left.o", D, a["heads"] * a["vdim"], 1.5)
            mat(p + "right.q", b["heads"] * b["dim"], D)
            mat(p + "right.k", b["heads"] * b["dim"], D)
            mat(p + "right.v", b["heads"] * b["vdim"], D)
            mat(p + "right.g", b["heads"] * b["vdim"], D)
            vec(p + "right.norm", b["heads"] * b["vdim"])
            mat(p + "right.o", D, b["heads"] * b["vdim"], 1.5)
        if L["mlp"]:
            vec(f"l{i}.norm2", D)
            mat(f"l{i}.mlp.gate", L["mlp"]["ff"], D)
            mat(f"l{i}.mlp.up", L["mlp"]["ff"], D)
            mat(f"l{i}.mlp.down", D, L["mlp"]["ff"])
    return {k: bf16_round(v) for k, v in w.items()}
