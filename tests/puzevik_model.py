"""Small Puzevik models for the tests: random bfloat16 weights written as a model folder, and the configurations the cases use."""
from __future__ import annotations

import json
import os
import struct

import numpy as np


def bf16_round(a):
    """fp32 numbers rounded to bfloat16 (nearest even), as fp32."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((bits + 0x7FFF + ((bits >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32)


def write_safetensors(path, tensors):
    head, blobs, off = {}, [], 0
    for name, a in tensors.items():
        raw = (bf16_round(a).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


def retention(heads=3, dim=24, vdim=20, dims=16, base=5e4, decay=None):
    decay = decay or [1.0 - 2.0 ** (-2 - 2 * h) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims}}


def latent(heads=3, dim=24, rot_dim=16, vdim=40, q_rank=56, kv_rank=72, scale=0.4, base=3e3):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def delta(heads=4, kv_heads=2, dim=40, vdim=36, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=104, vocab=149, eps=3e-4, scale=7.0):
    return {"architecture": "Puzevik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def weights(cfg, seed, a_rank=12, g_rank=28, a_log=(-3.0, 1.0)):
    """Random tensors; a_log is the range of the delta rule's decay rates (low: the state remembers far back)."""
    rng = np.random.default_rng(seed)
    D, w = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.normal(0, gain / np.sqrt(cols), (rows, cols))

    def vec(name, n):
        w[name] = 1.0 + 0.3 * rng.normal(size=n)

    w["embed"] = rng.normal(0, 1.0 / cfg["embedding"]["scale"], (cfg["vocab"], D))
    mat("head", cfg["vocab"], D)
    vec("final.norm", D)
    for i, L in enumerate(cfg["layers"]):
        p, m, t = f"l{i}.mix.", L["mixer"], L["type"]
        H, dv = m["heads"], m["vdim"]
        vec(f"l{i}.norm1", D)
        mat(p + "o", D, H * dv, 1.5)
        if t == "retention":
            mat(p + "q", H * m["dim"], D)
            mat(p + "k", H * m["dim"], D)
            mat(p + "v", H * dv, D)
            mat(p + "g", H * dv, D)
        elif t == "latent_attention":
            mat(p + "dq", m["q_rank"], D)
            vec(p + "dq.norm", m["q_rank"])
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], D)
            vec(p + "dkv.norm", m["kv_rank"])
            mat(p + "uk", H * m["dim"], m["kv_rank"])
            mat(p + "uv", H * dv, m["kv_rank"])
        else:
            G, d = m["kv_heads"], m["dim"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(p + n, rows, D)
                w[p + n + ".conv"] = rng.normal(0, 0.7, (rows, m["conv"]))
            mat(p + "b", H, D)
            w[p + "A_log"] = rng.uniform(*a_log, H)
            w[p + "dt_bias"] = rng.normal(0, 1.0, H * d)
            vec(p + "norm", dv)
            mat(p + "a1", a_rank, D)
            mat(p + "a2", H * d, a_rank)
            mat(p + "g1", g_rank, D)
            mat(p + "g2", H * dv, g_rank)
        if L["mlp"]:
            mat(f"l{i}.mlp.gate", L["mlp"]["ff"], D)
            mat(f"l{i}.mlp.up", L["mlp"]["ff"], D)
            mat(f"l{i}.mlp.down", D, L["mlp"]["ff"])
    return {k: bf16_round(v) for k, v in w.items()}


def write(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    return str(folder)
