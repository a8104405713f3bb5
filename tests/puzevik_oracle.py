"""Plain, slow restatement of the Puzevik layer stack in numpy: one function per mechanism, whole sequences from position 0, token after
token wherever the mechanism is a recurrence.  `real` (numpy float64 by default) is the arithmetic type.  Nothing here is shared with
the library."""
from __future__ import annotations

import json
import struct

import numpy as np


def read_model(folder, real=np.float64):
    """(config, {name: array}) of a folder with config.json and a bfloat16 model.safetensors."""
    with open(f"{folder}/config.json") as f:
        cfg = json.load(f)
    with open(f"{folder}/model.safetensors", "rb") as f:
        blob = f.read()
    n = struct.unpack("<Q", blob[:8])[0]
    head = json.loads(blob[8:8 + n])
    data = blob[8 + n:]
    w = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        lo, hi = e["data_offsets"]
        assert e["dtype"] == "BF16", (name, e["dtype"])
        bits = np.frombuffer(data[lo:hi], dtype="<u2").astype(np.uint32) << 16
        w[name] = bits.view(np.float32).reshape(e["shape"]).astype(real)
    return cfg, w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(np.zeros((), z.dtype), z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def rotate(x, pos, dims, base):
    """Half-split rotation of the first `dims` of the last axis; x is [tokens, heads, d], pos [tokens]."""
    half = dims // 2
    i = np.arange(half)
    f = np.power(np.float64(base), -2.0 * i / dims).astype(x.dtype)
    a = pos.astype(x.dtype)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def causal_conv(x, taps_w):
    """Depthwise convolution over time, last tap on the current token, zeros before the start; x [T, C], taps_w [C, taps]."""
    T, C = x.shape
    taps = taps_w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, C), x.dtype), x])
    return sum(pad[j:j + T] * taps_w[:, j] for j in range(taps))


def retention(h, w, mix, eps):
    T = h.shape[0]
    H, d, dv = mix["heads"], mix["dim"], mix["vdim"]
    pos = np.arange(T)
    q = rotate((h @ w["q"].T).reshape(T, H, d), pos, mix["rot"]["dims"], mix["rot"]["base"])
    k = rotate((h @ w["k"].T).reshape(T, H, d), pos, mix["rot"]["dims"], mix["rot"]["base"]) * h.dtype.type(d ** -0.5)
    v = (h @ w["v"].T).reshape(T, H, dv)
    a = np.array(mix["decay"], h.dtype)
    o = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        S = np.zeros((d, dv), h.dtype)
        for t in range(T):
            S = a[n] * S + np.outer(k[t, n], v[t, n])
            o[t, n] = S.T @ q[t, n]
    o = rms(o, eps).reshape(T, H * dv)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def latent_attention(h, w, mix, eps):
    T = h.shape[0]
    H, d, r, dv, rank = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    pos = np.arange(T)
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(T, H, d + r)
    kv = h @ w["dkv"].T
    c = rms(kv[:, :rank], eps) * w["dkv.norm"]
    kr = rotate(kv[:, None, rank:], pos, mix["rot"]["dims"], mix["rot"]["base"])[:, 0]
    qr = rotate(q[..., d:], pos, mix["rot"]["dims"], mix["rot"]["base"])
    k = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    o = np.zeros((T, H, dv), h.dtype)
    hidden = np.triu(np.ones((T, T), bool), 1)
    for n in range(H):
        s = (q[:, n, :d] @ k[:, n].T + qr[:, n] @ kr.T) * h.dtype.type(mix["scale"])
        s[hidden] = -np.inf
        p = np.exp(s - s.max(axis=1, keepdims=True))
        o[:, n] = (p / p.sum(axis=1, keepdims=True)) @ v[:, n]
    return o.reshape(T, H * dv) @ w["o"].T


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + x.dtype.type(1e-6))


def channel_delta(h, w, mix, eps):
    T = h.shape[0]
    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).reshape(T, G, d)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).reshape(T, G, d)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).reshape(T, H, dv)
    q, k = unit(q) * h.dtype.type(d ** -0.5), unit(k)
    beta = sigmoid(h @ w["b"].T)
    raw = ((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(T, H, d)
    g = np.exp(-np.exp(w["A_log"])[None, :, None] * softplus(raw))
    o = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        m = n // (H // G)
        S = np.zeros((d, dv), h.dtype)
        for t in range(T):
            S = g[t, n][:, None] * S
            u = beta[t, n] * (v[t, n] - S.T @ k[t, m])
            S = S + np.outer(k[t, m], u)
            o[t, n] = S.T @ q[t, m]
    o = rms(o, eps) * w["norm"]
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, dv)
    return (o * gate).reshape(T, H * dv) @ w["o"].T


def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"retention": retention, "latent_attention": latent_attention, "channel_delta": channel_delta}


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [tokens, vocab] of one sequence; layers_out (a list) receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    x = x * x.dtype.type(cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        h = rms(x, eps) * w[f"l{i}.norm1"]
        delta = MIXERS[layer["type"]](h, sub(w, f"l{i}.mix."), layer["mixer"], eps)
        if layer.get("mlp"):
            assert layer["mlp"]["kind"] == "dense"
            delta = delta + feed_forward(h, sub(w, f"l{i}.mlp."))
        x = x + delta
        if layers_out is not None:
            layers_out.append(x.copy())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
