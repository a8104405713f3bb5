"""Plain, slow restatement of the Sipadra layer stack in numpy: one function per mechanism, whole sequences from position 0, token after
token wherever the mechanism is a recurrence.  The arithmetic type is that of the weights (float64 in the tests).  Nothing here is shared
with the library."""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))


def yarn_frequencies(dims, base, scaling=None):
    """Angular steps per position of the dims / 2 pairs, and the factor on cosines and sines."""
    i = np.arange(dims // 2)
    f = np.power(float(base), -2.0 * i / dims)
    if scaling is None:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def pair_with_turns(turns):                              # which pair makes `turns` turns over the original context
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_with_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_with_turns(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, dims, base, scaling=None):
    """Half-split rotation of the first `dims` of the last axis by the token's index; x is [tokens, heads, d]."""
    f, mul = yarn_frequencies(dims, base, scaling)
    a = np.arange(x.shape[0])[:, None] * f[None, :]
    c, s = (np.cos(a) * mul).astype(x.dtype)[:, None], (np.sin(a) * mul).astype(x.dtype)[:, None]
    half = dims // 2
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def windowed_attention(h, w, mix, eps):
    """Grouped-query softmax attention over the last mask.size positions, query and key of unit mean square after the rotation."""
    T, H, G, d, dv = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    rot = mix["rot"]
    q = rms(rotate((h @ w["q"].T).reshape(T, H, d), rot["dims"], rot["base"], rot.get("scaling")), eps)
    k = rms(rotate((h @ w["k"].T).reshape(T, G, d), rot["dims"], rot["base"], rot.get("scaling")), eps)
    v = (h @ w["v"].T).reshape(T, G, dv)
    o = np.zeros((T, H, dv), h.dtype)
    for t in range(T):
        first = max(0, t - mix["mask"]["size"] + 1)
        for n in range(H):
            m = n // (H // G)
            s = (k[first:t + 1, m] @ q[t, n]) * h.dtype.type(mix["scale"])
            p = np.exp(s - s.max())
            o[t, n] = (p / p.sum()) @ v[first:t + 1, m]
    return o.reshape(T, H * dv) @ w["o"].T


def lightning_attention(h, w, mix, eps):
    T, H, d, dv = len(h), mix["heads"], mix["dim"], mix["vdim"]
    q, k, v = (silu(h @ w[n].T).reshape(T, H, -1) for n in "qkv")
    assert q.shape[2] == k.shape[2] == d and v.shape[2] == dv
    o = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        S = np.zeros((d, dv), h.dtype)
        for t in range(T):
            S = h.dtype.type(mix["decay"][n]) * S + np.outer(k[t, n], v[t, n])
            o[t, n] = S.T @ q[t, n]
    return (rms(o.reshape(T, H * dv), eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def side_by_side(h, w, mix, eps):
    left, right = windowed_attention(h, sub(w, "left."), mix["left"], eps), lightning_attention(h, sub(w, "right."), mix["right"], eps)
    return h.dtype.type(mix["left_scale"]) * left + h.dtype.type(mix["right_scale"]) * right


def token_shift(h, mu):
    """Every token's input leans towards the previous one's, zeros before the first."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv(h, w, mix, eps):
    T, H, d = len(h), mix["heads"], mix["dim"]
    r, k, v = ((token_shift(h, w["mu." + n]) @ w[n].T).reshape(T, H, d) for n in "rkv")
    gate = silu(token_shift(h, w["mu.g"]) @ w["g"].T)
    decay = np.exp(-np.exp(np.tanh(token_shift(h, w["mu.w"]) @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(T, H, d)
    o = np.zeros((T, H, d), h.dtype)
    for n in range(H):
        S = np.zeros((d, d), h.dtype)
        for t in range(T):
            kv = np.outer(k[t, n], v[t, n])
            o[t, n] = (S + w["u"][n][:, None] * kv).T @ r[t, n]
            S = decay[t, n][:, None] * S + kv
    return (rms(o, eps).reshape(T, H * d) * w["norm"] * gate) @ w["o"].T


def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"parallel": side_by_side, "wkv": wkv}


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, layers_out=None):
    """Logits [tokens, vocab] of one sequence; layers_out (a list) receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        x = x + rms(MIXERS[layer["type"]](x, sub(w, f"l{i}.mix."), layer["mixer"], eps), eps) * w[f"l{i}.norm1"]
        if layer.get("mlp"):
            assert layer["mlp"]["kind"] == "dense"
            x = x + rms(feed_forward(x, sub(w, f"l{i}.mlp.")), eps) * w[f"l{i}.norm2"]
        if layers_out is not None:
            layers_out.append(x.copy())
    return softcap((rms(x, eps) * w["final.norm"]) @ w["embed"].T, x.dtype.type(cfg["logit_softcap"]))
