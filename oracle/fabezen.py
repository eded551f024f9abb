"""Plain float64 statement of the Fabezen design: one function per mechanism, one token or one sequence at a time.

Written from the design's equations for the tests; it shares no code with the product and favours the obvious form over speed
(the delta rule walks token by token, attention forms every score).  Weights are a dict of numpy arrays under the names a model
folder uses ('l0.mix.q', ...), the configuration is the parsed config.json as a dict.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token of a sequence that starts with tokens[0]."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows[:len(tokens)]


def embedding(tokens, w, cfg):
    e = cfg["embedding"]
    x = w["embed"][np.asarray(tokens)] * e["scale"]
    b = e.get("bigram")
    if b is None:
        return x
    return x + w["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]


def short_conv(x, taps):
    """x [T, channels], taps [channels, n]: column n - 1 weighs token t, column 0 token t - n + 1; the result goes through silu."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return silu(sum(padded[j:j + len(x)] * taps[:, j] for j in range(n)))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, beta, g, state=None):
    """q, k [T, heads, dim], v [T, heads, vdim], beta [T, heads], g [T, heads, dim] (the decay of each key row).
    Returns (o [T, heads, vdim], final state [heads, dim, vdim])."""
    T, H, dim = q.shape
    s = np.zeros((H, dim, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        s = s * g[t][:, :, None]
        seen = np.einsum("hdv,hd->hv", s, k[t])
        u = beta[t][:, None] * (v[t] - seen)
        s = s + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", s, q[t])
    return o, s


def decay_per_head(h, w, p, mix):
    a = h @ w[p + "a"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(a))
    return np.repeat(g[:, :, None], mix["dim"], axis=2)


def decay_per_channel(h, w, p, mix):
    a = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(len(h), mix["heads"], mix["dim"])
    return np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(a))


def delta_mixer(h, w, p, mix, eps, channelwise):
    T, H, KV, dim, vdim = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, KV, dim)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, KV, dim)
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, H, vdim)
    q, k = unit(q) * dim ** -0.5, unit(k)
    owner = np.arange(H) // (H // KV)
    beta = sigmoid(h @ w[p + "b"].T)
    g = (decay_per_channel if channelwise else decay_per_head)(h, w, p, mix)
    o, _ = delta_rule(q[:, owner], k[:, owner], v, beta, g)
    if channelwise:
        gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    else:
        gate = silu(h @ w[p + "g"].T)
    o = rms_norm(o, w[p + "norm"], eps) * gate.reshape(T, H, vdim)
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def rotate(x, positions, base, dims):
    """The first `dims` entries of the last axis, in neighbouring pairs; x [T, ..., n]."""
    out = x.copy()
    shape = (len(positions),) + (1,) * (x.ndim - 2)
    for i in range(dims // 2):
        a = np.asarray(positions, dtype=np.float64).reshape(shape) * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def windowed_softmax_attention(score, value, size):
    """score [heads, T, T], value [T, heads, vdim]; a query's own position and the size - 1 before it are visible."""
    T = score.shape[1]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    s = np.where((i >= j) & (i - j < size), score, -np.inf)
    s = np.exp(s - s.max(axis=-1, keepdims=True))
    s /= s.sum(axis=-1, keepdims=True)
    return np.einsum("hij,jhv->ihv", s, value)


def latent_attention_mixer(h, w, p, mix, eps):
    T, H, dim, rd, vdim, rank = len(h), mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    pos = np.arange(T)
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, dim + rd)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    k_rot = rotate(down[:, rank:], pos, mix["rot"]["base"], mix["rot"]["dims"])
    q_rot = rotate(q[:, :, dim:], pos, mix["rot"]["base"], mix["rot"]["dims"])
    k = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vdim)
    score = (np.einsum("ihd,jhd->hij", q[:, :, :dim], k) + np.einsum("ihd,jd->hij", q_rot, k_rot)) * mix["scale"]
    o = windowed_softmax_attention(score, v, mix["mask"]["size"])
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(tokens, w, cfg, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out, when a list, receives the residual stream after every layer."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embedding(tokens, w, cfg)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention_mixer(h, w, p + "mix.", layer["mixer"], eps)
        else:
            y = delta_mixer(h, w, p + "mix.", layer["mixer"], eps, layer["type"] == "channel_delta")
        x = x + m * y
        if layer.get("mlp"):
            x = x + m * dense(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
