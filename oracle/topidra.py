"""Plain float64 statement of the Topidra design: one function per mechanism, one token or one sequence at a time.

Written from the design's equations for the tests; it shares no code with the product and favours the obvious form over speed
(the linear recurrence walks token by token, attention forms every score).  Weights are a dict of numpy arrays under the names a
model folder uses ('l0.mix.q', ...), the configuration is the parsed config.json as a dict.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def visible(queries, keys, size):
    """[T, T]: key position j is inside the window of `size` positions that ends at query position i."""
    back = np.asarray(queries)[:, None] - np.asarray(keys)[None, :]
    return (back >= 0) & (back < size)


def sink_softmax(score, sink, see):
    """score [heads, T, T], sink [heads]: weights whose sum falls short of 1 by the share of the sink."""
    s = np.where(see, score, -np.inf)
    top = np.maximum(s.max(axis=-1), sink[:, None])
    e = np.exp(s - top[..., None])
    return e / (e.sum(axis=-1) + np.exp(sink[:, None] - top))[..., None]


def attention_mixer(h, w, p, mix, eps):
    T, H, G, dim, vdim = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, dim)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, dim)
    v = (h @ w[p + "v"].T).reshape(T, G, vdim)
    owner = np.arange(H) // (H // G)
    score = np.einsum("ihd,jhd->hij", q, k[:, owner]) * mix["scale"]
    a = sink_softmax(score, w[p + "sink"], visible(np.arange(T), np.arange(T), mix["mask"]["size"]))
    o = np.einsum("hij,jhv->ihv", a, v[:, owner])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def decayed_memory(q, k, v, decay, state=None):
    """q, k [T, heads, dim], v [T, heads, vdim], decay [heads].  Returns (o [T, heads, vdim], final state [heads, dim, vdim])."""
    T, H, dim = q.shape
    s = np.zeros((H, dim, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    decay = np.asarray(decay, dtype=np.float64)
    for t in range(T):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", s, q[t])
    return o, s


def lightning_mixer(h, w, p, mix, eps):
    T, H, dim, vdim = len(h), mix["heads"], mix["dim"], mix["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, dim)
    k = silu(h @ w[p + "k"].T).reshape(T, H, dim)
    v = silu(h @ w[p + "v"].T).reshape(T, H, vdim)
    o, _ = decayed_memory(q, k, v, mix["decay"])
    o = rms_norm(o.reshape(T, H * vdim), w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def dense(h, w, p):
    return (np.maximum(h @ w[p + "gate"].T, 0.0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer(x, w, p, entry, eps):
    mixer = {"attention": attention_mixer, "lightning": lightning_mixer}[entry["type"]]
    x = x + rms_norm(mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", entry["mixer"], eps), w[p + "norm1b"], eps)
    if entry.get("mlp"):
        x = x + rms_norm(dense(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
    return x


def runs(cfg):
    """[(layer, the embedding output is added before it)] in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return out + [(i, False) for i in range(loop["stop"], n)]


def forward(tokens, w, cfg, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out, when a list, receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    embedded = w["embed"][np.asarray(tokens)]
    x = embedded
    for i, again in runs(cfg):
        if again:
            x = x + embedded
        x = layer(x, w, f"l{i}.", cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
