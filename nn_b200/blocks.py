"""Building blocks of decoders with a 32-bit residual stream: products, and the layers' mixers and feed-forwards.

A block is made once from its weights and sizes and may serve several layers; what a layer carries from step to step is reserved
in a SequenceStates per layer.  A pass works on ``m = batch * steps`` rows; every product leaves a ``Source`` that the row kernel
behind it reads (split-K partial sums in the device object's scratch block for bf16, a matrix for float32).  The scratch block
holds one product at a time, so whatever is needed past the next product lies in a buffer of its own; projections that share
their input are one product.

Two number formats: bf16 (weights, activations between products and cached rows are bf16, sums 32-bit) and float32 (everything
32-bit).  Norms, angles, attention scores and weights, decays, step sizes, recurrent states and the residual stream are 32-bit in
both.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import numpy as np

from . import native as N
from .device import Device, _SIZE
from .state import Reservation, SequenceStates


# Passes of more rows than this (a prompt's portion) are bound by bytes, not by the number of launches.
FEW_ROWS = 256


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class Source:
    """A product as the next row kernel reads it (ns_b200.h)."""
    ptr: int
    splits: int
    dtype: int
    ld: int

    @property
    def args(self):
        return C.c_uint64(self.ptr), self.splits, self.dtype, self.ld


class Workspace:
    """Buffers shared by the blocks of a model: every block names what it needs per row, then they are allocated once."""

    def __init__(self, dev: Device, dtype: int):
        self.dev, self.dtype = dev, dtype
        self._need: dict[str, tuple[int, set]] = {}
        self._buf: dict[str, object] = {}

    def need(self, name: str, per_row: int, dtype: int | None = None, extra: int = 0) -> None:
        """per_row elements for each of a pass's rows, and for `extra` more rows per sequence."""
        dtype = self.dtype if dtype is None else dtype
        have = self._need.setdefault(name, (dtype, set()))
        assert have[0] == dtype
        have[1].add((per_row, extra))

    def allocate(self, rows: int, batch: int) -> None:
        self.rows = rows
        for name, (dtype, sizes) in self._need.items():
            self._buf[name] = self.dev.zeros(max(per_row * (rows + batch * extra) for per_row, extra in sizes), dtype)

    def __getitem__(self, name: str) -> int:
        return self._buf[name].ptr


@dataclass
class Step:
    """One pass: `batch` sequences in `slots` (device address of their slot numbers), `steps` new tokens each."""
    batch: int
    steps: int
    slots: int
    pos: int
    longest: int = 0         # the most tokens one of the sequences has behind it
    launches: int = 0

    @property
    def m(self) -> int:
        return self.batch * self.steps


def f32(a: np.ndarray) -> np.ndarray:
    """A weight as float32 (bf16 bits are widened)."""
    a = np.asarray(a)
    if a.dtype == np.uint16:
        return (a.astype(np.uint32) << 16).view(np.float32)
    return np.ascontiguousarray(a, dtype=np.float32)


def bf16_bits(a: np.ndarray) -> np.ndarray:
    """A weight as bf16 bits (float32 is rounded to nearest even)."""
    a = np.asarray(a)
    if a.dtype == np.uint16:
        return a
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class Product:
    """y = x . W^T for weights [n, k] given as bf16 bits (uint16) or float32; several matrices with the same input become one
    product, their outputs side by side at ``cols``.  Input rows are ``k_ld`` long, output rows ``ld``.  wide: the product is also
    asked for as ``wide``."""

    def __init__(self, ws: Workspace, *weights: np.ndarray, wide: bool = False):
        self.dev, self.ws = ws.dev, ws
        k = weights[0].shape[1]
        self.cols, at = [], 0
        for w in weights:
            assert w.shape[1] == k
            self.cols.append(at)
            at += w.shape[0]
        self.k, self.n = k, at
        self.k_ld, self.ld = pad8(k), pad8(at)
        self.handle = None
        if ws.dtype == N.NS_BF16:
            w = np.ascontiguousarray(np.concatenate([bf16_bits(x) for x in weights]))
            h = C.c_void_p()
            N.call("ns_linear_create_bf16", self.dev.handle, self.n, k, w.ctypes.data_as(C.c_void_p), C.byref(h))
            self.handle = h
            ptr = C.c_uint64()
            N.call("ns_linear_info", h, None, None, None, C.byref(ptr), None, None)
            self.w_ptr = ptr.value
            if wide:
                ws.need("wide", self.ld)
        else:
            w = np.zeros((self.ld, self.k_ld), np.float32)
            w[:at, :k] = np.concatenate([f32(x) for x in weights])
            self.w = self.dev.from_numpy(w)
            self.w_ptr = self.w.ptr
            ws.need("product", self.ld, N.NS_F32)

    def __call__(self, x: int, step: Step) -> Source:
        m = step.m
        if self.handle is None:
            self.into(x, m, self.ws["product"])
            step.launches += 1
            return Source(self.ws["product"], 1, N.NS_F32, self.ld)
        ptr, splits = C.c_uint64(), C.c_int()
        N.call("ns_linear_forward_partial", self.dev.handle, self.handle, C.c_uint64(x), m, C.byref(ptr), C.byref(splits))
        step.launches += 1
        return Source(ptr.value, splits.value, N.NS_F32, self.ld)

    def wide(self, x: int, step: Step) -> Source:
        """The same for outputs that may be bf16: a pass of many rows (bf16 models) leaves one bf16 matrix in the workspace's "wide"
        buffer, half the bytes of float sums; it stays until the next wide product."""
        if self.handle is None or step.m <= FEW_ROWS:
            return self(x, step)
        self.into(x, step.m, self.ws["wide"], N.NS_BF16)
        step.launches += 1
        return Source(self.ws["wide"], 1, N.NS_BF16, self.ld)

    def into(self, x: int, m: int, y: int, dtype: int = N.NS_F32) -> None:
        """Output [m, ld] at y (bf16 layers: of either type)."""
        if self.handle is None:
            assert dtype == N.NS_F32
            N.call("ns_f32_batched_matmul", self.dev.handle, C.c_uint64(x), C.c_uint64(self.w_ptr), C.c_uint64(y), 1, m, self.ld, self.k_ld, 0, 1,
                   C.c_float(0.0))
        else:
            N.call("ns_linear_forward", self.dev.handle, self.handle, C.c_uint64(x), C.c_uint64(0), m, N.EPI_NONE, C.c_uint64(0), N.NS_F32, dtype,
                   C.c_uint64(y))

    def close(self) -> None:
        if self.handle is not None:
            N.call("ns_linear_destroy", self.handle)
            self.handle = None


def rms_rows(step: Step, dev: Device, x: int, source: Source | None, alpha: float, x_out: int, weight, eps: float, cols: int, y: int, dtype: int, y_ld: int,
             rows: int | None = None, row_map: int = 0) -> None:
    """x_out = x + alpha * source; y = RMS norm of it (weight None: no norm)."""
    s = source or Source(0, 1, N.NS_F32, 0)
    N.call("ns_rms_rows", dev.handle, C.c_uint64(x), *s.args, C.c_float(alpha), C.c_uint64(x_out), C.c_uint64(weight.ptr if weight else 0), C.c_float(eps),
           C.c_uint64(row_map), C.c_int64(step.m), C.c_int64(rows if rows is not None else step.m), cols, dtype, C.c_uint64(y), y_ld)
    step.launches += 1


def rms_post_rows(step: Step, dev: Device, x: int, source: Source, post, plus: int, x_out: int, weight, eps: float, cols: int, y: int, dtype: int, y_ld: int) -> None:
    """x_out = x + RMS norm of the source with `post` (+ the rows at `plus`); y = RMS norm of it (weight None: no norm)."""
    N.call("ns_rms_post_rows", dev.handle, C.c_uint64(x), *source.args, C.c_uint64(post.ptr), C.c_uint64(plus), C.c_uint64(x_out),
           C.c_uint64(weight.ptr if weight else 0), C.c_float(eps), C.c_int64(step.m), cols, dtype, C.c_uint64(y), y_ld)
    step.launches += 1


class DenseGlu:
    """W_down (act(W_gate h) * (W_up h)), act gelu (tanh form) or relu."""

    def __init__(self, ws: Workspace, gate, up, down, act: int = N.ACT_GELU):
        self.dev, self.ws, self.act = ws.dev, ws, act
        self.ff = gate.shape[0]
        self.gate_up = Product(ws, gate, up, wide=True)
        self.down = Product(ws, down)
        ws.need("act", self.down.k_ld)

    def forward(self, h: int, step: Step) -> Source:
        s = self.gate_up.wide(h, step)
        act = self.ws["act"]
        N.call("ns_glu_rows", self.dev.handle, *s.args, C.c_int64(step.m), self.ff, self.act, self.ws.dtype, C.c_uint64(act),
               self.down.k_ld)
        step.launches += 1
        return self.down(act, step)

    def close(self) -> None:
        self.gate_up.close()
        self.down.close()


class DeltaMixer:
    """Gated delta rule with short convolutions (ns_delta.cu, ns_delta_chunk.cu).

    weights: q, k, v, b, o, their convolutions q_conv, k_conv, v_conv, A_log, dt_bias, norm, and either a, g (one decay per head,
    read-out gated by silu) or a1, a2, g1, g2 (a decay for every key channel of a head through a low-rank pair, read-out gated by the
    sigmoid of another).

    A few tokens go through the recurrence one by one, a prompt's portion (bf16 models) in chunks on the tensor cores; the choice
    depends on the portion's length alone."""

    CHUNK_STEPS = 24         # portions of at least this many tokens are chunked

    def __init__(self, ws: Workspace, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float, w: dict):
        assert heads % kv_heads == 0
        self.dev, self.ws, self.eps = ws.dev, ws, eps
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = heads, kv_heads, dim, vdim, taps
        self.channelwise = "a1" in w
        self.chunks = ws.dtype == N.NS_BF16 and dim <= 128 and dim % 4 == 0 and vdim % 2 == 0
        dev = self.dev
        up = lambda a: dev.from_numpy(f32(a).reshape(-1))
        self.conv = [up(w[n + "_conv"]) for n in "qkv"]
        self.a_log, self.dt_bias, self.norm = up(w["A_log"]), up(w["dt_bias"]), up(w["norm"])
        self.channels = [kv_heads * dim, kv_heads * dim, heads * vdim]
        if self.channelwise:
            r1, r2 = w["a1"].shape[0], w["g1"].shape[0]
            names = ("b", "a1", "g1")
            self.inputs = Product(ws, w["q"], w["k"], w["v"], *(w[n] for n in names), wide=True)
            # both low-rank pairs end in one product: block-diagonal, the outputs side by side
            second = np.zeros((heads * dim + heads * vdim, r1 + r2), np.float32)
            second[:heads * dim, :r1] = f32(w["a2"])
            second[heads * dim:, r1:] = f32(w["g2"])
            self.second = Product(ws, second)
            self.low_rank = r1 + r2
            ws.need("low_rank", self.second.k_ld)
            ws.need("beta", pad8(heads), N.NS_F32)
        else:
            names = ("b", "a")
            self.inputs = Product(ws, w["q"], w["k"], w["v"], w["b"], w["a"], w["g"], wide=True)
            self.second = None
        # what enters the recurrence besides q, k, v stays float where the rest of a long pass is bf16: its own small product
        self.small = Product(ws, *(w[n] for n in names)) if ws.dtype == N.NS_BF16 else None
        self.out = Product(ws, w["o"])
        for n, c in zip("qkv", self.channels):
            ws.need("conv_" + n, c, N.NS_F32)
        ws.need("read", heads * vdim, N.NS_F32)
        ws.need("mixed", self.out.k_ld)

    def reserve(self, states: SequenceStates, max_steps: int) -> dict:
        return {"hist": [states.reserve(self.taps * c, N.NS_F32, True) for c in self.channels],
                "state": states.reserve(self.heads * self.dim * self.vdim, N.NS_F32, True)}

    def forward(self, h: int, cache: dict, step: Step) -> Source:
        ws, hd, H = self.ws, self.dev.handle, self.heads
        s = wide = self.inputs.wide(h, step)
        cols = list(self.inputs.cols)
        fields, scales = [], []
        for i, n in enumerate("qkv"):
            heads, width = (H, self.vdim) if n == "v" else (self.kv_heads, self.dim)
            fields += [cols[i], heads, width, self.taps, int(n != "v"), self.conv[i].ptr, cache["hist"][i].ptr, ws["conv_" + n], self.channels[i]]
            scales.append(self.dim ** -0.5 if n == "q" else 1.0)
        N.call("ns_short_conv", hd, *s.args, 3, (C.c_int64 * 27)(*fields), (C.c_float * 3)(*scales), C.c_int64(cache["hist"][0].stride),
               C.c_uint64(step.slots), C.c_uint64(step.pos), step.batch, step.steps, N.NS_F32)
        step.launches += 1
        if wide.dtype == N.NS_BF16:
            s = self.small(h, step)
            cols[3:3 + len(self.small.cols)] = self.small.cols
        if self.channelwise:
            m = step.m
            N.call("ns_copy_cols", hd, *s.args, cols[3], C.c_int64(m), H, N.NS_F32, C.c_uint64(ws["beta"]), pad8(H))
            N.call("ns_copy_cols", hd, *s.args, cols[4], C.c_int64(m), self.low_rank, ws.dtype, C.c_uint64(ws["low_rank"]), self.second.k_ld)
            step.launches += 2
            beta, beta_col = Source(ws["beta"], 1, N.NS_F32, pad8(H)), 0
            s = wide = self.second(ws["low_rank"], step)
            a_col, gate_col, act = 0, H * self.dim, N.ACT_SIGMOID
        else:
            beta, beta_col = s, cols[3]
            a_col, gate_col, act = cols[4], cols[5], N.ACT_SILU
        state: Reservation = cache["state"]
        u = C.c_uint64
        N.call("ns_delta_chunked" if self.chunks and step.steps >= self.CHUNK_STEPS else "ns_delta_recurrent", hd, u(ws["conv_q"]), self.channels[0], u(ws["conv_k"]), self.channels[1], u(ws["conv_v"]), self.channels[2],
               u(s.ptr), s.splits, s.ld, a_col, u(beta.ptr), beta.splits, beta.ld, beta_col, u(self.a_log.ptr), u(self.dt_bias.ptr), int(self.channelwise),
               u(state.ptr), C.c_int64(state.stride), u(step.slots), step.batch, step.steps, H, self.kv_heads, self.dim, self.vdim, u(ws["read"]), H * self.vdim)
        N.call("ns_gated_norm", hd, u(ws["read"]), H * self.vdim, *wide.args, gate_col, act, u(self.norm.ptr), C.c_float(self.eps), C.c_int64(step.m), H, self.vdim,
               ws.dtype, u(ws["mixed"]), self.out.k_ld)
        step.launches += 2
        return self.out(ws["mixed"], step)

    def close(self) -> None:
        for p in (self.inputs, self.second, self.small, self.out):
            if p is not None:
                p.close()


class LightningMixer:
    """Linear attention with a fixed decay per head (ns_lightning.cu): q, k, v through silu, the heads' outputs normalised together, times a
    sigmoid gate per channel.

    weights: q, k, v, g, o, norm.

    A few tokens go through the recurrence one by one, a prompt's portion (bf16 models) in chunks on the tensor cores; the choice
    depends on the portion's length alone."""

    CHUNK_STEPS = 16         # portions of at least this many tokens are chunked

    def __init__(self, ws: Workspace, heads: int, dim: int, vdim: int, decay, eps: float, w: dict):
        decay = np.asarray(decay, np.float64)
        if decay.shape != (heads,) or not np.all(decay >= 0.0):
            raise ValueError(f"{heads} heads need {heads} decays that are not negative")
        self.dev, self.ws, self.eps = ws.dev, ws, eps
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.chunks = ws.dtype == N.NS_BF16 and dim <= 128
        with np.errstate(divide="ignore"):
            log2 = np.maximum(np.log2(decay), -1e4)          # a decay of 0: powers of it are 0 (and its 0th power 1)
        up = lambda a: self.dev.from_numpy(np.ascontiguousarray(a, np.float32).reshape(-1))
        self.decay, self.decay_log2, self.norm = up(decay), up(log2), up(f32(w["norm"]))
        self.inputs = Product(ws, w["q"], w["k"], w["v"], w["g"], wide=True)
        self.out = Product(ws, w["o"])
        ws.need("read", heads * vdim, N.NS_F32)
        ws.need("mixed", self.out.k_ld)

    def reserve(self, states: SequenceStates, max_steps: int) -> Reservation:
        return states.reserve(self.heads * self.dim * self.vdim, N.NS_F32, True)

    def forward(self, h: int, cache: Reservation, step: Step) -> Source:
        ws, hd, u = self.ws, self.dev.handle, C.c_uint64
        s, n = self.inputs.wide(h, step), self.heads * self.vdim
        q, k, v, g = self.inputs.cols
        args = (hd, *s.args, q, k, v, u(self.decay.ptr), u(self.decay_log2.ptr), u(cache.ptr), C.c_int64(cache.stride), u(step.slots), step.batch, step.steps, self.heads,
                self.dim, self.vdim, u(ws["read"]), n)
        if self.chunks and step.steps >= self.CHUNK_STEPS:
            N.call("ns_lightning_chunked", *args, 0)
        else:
            N.call("ns_lightning_recurrent", *args)
        N.call("ns_gated_norm", hd, u(ws["read"]), n, *s.args, g, N.ACT_SIGMOID, u(self.norm.ptr), C.c_float(self.eps), C.c_int64(step.m), 1, n, ws.dtype,
               u(ws["mixed"]), self.out.k_ld)
        step.launches += 2
        return self.out(ws["mixed"], step)

    def close(self) -> None:
        self.inputs.close()
        self.out.close()


class WindowAttentionMixer:
    """Grouped-query attention over a sliding window (ns_window.cu; a prompt's portion: ns_attention_prefill.cu).

    weights: q, k, v, o, and, each optional, q_norm and k_norm (RMS norm over all heads together), sink (a learned term of every
    head's softmax sum), g (a sigmoid gate per head on its output).

    Portions of a few tokens and longer ones take different kernels; the choice depends on the portion's length alone."""

    PREFILL_STEPS = 32       # portions of at least this many tokens are a prompt's
    RING_ROWS = 128          # ring lengths are multiples of this

    def __init__(self, ws: Workspace, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, eps: float, w: dict):
        if heads % kv_heads != 0:
            raise ValueError(f"{heads} heads do not divide over {kv_heads} key/value heads")
        if window < 1:
            raise ValueError(f"a window of {window} positions")
        self.dev, self.ws, self.eps, self.window = ws.dev, ws, eps, window
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.k_ld, self.v_ld = pad8(dim), pad8(vdim)
        bf16 = ws.dtype == N.NS_BF16
        self.tiles = bf16 and self.k_ld <= 256 and self.v_ld <= 256
        self.prefill = bf16 and self.k_ld <= 128 and self.v_ld <= 128 and vdim % 8 == 0
        up = lambda name, sign=1.0: self.dev.from_numpy(f32(w[name]).reshape(-1) * np.float32(sign)) if w.get(name) is not None else None
        # the kernels take a positive scale: the queries carry its sign
        sign = 1.0 if scale > 0.0 else (-1.0 if scale < 0.0 else 0.0)
        self.scale = abs(scale) or 1.0
        q = w["q"]
        if sign != 1.0 and w.get("q_norm") is None:
            q, sign = f32(q) * np.float32(sign), 1.0
        self.q_norm, self.k_norm, self.sink = up("q_norm", sign), up("k_norm"), up("sink")
        self.gated = w.get("g") is not None
        self.inputs = Product(ws, q, w["k"], w["v"], *((w["g"],) if self.gated else ()), wide=True)
        self.out = Product(ws, w["o"])
        ws.need("q_heads", heads * self.k_ld)
        if self.gated:
            ws.need("gate", heads, N.NS_F32)
        # the columns that pad a row of the output product's input are never written: a buffer of this width's own keeps them zero
        self.mixed = f"mixed_{heads * vdim}"
        ws.need(self.mixed, self.out.k_ld)

    def reserve(self, states: SequenceStates, max_steps: int) -> dict:
        """The rings are cleared when a sequence opens: the kernels read whole tiles of rows and mask by position, so every row has to be finite."""
        n = -(-(self.window - 1 + max_steps) // self.RING_ROWS) * self.RING_ROWS
        return {"k": states.reserve(self.kv_heads * n * self.k_ld, self.ws.dtype, True), "v": states.reserve(self.kv_heads * n * self.v_ld, self.ws.dtype, True),
                "len": n, "slots": states.slots}

    def forward(self, h: int, cache: dict, step: Step) -> Source:
        ws, hd, u, i64 = self.ws, self.dev.handle, C.c_uint64, C.c_int64
        k, v = cache["k"], cache["v"]
        rings = (u(k.ptr), u(v.ptr), i64(k.stride), i64(v.stride))
        lens = (cache["len"], self.k_ld, self.v_ld)
        at = (u(step.slots), u(step.pos), step.batch, step.steps)
        s, cols = self.inputs.wide(h, step), self.inputs.cols
        q, gate, mixed = u(ws["q_heads"]), u(ws["gate"] if self.gated else 0), u(ws[self.mixed])
        ptr = lambda a: u(a.ptr if a is not None else 0)
        N.call("ns_window_append", hd, *s.args, cols[0], cols[1], cols[2], cols[3] if self.gated else 0, self.heads, self.kv_heads, self.dim, self.vdim,
               ptr(self.q_norm), ptr(self.k_norm), C.c_float(self.eps), *at, ws.dtype, q, gate, *rings, *lens)
        rest = (ptr(self.sink), gate, *at, self.heads, self.kv_heads, self.dim, self.vdim, self.window, C.c_float(self.scale), mixed, i64(self.out.k_ld))
        if self.prefill and step.steps >= self.PREFILL_STEPS:
            N.call("ns_window_prefill", hd, q, *rings, cache["slots"], *lens, *rest)
        elif self.tiles:
            N.call("ns_window_decode", hd, q, *rings, *lens, *rest)
        else:
            N.call("ns_window_attend", hd, ws.dtype, q, *rings, *lens, *rest)
        step.launches += 2
        return self.out(ws[self.mixed], step)

    def close(self) -> None:
        self.inputs.close()
        self.out.close()


class LatentAttentionMixer:
    """Attention over cached latents with a sliding window (ns_latent.cu, ns_latent_tc.cu).

    weights: dq, dq_norm, uq, dkv, dkv_norm, uk, uv, o.

    Two forms of the same attention.  Few tokens: the unrotated query goes through its head's key matrix, attention runs over the
    cached latents as one key / value head shared by all, the weighted latent goes through the head's value matrix.  A prompt's
    portion (bf16): keys and values of the window are expanded by one product and attention runs per head.  The choice depends on
    the portion's length alone, so a sequence goes through the same arithmetic in any batch."""

    EXPAND_STEPS = 32        # portions of at least this many tokens are expanded

    def __init__(self, ws: Workspace, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, window: int, rot_base: float,
                 rot_dims: int, eps: float, w: dict):
        self.dev, self.ws, self.eps, self.scale, self.window = ws.dev, ws, eps, scale, window
        self.heads, self.dim, self.rot_dim, self.vdim, self.q_rank, self.kv_rank, self.rot_dims = heads, dim, rot_dim, vdim, q_rank, kv_rank, rot_dims
        dev = self.dev
        self.width = kv_rank + rot_dim
        self.q_norm, self.kv_norm = dev.from_numpy(f32(w["dq_norm"])), dev.from_numpy(f32(w["dkv_norm"]))
        i = np.arange(max(rot_dims // 2, 1), dtype=np.float64)
        self.freq = dev.from_numpy((float(rot_base) ** (-2.0 * i / max(rot_dims, 1))).astype(np.float32))
        self.down = Product(ws, w["dq"], w["dkv"])
        self.uq = Product(ws, w["uq"], wide=True)
        # its input rows are whole cached rows: the columns of the rotated part are zero
        self.kv = Product(ws, *(np.pad(w[n], ((0, 0), (0, rot_dim))) for n in ("uk", "uv")))
        self.out = Product(ws, w["o"])
        self.expands = ws.dtype == N.NS_BF16 and vdim <= 256 and dim + rot_dim <= 256
        ws.need("cq", self.uq.k_ld)
        ws.need("plain", heads * dim)
        ws.need("carried", heads * self.width)
        ws.need("weighted", heads * kv_rank)
        if self.expands:
            ws.need("q_heads", heads * (dim + rot_dim))
            ws.need("keys", pad8(self.width), extra=window - 1)
            ws.need("kv", self.kv.ld, extra=window - 1)
        # the columns that pad a row of the output product's input are never written: a buffer of this width's own keeps them zero
        self.mixed = f"mixed_{heads * vdim}"
        ws.need(self.mixed, self.out.k_ld)

    def reserve(self, states: SequenceStates, max_steps: int) -> dict:
        ring = self.window - 1 + max_steps
        return {"ring": states.reserve(ring * pad8(self.width), self.ws.dtype, False), "len": ring}

    def forward(self, h: int, cache: dict, step: Step) -> Source:
        ws, hd, H, R, W, dt = self.ws, self.dev.handle, self.heads, self.kv_rank, self.width, self.ws.dtype
        u, i64 = C.c_uint64, C.c_int64
        ring: Reservation = cache["ring"]
        at = (u(step.slots), u(step.pos), step.batch, step.steps)
        ring_args = (u(ring.ptr), i64(ring.stride), cache["len"], pad8(W))
        s = self.down(h, step)
        N.call("ns_latent_append", hd, *s.args, self.q_rank, R, self.rot_dim, self.rot_dims, u(self.q_norm.ptr), u(self.kv_norm.ptr), C.c_float(self.eps),
               u(self.freq.ptr), *at, dt, u(ws["cq"]), self.uq.k_ld, *ring_args)
        s = self.uq.wide(ws["cq"], step)
        rotate = (hd, *s.args, H, self.dim, self.rot_dim, self.rot_dims, u(self.freq.ptr), *at)
        mixed = ws[self.mixed]
        if self.expands and step.steps >= self.EXPAND_STEPS:
            qw = self.dim + self.rot_dim
            q, past = ws["q_heads"], min(self.window - 1, step.longest)
            N.call("ns_rotate_heads", *rotate, dt, u(q), i64(H * qw), qw, dt, u(q + 2 * self.dim), i64(H * qw), qw)
            N.call("ns_latent_gather", hd, *ring_args, past, u(step.slots), u(step.pos), step.batch, past + step.steps, u(ws["keys"]))
            self.kv.into(ws["keys"], step.batch * (past + step.steps), ws["kv"], dt)
            N.call("ns_latent_prefill", hd, u(q), i64(H * qw), u(ws["kv"]), i64(self.kv.ld), u(ws["keys"]), i64(pad8(W)), R, *at, H, self.dim, self.rot_dim,
                   self.vdim, past, self.window, C.c_float(self.scale), u(mixed), i64(self.out.k_ld))
            step.launches += 5
            return self.out(mixed, step)
        el, carried, k_ld = _SIZE[dt], ws["carried"], self.kv.k_ld
        N.call("ns_rotate_heads", *rotate, dt, u(ws["plain"]), i64(H * self.dim), self.dim, dt, u(carried + el * R), i64(H * W), W)
        # the unrotated query through the head's key matrix: its score with a latent is then one dot product
        N.call("ns_head_matmul", hd, dt, u(ws["plain"]), i64(H * self.dim), self.dim, dt, u(self.kv.w_ptr), i64(self.dim * k_ld), i64(k_ld), i64(1), dt,
               u(carried), i64(H * W), W, step.m, H, self.dim, R)
        attend = (*ring_args, R, W, self.window, C.c_float(self.scale), *at, H, u(ws["weighted"]))
        if dt == N.NS_BF16:
            N.call("ns_latent_decode", hd, u(carried), *attend)
        else:
            N.call("ns_latent_attend", hd, u(carried), dt, *attend)
        N.call("ns_head_matmul", hd, dt, u(ws["weighted"]), i64(H * R), R, dt, u(self.kv.w_ptr + el * H * self.dim * k_ld), i64(self.vdim * k_ld), i64(1), i64(k_ld),
               dt, u(mixed), i64(self.out.k_ld), self.vdim, step.m, H, R, self.vdim)
        step.launches += 5
        return self.out(mixed, step)

    def close(self) -> None:
        for p in (self.down, self.uq, self.kv, self.out):
            p.close()
