"""The operators behind Topidra's layers, each alone against its plain float64 statement (oracle/topidra.py)."""
import ctypes as C

import numpy as np
import pytest

from nn_b200 import native as N
from nn_b200.blocks import bf16_bits, f32, pad8
from oracle import topidra as F
from tests.test_fabezen_ops import Slots, close, rng_for, split_source

pytestmark = pytest.mark.gpu
u, i64, fl = C.c_uint64, C.c_int64, C.c_float
BITS = {N.NS_F32: lambda a: np.ascontiguousarray(a, np.float32), N.NS_BF16: bf16_bits}


def as_bf16(a):
    return f32(bf16_bits(np.asarray(a, np.float32)))


def filled(dev, count, dtype, value):
    return dev.from_numpy(np.full(count, value, np.float32 if dtype == N.NS_F32 else np.uint16))


def read(s, shape, dtype):
    a = s.download(shape)
    return a if dtype == N.NS_F32 else f32(a)


# ------------------------------------------------------------------------------------------------ rows
@pytest.mark.parametrize("plus", [False, True])
@pytest.mark.parametrize("rows,cols,splits,out", [(5, 64, 3, N.NS_BF16), (3, 61, 1, N.NS_F32), (130, 2048, 2, N.NS_BF16), (4, 1028, 1, N.NS_F32),
                                                  (3, 4096, 1, N.NS_BF16), (2, 8000, 2, N.NS_F32), (2, 9000, 1, N.NS_BF16)])
def test_residual_with_both_norms(dev, rows, cols, splits, out, plus):
    rng = rng_for(1, rows, cols)
    x, s, extra = (rng.standard_normal((rows, cols)).astype(np.float32) for _ in range(3))
    post, w = (1 + 0.1 * rng.standard_normal(cols).astype(np.float32) for _ in range(2))
    s *= 1e-2                                                     # eps matters
    dx, dp, dw, de = dev.from_numpy(x), dev.from_numpy(post.astype(np.float32)), dev.from_numpy(w.astype(np.float32)), dev.from_numpy(extra)
    ds, ld = split_source(dev, s, splits, pad8(cols))
    y_ld = pad8(cols)
    y = filled(dev, rows * y_ld, out, 7)
    N.call("ns_rms_post_rows", dev.handle, u(dx.ptr), u(ds.ptr), splits, N.NS_F32, ld, u(dp.ptr), u(de.ptr if plus else 0), u(dx.ptr), u(dw.ptr), fl(1e-4), i64(rows),
           cols, out, u(y.ptr), y_ld)
    dev.synchronize()
    want = x + F.rms_norm(s.astype(np.float64), post, 1e-4) + (extra if plus else 0.0)
    close(dx.download((rows, cols)), want, 3e-5)
    got = read(y, (rows, y_ld), out)
    close(got[:, :cols], F.rms_norm(want, w, 1e-4), 3e-5 if out == N.NS_F32 else 2e-2)
    assert not got[:, cols:].any()
    # without a second norm only the sum is written
    dx.upload(x)
    N.call("ns_rms_post_rows", dev.handle, u(dx.ptr), u(ds.ptr), splits, N.NS_F32, ld, u(dp.ptr), u(de.ptr if plus else 0), u(dx.ptr), u(0), fl(1e-4), i64(rows), cols, out,
           u(0), 0)
    dev.synchronize()
    close(dx.download((rows, cols)), want, 3e-5)


@pytest.mark.parametrize("rows,ff,splits,out", [(3, 20, 2, N.NS_F32), (7, 37, 1, N.NS_BF16), (300, 512, 1, N.NS_BF16)])
def test_relu_gate(dev, rows, ff, splits, out):
    x = rng_for(4, rows, ff).standard_normal((rows, 2 * ff)) * 2
    s, ld = split_source(dev, x, splits, pad8(2 * ff))
    y_ld = pad8(ff)
    y = filled(dev, rows * y_ld, out, 9)
    N.call("ns_glu_rows", dev.handle, u(s.ptr), splits, N.NS_F32, ld, i64(rows), ff, N.ACT_RELU, out, u(y.ptr), y_ld)
    dev.synchronize()
    got = read(y, (rows, y_ld), out)
    close(got[:, :ff], np.maximum(x[:, :ff], 0) * x[:, ff:], 3e-6 if out == N.NS_F32 else 5e-2)
    assert not got[:, ff:].any()
    with pytest.raises(N.NsError):
        N.call("ns_glu_rows", dev.handle, u(s.ptr), splits, N.NS_F32, ld, i64(rows), ff, N.ACT_SILU, out, u(y.ptr), y_ld)


@pytest.mark.parametrize("out", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("rows,n", [(5, 1), (3, 100), (7, 132), (4, 601), (3, 2052), (2, 4100), (2, 9000)])
def test_gated_norm_of_whole_rows(dev, rows, n, out):
    rng = rng_for(6, rows, n)
    o, z, w = (1e-2 * rng.standard_normal((rows, n))).astype(np.float32), rng.standard_normal((rows, n)) * 3, (1 + 0.2 * rng.standard_normal(n)).astype(np.float32)
    ds, ld = split_source(dev, np.concatenate([np.zeros((rows, 8)), z], 1), 2, pad8(n + 8))
    o_ld = pad8(n)
    do, dw, y = dev.from_numpy(np.pad(o, ((0, 0), (0, o_ld - n)))), dev.from_numpy(w), filled(dev, rows * o_ld, out, 3)
    N.call("ns_gated_norm", dev.handle, u(do.ptr), o_ld, u(ds.ptr), 2, N.NS_F32, ld, 8, N.ACT_SIGMOID, u(dw.ptr), fl(1e-4), i64(rows), 1, n, out, u(y.ptr), o_ld)
    dev.synchronize()
    got = read(y, (rows, o_ld), out)
    close(got[:, :n], F.rms_norm(o.astype(np.float64), w, 1e-4) * F.sigmoid(z), 2e-5 if out == N.NS_F32 else 3e-2)
    assert not got[:, n:].any()


# ------------------------------------------------------------------------------------------------ linear attention
def run_lightning(dev, name, x, decay, H, dim, vdim, cuts, source=N.NS_F32, segments=0, sequences=2):
    """Sequence b of x [sequences, T, columns] in slot 2 - b, portion by portion; (outputs, states)."""
    T, ld = x.shape[1], pad8(x.shape[2])
    st = Slots(dev, [2 - b for b in range(sequences)], [0] * sequences, 3)
    state = dev.zeros(3 * H * dim * vdim)
    dec, log2 = dev.from_numpy(np.asarray(decay, np.float32)), dev.from_numpy(np.maximum(np.log2(np.maximum(decay, 1e-300)), -1e4).astype(np.float32))
    got, at = np.zeros((sequences, T, H * vdim)), 0
    for n in cuts:
        rows = np.ascontiguousarray(np.pad(x[:, at:at + n].reshape(sequences * n, -1), ((0, 0), (0, ld - x.shape[2]))), np.float32)
        src = dev.from_numpy(BITS[source](rows))
        o = filled(dev, sequences * n * H * vdim, N.NS_F32, np.nan)
        extra = (segments,) if name == "ns_lightning_chunked" else ()
        N.call(name, dev.handle, u(src.ptr), 1, source, ld, 0, H * dim, 2 * H * dim, u(dec.ptr), u(log2.ptr), u(state.ptr), i64(H * dim * vdim), u(st.slots.ptr), sequences, n, H,
               dim, vdim, u(o.ptr), H * vdim, *extra)
        dev.synchronize()
        got[:, at:at + n] = o.download((sequences, n, H * vdim))
        at += n
    return got, state.download((3, H, dim, vdim))


def lightning_case(seed, H, dim, vdim, T, sequences=2):
    rng = rng_for(seed, H, dim, vdim, T)
    x = rng.standard_normal((sequences, T, H * (2 * dim + vdim)))
    decay = rng.permutation(np.concatenate([[1.0, 0.0, 0.999, 0.2], rng.uniform(0.3, 1.0, 8)]))[:H]
    return x, decay


def lightning_want(x, decay, H, dim, vdim, rounded):
    outs, states = [], []
    for seq in x:
        act = F.silu(as_bf16(seq).astype(np.float64) if rounded else seq)
        if rounded:
            act = as_bf16(act).astype(np.float64)
        q, k, v = np.split(act, [H * dim, 2 * H * dim], axis=1)
        o, s = F.decayed_memory(q.reshape(-1, H, dim), k.reshape(-1, H, dim), v.reshape(-1, H, vdim), decay)
        outs.append(o.reshape(len(seq), -1)), states.append(s)
    return np.stack(outs), np.stack(states)


SIZES = [(3, 20, 28), (1, 1, 1), (2, 64, 64), (2, 128, 72), (4, 96, 130), (2, 33, 7), (1, 32, 200)]


@pytest.mark.parametrize("H,dim,vdim", SIZES + [(1, 200, 40), (2, 256, 129)])
def test_recurrence_token_by_token(dev, H, dim, vdim):
    x, decay = lightning_case(10, H, dim, vdim, 40)
    want, states = lightning_want(x, decay, H, dim, vdim, False)
    for cuts in ((40,), (1,) * 40, (2, 7, 1, 30)):
        got, s = run_lightning(dev, "ns_lightning_recurrent", x, decay, H, dim, vdim, cuts)
        close(got, want, 1e-5)
        close(s[[2, 1]], states, 1e-5)
        assert not s[0].any()


@pytest.mark.parametrize("source", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("H,dim,vdim", SIZES)
def test_recurrence_in_chunks(dev, H, dim, vdim, source):
    """Against products of the same rounded activations: what is left is 32-bit and the two bf16 halves."""
    x, decay = lightning_case(11, H, dim, vdim, 333)
    x = as_bf16(x).astype(np.float64)
    want, states = lightning_want(x, decay, H, dim, vdim, True)
    for cuts, segments in (((333,), 1), ((333,), 2), ((333,), 4), ((333,), 0), ((64, 64, 205), 0), ((63, 65, 2, 1, 130, 72), 1), ((128, 205), 3)):
        got, s = run_lightning(dev, "ns_lightning_chunked", x, decay, H, dim, vdim, cuts, source, segments)
        # an activation halfway between two bf16 values may round the other way: an ulp of single terms
        close(got, want, 3e-2)
        assert np.sqrt(np.mean((got - want) ** 2)) < 5e-4 * np.sqrt(np.mean(want ** 2))
        close(s[[2, 1]], states, 3e-2)
        assert not s[0].any()


def test_chunks_continue_the_recurrence(dev):
    """Portions of both forms take turns on one state."""
    H, dim, vdim, cuts = 3, 48, 40, (70, 3, 1, 200, 1, 1, 58)
    x, decay = lightning_case(12, H, dim, vdim, sum(cuts))
    want, states = lightning_want(x, decay, H, dim, vdim, False)
    st, state = Slots(dev, [1, 0], [0, 0]), dev.zeros(2 * H * dim * vdim)
    dec, log2 = dev.from_numpy(np.asarray(decay, np.float32)), dev.from_numpy(np.maximum(np.log2(np.maximum(decay, 1e-300)), -1e4).astype(np.float32))
    at, got = 0, np.zeros_like(want)
    for n in cuts:
        src, o = dev.from_numpy(np.ascontiguousarray(x[:, at:at + n], np.float32)), dev.empty(2 * n * H * vdim)
        name, extra = ("ns_lightning_chunked", (0,)) if n > 16 else ("ns_lightning_recurrent", ())
        N.call(name, dev.handle, u(src.ptr), 1, N.NS_F32, x.shape[2], 0, H * dim, 2 * H * dim, u(dec.ptr), u(log2.ptr), u(state.ptr), i64(H * dim * vdim), u(st.slots.ptr), 2, n, H,
               dim, vdim, u(o.ptr), H * vdim, *extra)
        dev.synchronize()
        got[:, at:at + n] = o.download((2, n, H * vdim))
        at += n
    assert np.sqrt(np.mean((got - want) ** 2)) < 6e-3 * np.sqrt(np.mean(want ** 2))


def test_a_far_write_is_still_there(dev):
    """One loud key at the beginning, a query for it a thousand tokens later, other keys quiet; decay 1 and 0.999 keep it, 0.9 does not."""
    T, H, dim, vdim, decay = 1100, 3, 32, 32, [1.0, 0.999, 0.9]
    x = np.full((1, T, H * (2 * dim + vdim)), 1e-3)
    x[0, 3, H * dim:2 * H * dim] = 6.0
    x[0, 3, 2 * H * dim:] = np.linspace(1.0, 5.0, H * vdim)
    x[0, T - 1, :H * dim] = 4.0
    x = as_bf16(x).astype(np.float64)
    want, _ = lightning_want(x, decay, H, dim, vdim, True)
    assert (want[0, -1, :vdim] > 500).any() and (want[0, -1, 2 * vdim:] < 1).all()
    for cuts in ((T,), (700, 400), (64,) * 17 + (12,)):
        got, _ = run_lightning(dev, "ns_lightning_chunked", x, decay, H, dim, vdim, cuts, N.NS_BF16, 0, 1)
        np.testing.assert_allclose(got[0, -1], want[0, -1], rtol=2e-3, atol=1e-3)
    got, _ = run_lightning(dev, "ns_lightning_recurrent", x, decay, H, dim, vdim, (T,), N.NS_F32, 0, 1)
    np.testing.assert_allclose(got[0, -1], want[0, -1], rtol=2e-2, atol=1e-3)


# ------------------------------------------------------------------------------------------------ window attention
@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("H,G,dim,vdim,splits", [(6, 2, 20, 28, 2), (1, 1, 1, 1, 1), (5, 5, 33, 7, 1), (8, 4, 64, 128, 3), (16, 16, 128, 64, 1)])
def test_append_normalises_and_wraps(dev, H, G, dim, vdim, splits, dtype):
    rng, eps, ring, steps = rng_for(20, H, dim), 1e-3, 128, 9
    nq, nk, nv = H * dim, G * dim, G * vdim
    x = rng.standard_normal((2 * steps, nq + nk + nv + H)) * 0.05
    qw, kw = (1 + 0.2 * rng.standard_normal(nq)).astype(np.float32), (1 + 0.2 * rng.standard_normal(nk)).astype(np.float32)
    src, ld = split_source(dev, x, splits, pad8(x.shape[1]))
    st = Slots(dev, [2, 0], [124, 5], 3)
    k_ld, v_ld = pad8(dim), pad8(vdim)
    kr, vr = dev.zeros(3 * G * ring * k_ld, dtype), dev.zeros(3 * G * ring * v_ld, dtype)
    q, gate, dq, dk = filled(dev, 2 * steps * H * k_ld, dtype, 5), dev.empty(2 * steps * H), dev.from_numpy(qw), dev.from_numpy(kw)
    N.call("ns_window_append", dev.handle, u(src.ptr), splits, N.NS_F32, ld, 0, nq, nq + nk, nq + nk + nv, H, G, dim, vdim, u(dq.ptr), u(dk.ptr), fl(eps), u(st.slots.ptr),
           u(st.pos.ptr), 2, steps, dtype, u(q.ptr), u(gate.ptr), u(kr.ptr), u(vr.ptr), i64(G * ring * k_ld), i64(G * ring * v_ld), ring, k_ld, v_ld)
    dev.synchronize()
    tol = 1e-5 if dtype == N.NS_F32 else 2e-2
    got = read(q, (2 * steps, H, k_ld), dtype)
    close(got[:, :, :dim], F.rms_norm(x[:, :nq], qw, eps).reshape(-1, H, dim), tol)
    assert not got[:, :, dim:].any()
    close(gate.download((2 * steps, H)), F.sigmoid(x[:, nq + nk + nv:]), 1e-5)
    want_k = np.zeros((3, ring, G, k_ld))
    want_v = np.zeros((3, ring, G, v_ld))
    for b, (slot, pos) in enumerate(((2, 124), (0, 5))):
        for i in range(steps):
            row = x[b * steps + i]
            want_k[slot, (pos + i) % ring, :, :dim] = F.rms_norm(row[nq:nq + nk], kw, eps).reshape(G, dim)
            want_v[slot, (pos + i) % ring, :, :vdim] = row[nq + nk:nq + nk + nv].reshape(G, vdim)
    for ring_dev, want in ((kr, want_k), (vr, want_v)):
        got = read(ring_dev, (3, G, ring, want.shape[-1]), dtype).transpose(0, 2, 1, 3)
        close(got, want, tol * 10)
        assert not got[want == 0].any()


@pytest.mark.parametrize("norms", [True, False])
@pytest.mark.parametrize("H,G,dim,vdim", [(6, 2, 24, 40), (1, 1, 8, 8), (16, 4, 128, 64), (5, 5, 48, 16), (30, 2, 256, 24), (3, 1, 16, 8)])
def test_append_from_a_bf16_matrix(dev, H, G, dim, vdim, norms):
    rng, eps, ring, steps = rng_for(21, H, dim), 1e-3, 128, 9
    nq, nk, nv = H * dim, G * dim, G * vdim
    x = as_bf16(rng.standard_normal((2 * steps, nq + nk + nv + H)) * 0.05)
    ld = pad8(x.shape[1])
    src = dev.from_numpy(bf16_bits(np.pad(x, ((0, 0), (0, ld - x.shape[1])))))
    qw, kw = (1 + 0.2 * rng.standard_normal(nq)).astype(np.float32), (1 + 0.2 * rng.standard_normal(nk)).astype(np.float32)
    st, dq, dk = Slots(dev, [2, 0], [124, 5], 3), dev.from_numpy(qw), dev.from_numpy(kw)
    kr, vr = dev.zeros(3 * G * ring * dim, N.NS_BF16), dev.zeros(3 * G * ring * vdim, N.NS_BF16)
    q, gate = filled(dev, 2 * steps * H * dim, N.NS_BF16, 5), dev.empty(2 * steps * H)
    N.call("ns_window_append", dev.handle, u(src.ptr), 1, N.NS_BF16, ld, 0, nq, nq + nk, nq + nk + nv, H, G, dim, vdim, u(dq.ptr if norms else 0), u(dk.ptr if norms else 0),
           fl(eps), u(st.slots.ptr), u(st.pos.ptr), 2, steps, N.NS_BF16, u(q.ptr), u(gate.ptr), u(kr.ptr), u(vr.ptr), i64(G * ring * dim), i64(G * ring * vdim), ring, dim, vdim)
    dev.synchronize()
    norm = (lambda a, w: F.rms_norm(a.astype(np.float64), w, eps)) if norms else (lambda a, w: a)
    close(read(q, (2 * steps, nq), N.NS_BF16), norm(x[:, :nq], qw), 2e-2)
    close(gate.download((2 * steps, H)), F.sigmoid(x[:, nq + nk + nv:]), 1e-5)
    got_k, got_v = read(kr, (3, G, ring, dim), N.NS_BF16), read(vr, (3, G, ring, vdim), N.NS_BF16)
    for b, (slot, pos) in enumerate(((2, 124), (0, 5))):
        rows, at = x[b * steps:(b + 1) * steps], (pos + np.arange(steps)) % ring
        close(got_k[slot][:, at].transpose(1, 0, 2).reshape(steps, nk), norm(rows[:, nq:nq + nk], kw), 2e-2)
        assert np.array_equal(got_v[slot][:, at].transpose(1, 0, 2).reshape(steps, nv), rows[:, nq + nk:nq + nk + nv])
        rest = np.setdiff1d(np.arange(ring), at)
        assert not got_k[slot][:, rest].any() and not got_v[slot][:, rest].any()


class WindowCase:
    """Queries, keys and values of two sequences, in rings whose other rows hold loud keys and values.  The key just outside the window
    of one row (the first of sequence 0, the last of sequence 1) would take all of its weight, the one just inside takes much of it,
    and the sinks weigh as much as the keys of that row."""

    def __init__(self, H, G, dim, vdim, window, steps, starts, seed=0):
        rng = rng_for(30, H, dim, window, steps, seed)
        self.sizes, self.window, self.steps, self.starts = (H, G, dim, vdim), window, steps, starts
        self.scale = 0.7 / np.sqrt(dim)
        self.ring = -(-(window - 1 + steps) // 128) * 128
        self.q = as_bf16(rng.standard_normal((2, steps, H, dim)))
        # queries of neighbouring tokens look in one direction that an edge key shares
        edge = rng.standard_normal((2, G, dim)) * 2.0
        self.q = as_bf16(self.q * 0.5 + np.repeat(edge, H // G, axis=1)[:, None])
        self.k, self.v = [], []
        for b, p in enumerate(starts):
            n = p + steps
            k, v = rng.standard_normal((n, G, dim)) * 0.5, rng.standard_normal((n, G, vdim))
            at = p + b * (steps - 1)
            for back, size in ((window, 4.0), (window - 1, 0.6)):
                if at - back >= 0:
                    k[at - back] += size * edge[b]
            self.k.append(as_bf16(k)), self.v.append(as_bf16(v))
        last = np.einsum("hd,jhd->hj", self.q[1, -1].astype(np.float64), self.k[1][max(0, starts[1] + steps - window):][:, np.arange(H) // (H // G)]) * self.scale
        top = last.max(axis=1)
        self.sink = (top + np.log(np.exp(last - top[:, None]).sum(axis=1)) + 0.5 * rng.standard_normal(H)).astype(np.float32)
        self.gate = rng.uniform(0.1, 1.0, (2 * steps, H)).astype(np.float32)

    def check(self, dev, name, sink=True, gate=True):
        """bf16: what is rounded is the weights, as operands of the second product, and the output -- 2^-8 each of a sum of absolute values."""
        got, want, size = self.run(dev, name, N.NS_BF16, sink, gate), self.want(sink, gate), self.want(sink, gate, values=[np.abs(v) for v in self.v])
        over = float((np.abs(got - want) / (size + 1e-6)).max()) * 2.0 ** 8
        assert over < 2.3, f"{over:.3g} roundings of the absolute values' sum"

    def want(self, sink=True, gate=True, window=None, values=None):
        H, G, dim, vdim = self.sizes
        out, owner = [], np.arange(H) // (H // G)
        for b, p in enumerate(self.starts):
            score = np.einsum("ihd,jhd->hij", self.q[b].astype(np.float64), self.k[b][:, owner]) * self.scale
            s = self.sink.astype(np.float64) if sink else np.full(H, -1e30)
            a = F.sink_softmax(score, s, F.visible(np.arange(p, p + self.steps), np.arange(p + self.steps), window or self.window))
            o = np.einsum("hij,jhv->ihv", a, (values or self.v)[b][:, owner])
            out.append(o * self.gate[b * self.steps:(b + 1) * self.steps, :, None] if gate else o)
        return np.stack(out)

    def run(self, dev, name, dtype, sink=True, gate=True):
        H, G, dim, vdim = self.sizes
        k_ld, v_ld, ring, rng = pad8(dim), pad8(vdim), self.ring, rng_for(31)
        k, v = np.zeros((4, G, ring, k_ld), np.float32), np.zeros((4, G, ring, v_ld), np.float32)
        k[..., :dim], v[..., :vdim] = 30.0 * rng.standard_normal((4, G, ring, dim)), 100.0
        slots = [3, 1]
        for b, slot in enumerate(slots):
            for j in range(max(0, len(self.k[b]) - ring), len(self.k[b])):
                k[slot, :, j % ring, :dim], v[slot, :, j % ring, :vdim] = self.k[b][j], self.v[b][j]
        q = np.zeros((2 * self.steps, H, k_ld), np.float32)
        q[..., :dim] = self.q.reshape(-1, H, dim)
        st = Slots(dev, slots, list(self.starts), 4)
        up = lambda a: dev.from_numpy(BITS[dtype](a))
        dq, dk, dv, ds, dg = up(q), up(k), up(v), dev.from_numpy(self.sink), dev.from_numpy(self.gate)
        o_ld = pad8(H * vdim)
        o = dev.zeros(2 * self.steps * o_ld, dtype)
        rings = (u(dk.ptr), u(dv.ptr), i64(G * ring * k_ld), i64(G * ring * v_ld))
        rest = (ring, k_ld, v_ld, u(ds.ptr if sink else 0), u(dg.ptr if gate else 0), u(st.slots.ptr), u(st.pos.ptr), 2, self.steps, H, G, dim, vdim, self.window,
                fl(self.scale), u(o.ptr), i64(o_ld))
        if name == "ns_window_attend":
            N.call(name, dev.handle, dtype, u(dq.ptr), *rings, *rest)
        elif name == "ns_window_decode":
            N.call(name, dev.handle, u(dq.ptr), *rings, *rest)
        else:
            N.call(name, dev.handle, u(dq.ptr), *rings, 4, *rest)
        dev.synchronize()
        got = read(o, (2 * self.steps, o_ld), dtype)
        assert not got[:, H * vdim:].any()
        return got[:, :H * vdim].reshape(2, self.steps, H, vdim)


HEADS = [(6, 2, 20, 28), (1, 1, 8, 8), (4, 4, 64, 64), (8, 1, 128, 128), (3, 3, 72, 40), (2, 2, 128, 48), (4, 2, 40, 104)]
WINDOWS = [1, 2, 15, 16, 17, 100, 127, 128, 129, 300]


def test_the_window_case_shows_an_edge():
    """The test's own inputs: a window one token off, a sink or a gate left out is far outside the tolerances used below."""
    c = WindowCase(4, 2, 32, 24, 50, 20, (200, 31))
    full = c.want()
    rms = np.sqrt(np.mean(full ** 2))
    for other in (c.want(window=49), c.want(window=51), c.want(sink=False), c.want(gate=False)):
        assert np.abs(other - full).max() > 0.5 * rms


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("H,G,dim,vdim", [(6, 2, 20, 28), (2, 2, 264, 300), (5, 1, 7, 65)])
def test_float32_attention(dev, H, G, dim, vdim, window):
    for steps, starts in ((1, (0, 700)), (1, (window, window - 1)), (3, (126, 5)), (33, (130, 0))):
        c = WindowCase(H, G, dim, vdim, window, steps, starts)
        close(c.run(dev, "ns_window_attend", N.NS_F32), c.want(), 5e-4)
    c = WindowCase(H, G, dim, vdim, window, 2, (9, 260))
    close(c.run(dev, "ns_window_attend", N.NS_F32, sink=False, gate=False), c.want(False, False), 5e-4)
    c.check(dev, "ns_window_attend")


@pytest.mark.parametrize("window", WINDOWS + [1500])
@pytest.mark.parametrize("H,G,dim,vdim", HEADS + [(3, 1, 200, 256), (2, 2, 256, 136)])
def test_few_tokens(dev, H, G, dim, vdim, window):
    for steps, starts in ((1, (0, 2000)), (1, (window, window - 1)), (2, (126, 15)), (5, (16, 511)), (31, (700, 0))):
        c = WindowCase(H, G, dim, vdim, window, steps, starts)
        c.check(dev, "ns_window_decode")
    c = WindowCase(H, G, dim, vdim, window, 2, (9, 260))
    c.check(dev, "ns_window_decode", sink=False, gate=False)


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("H,G,dim,vdim", [h for h in HEADS if h[3] % 8 == 0])
def test_a_prompts_portion(dev, H, G, dim, vdim, window):
    for steps, starts in ((1, (0, 700)), (2, (window, window - 1)), (32, (0, 127)), (128, (0, 128)), (129, (65, 1000)), (300, (0, 383))):
        c = WindowCase(H, G, dim, vdim, window, steps, starts)
        c.check(dev, "ns_window_prefill")
    c = WindowCase(H, G, dim, vdim, window, 140, (9, 260))
    c.check(dev, "ns_window_prefill", sink=False, gate=False)


@pytest.mark.parametrize("name", ["ns_window_attend", "ns_window_decode", "ns_window_prefill"])
def test_sinks_of_any_size(dev, name):
    for value in (-200.0, 0.0, 200.0):
        c = WindowCase(4, 2, 32, 24, 20, 40, (100, 3))
        c.sink[:] = [value, 0.0, -value, 1.0]
        c.check(dev, name)


def test_bad_calls_are_refused(dev):
    z = dev.zeros(4 * 2 * 128 * 32, N.NS_BF16)

    def call(name, heads=4, vdim=24, window=20, ring=128):
        lens = (4,) if name == "ns_window_prefill" else ()
        N.call(name, dev.handle, u(z.ptr), u(z.ptr), u(z.ptr), i64(0), i64(0), *lens, ring, 32, 24, u(0), u(0), u(z.ptr), u(z.ptr), 1, 40, heads, 2, 32, vdim, window, fl(1.0),
               u(z.ptr), i64(160))

    for name in ("ns_window_decode", "ns_window_prefill"):
        for bad in ({"ring": 64}, {"window": 129}, {"heads": 5}, {"vdim": 25}):
            with pytest.raises(N.NsError):
                call(name, **bad)
    with pytest.raises(N.NsError):
        call("ns_window_prefill", vdim=20)                               # values that are no multiple of 8
