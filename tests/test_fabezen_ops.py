"""The operators behind Fabezen's layers, each alone against its plain float64 statement (oracle/fabezen.py)."""
import ctypes as C

import numpy as np
import pytest

from nn_b200 import native as N
from nn_b200.blocks import bf16_bits, f32
from oracle import fabezen as F

pytestmark = pytest.mark.gpu
u, i64, fl = C.c_uint64, C.c_int64, C.c_float


def rng_for(*key):
    return np.random.default_rng(list(key))


def close(got, want, tol):
    scale = max(1e-6, float(np.sqrt(np.mean(np.square(want)))))
    err = float(np.abs(got - want).max()) / scale
    assert err <= tol, f"largest error {err:.3g} of the root mean square"


class Slots:
    """slots, positions and last tokens of a step on the device."""

    def __init__(self, dev, slots, pos, total=None):
        total = total or max(slots) + 1
        p = np.zeros(total, np.int32)
        p[slots] = pos
        self.dev, self.slots = dev, dev.from_numpy(np.asarray(slots, np.int32))
        self.pos, self.last = dev.from_numpy(p), dev.from_numpy(np.full(total, -1, np.int32))


def split_source(dev, x, splits, ld=None):
    """x as `splits` float slabs that add up to it."""
    rows, cols = x.shape
    ld = ld or cols
    parts = np.zeros((splits, rows, ld), np.float32)
    parts[:, :, :cols] = rng_for(splits, rows, cols).standard_normal((splits, rows, cols)).astype(np.float32)
    parts[0, :, :cols] = (x - parts[1:, :, :cols].sum(0)).astype(np.float32)
    return dev.from_numpy(parts), ld


# ------------------------------------------------------------------------------------------------ embedding
@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
def test_embedding_with_bigrams_across_steps(dev, dtype):
    V, D, buckets, mp, mc = 50, 36, 23, 17, 3
    rng = rng_for(1)
    w = {"embed": f32(bf16_bits(rng.standard_normal((V, D)))), "bigram": f32(bf16_bits(rng.standard_normal((buckets + 1, D))))}
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    seqs = rng.integers(0, V, (2, 9)).astype(np.int32)
    want = np.stack([F.embedding(s, w, cfg) for s in seqs])
    conv = (lambda a: dev.from_numpy(a)) if dtype == N.NS_F32 else (lambda a: dev.from_numpy(bf16_bits(a)))
    table, big = conv(w["embed"]), conv(w["bigram"])
    st = Slots(dev, [2, 0], [0, 0])
    got, at = np.zeros_like(want), 0
    for n in (1, 3, 1, 4):
        ids = dev.from_numpy(np.ascontiguousarray(seqs[:, at:at + n]))
        y = dev.empty(2 * n * D)
        N.call("ns_embed_ngram", dev.handle, u(ids.ptr), u(table.ptr), dtype, D, fl(2.5), u(big.ptr), D, buckets, i64(mp), i64(mc), u(st.slots.ptr),
               u(st.last.ptr), 2, n, D, V, u(y.ptr))
        N.call("ns_seq_advance", dev.handle, u(ids.ptr), u(st.slots.ptr), 2, n, u(st.pos.ptr), u(st.last.ptr))
        dev.synchronize()
        got[:, at:at + n] = y.download((2, n, D))
        at += n
    close(got, want, 1e-6)
    assert list(st.pos.download()) == [9, 0, 9]
    assert list(st.last.download()[[2, 0]]) == list(seqs[:, -1])


def test_bigram_rows_with_large_multipliers(dev):
    V, D, buckets, mp, mc = 70000, 4, 65521, 2147483647, 1000003
    w = {"embed": np.zeros((V, D), np.float32), "bigram": np.repeat(np.arange(buckets + 1, dtype=np.float32)[:, None], D, 1)}
    ids = np.array([[69999, 69998, 3, 69999]], np.int32)
    st = Slots(dev, [0], [0])
    y = dev.empty(4 * D)
    t, b, di = dev.from_numpy(w["embed"]), dev.from_numpy(w["bigram"]), dev.from_numpy(ids)
    N.call("ns_embed_ngram", dev.handle, u(di.ptr), u(t.ptr), N.NS_F32, D, fl(1.0), u(b.ptr), D, buckets, i64(mp), i64(mc), u(st.slots.ptr), u(st.last.ptr), 1, 4,
           D, V, u(y.ptr))
    dev.synchronize()
    assert list(y.download((4, D))[:, 0].astype(int)) == F.bigram_rows(ids[0], buckets, mp, mc)


# ------------------------------------------------------------------------------------------------ rows
@pytest.mark.parametrize("rows,cols,splits,out", [(5, 64, 3, N.NS_BF16), (3, 61, 1, N.NS_F32), (130, 2048, 2, N.NS_BF16), (4, 5000, 1, N.NS_F32)])
def test_residual_and_rms(dev, rows, cols, splits, out):
    rng = rng_for(2, rows, cols)
    x, s, w = rng.standard_normal((rows, cols)), rng.standard_normal((rows, cols)), 1 + 0.1 * rng.standard_normal(cols)
    dx, dw = dev.from_numpy(x.astype(np.float32)), dev.from_numpy(w.astype(np.float32))
    ds, ld = split_source(dev, s, splits, (cols + 7) // 8 * 8)
    y_ld = (cols + 7) // 8 * 8
    y = dev.from_numpy(np.full(rows * y_ld, 7, np.float32 if out == N.NS_F32 else np.uint16))
    N.call("ns_rms_rows", dev.handle, u(dx.ptr), u(ds.ptr), splits, N.NS_F32, ld, fl(0.3), u(dx.ptr), u(dw.ptr), fl(1e-3), u(0), i64(rows), i64(rows), cols, out,
           u(y.ptr), y_ld)
    dev.synchronize()
    stream = x + 0.3 * s
    close(dx.download((rows, cols)), stream, 2e-6)
    got = y.download((rows, y_ld)) if out == N.NS_F32 else f32(y.download((rows, y_ld)))
    close(got[:, :cols], F.rms_norm(stream, w, 1e-3), 2e-6 if out == N.NS_F32 else 2e-2)
    assert not got[:, cols:].any()


def test_rms_of_named_rows_and_small_values(dev):
    rows, cols = 6, 40
    x = (rng_for(3).standard_normal((rows, cols)) * 1e-3).astype(np.float32)     # eps matters
    m = np.array([5, 0, 0, 3], np.int32)
    dx, dm, dw, y = dev.from_numpy(x), dev.from_numpy(m), dev.from_numpy(np.ones(cols, np.float32)), dev.empty(4 * cols)
    N.call("ns_rms_rows", dev.handle, u(dx.ptr), u(0), 1, N.NS_F32, 0, fl(0), u(0), u(dw.ptr), fl(1e-5), u(dm.ptr), i64(rows), i64(4), cols, N.NS_F32, u(y.ptr), cols)
    dev.synchronize()
    close(y.download((4, cols)), F.rms_norm(x[m].astype(np.float64), 1.0, 1e-5), 2e-6)


@pytest.mark.parametrize("rows,ff,splits,out", [(3, 20, 2, N.NS_F32), (7, 37, 1, N.NS_BF16), (300, 512, 1, N.NS_BF16)])
def test_gated_linear_unit(dev, rows, ff, splits, out):
    x = rng_for(4, rows, ff).standard_normal((rows, 2 * ff)) * 2
    s, ld = split_source(dev, x, splits, (2 * ff + 7) // 8 * 8)
    y_ld = (ff + 7) // 8 * 8
    y = dev.from_numpy(np.full(rows * y_ld, 9, np.float32 if out == N.NS_F32 else np.uint16))
    N.call("ns_glu_rows", dev.handle, u(s.ptr), splits, N.NS_F32, ld, i64(rows), ff, N.ACT_GELU, out, u(y.ptr), y_ld)
    dev.synchronize()
    got = y.download((rows, y_ld)) if out == N.NS_F32 else f32(y.download((rows, y_ld)))
    close(got[:, :ff], F.gelu_tanh(x[:, :ff]) * x[:, ff:], 3e-6 if out == N.NS_F32 else 5e-2)
    assert not got[:, ff:].any()


# ------------------------------------------------------------------------------------------------ short convolution
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("cuts", [(40,), (2, 1, 3, 2, 31, 1), (17, 23), (1,) * 12])
def test_short_convolution_over_cuts(dev, taps, cuts):
    T, kv, dim, H, vdim = sum(cuts), 2, 20, 3, 70
    rng = rng_for(5, taps, T)
    widths = [kv * dim, H * vdim]
    x = rng.standard_normal((T, sum(widths)))
    w = [rng.standard_normal((c, taps)).astype(np.float32) for c in widths]
    want = [F.unit(F.short_conv(x[:, :widths[0]], w[0].astype(np.float64)).reshape(T, kv, dim)).reshape(T, -1) * 0.25,
            F.short_conv(x[:, widths[0]:], w[1].astype(np.float64))]
    st = Slots(dev, [1], [0])
    hist = [dev.zeros(2 * taps * sum(widths)) for _ in range(1)][0]
    stride = taps * sum(widths)
    dw = [dev.from_numpy(a) for a in w]
    got, at = [np.zeros((T, c)) for c in widths], 0
    for n in cuts:
        src, ld = split_source(dev, x[at:at + n], 2, sum(widths) + 8)
        out = [dev.empty(n * c) for c in widths]
        fields = [0, kv, dim, taps, 1, dw[0].ptr, hist.ptr, out[0].ptr, widths[0], widths[0], H, vdim, taps, 0, dw[1].ptr, hist.ptr + 4 * taps * widths[0],
                  out[1].ptr, widths[1]]
        N.call("ns_short_conv", dev.handle, u(src.ptr), 2, N.NS_F32, ld, 2, (C.c_int64 * 18)(*fields), (C.c_float * 2)(0.25, 1.0), i64(stride), u(st.slots.ptr),
               u(st.pos.ptr), 1, n, N.NS_F32)
        dev.synchronize()
        for g, o, c in zip(got, out, widths):
            g[at:at + n] = o.download((n, c))
        at += n
        st.pos.upload(np.array([0, at], np.int32))
    for g, e in zip(got, want):
        close(g, e, 1e-5)


# ------------------------------------------------------------------------------------------------ delta rule
def run_delta(dev, data, cuts, H, kv, dim, vdim, channelwise, slots=(0,), chunk_from=1 << 30):
    """o [B, T, H, vdim] and final states, the sequences fed in `cuts`."""
    q, k, v, a, b, a_log, dt = data
    B, T = q.shape[:2]
    st = Slots(dev, list(slots), [0] * B, max(slots) + 1)
    stride = H * dim * vdim + 16
    state = dev.zeros((max(slots) + 1) * stride)
    da, dd = dev.from_numpy(a_log.astype(np.float32)), dev.from_numpy(dt.astype(np.float32))
    got, at = np.zeros((B, T, H * vdim)), 0
    ac = H * dim if channelwise else H
    for n in cuts:
        up = lambda z: dev.from_numpy(np.ascontiguousarray(z[:, at:at + n].reshape(B * n, -1), dtype=np.float32))
        dq, dk, dv = up(q), up(k), up(v)
        ab, ld = split_source(dev, np.concatenate([a[:, at:at + n].reshape(B * n, ac), b[:, at:at + n].reshape(B * n, H)], 1), 2, (ac + H + 7) // 8 * 8)
        o = dev.empty(B * n * H * vdim)
        N.call("ns_delta_chunked" if n >= chunk_from else "ns_delta_recurrent", dev.handle, u(dq.ptr), kv * dim, u(dk.ptr), kv * dim, u(dv.ptr), H * vdim, u(ab.ptr), 2, ld, 0, u(ab.ptr), 2, ld, ac,
               u(da.ptr), u(dd.ptr), int(channelwise), u(state.ptr), i64(stride), u(st.slots.ptr), B, n, H, kv, dim, vdim, u(o.ptr), H * vdim)
        dev.synchronize()
        got[:, at:at + n] = o.download((B, n, H * vdim))
        at += n
    s = state.download((max(slots) + 1, stride))[:, :H * dim * vdim].reshape(-1, H, dim, vdim)
    return got.reshape(B, T, H, vdim), s[list(slots)]


def delta_data(B, T, H, kv, dim, vdim, channelwise, seed=6):
    rng = rng_for(seed, T, H, dim, vdim)
    q, k = F.unit(rng.standard_normal((B, T, kv, dim))) * dim ** -0.5, F.unit(rng.standard_normal((B, T, kv, dim)))
    v = rng.standard_normal((B, T, H, vdim))
    a = rng.standard_normal((B, T, H, dim) if channelwise else (B, T, H)) * 2
    b = rng.standard_normal((B, T, H))
    a_log, dt = rng.uniform(-3, 1.5, H), rng.uniform(-3, 1, (H, dim) if channelwise else H)
    return q, k, v, a, b, a_log, dt


def delta_oracle(data, channelwise):
    q, k, v, a, b, a_log, dt = data
    B, T, kv, dim = q.shape
    H = v.shape[2]
    owner = np.arange(H) // (H // kv)
    outs = []
    for i in range(B):
        rate = np.exp(a_log)
        g = np.exp(-rate[None, :, None] * F.softplus(a[i] + dt)) if channelwise else np.repeat(np.exp(-rate * F.softplus(a[i] + dt))[:, :, None], dim, 2)
        outs.append(F.delta_rule(q[i][:, owner], k[i][:, owner], v[i], F.sigmoid(b[i]), g))
    return np.stack([o for o, _ in outs]), np.stack([s for _, s in outs])


SIZES = [(1, 1, 16, 16), (6, 2, 20, 36), (4, 1, 64, 64), (3, 3, 100, 130), (2, 1, 128, 128), (2, 2, 200, 96)]


@pytest.mark.parametrize("channelwise", [False, True])
@pytest.mark.parametrize("H,kv,dim,vdim", SIZES)
def test_delta_rule(dev, H, kv, dim, vdim, channelwise):
    data = delta_data(2, 37, H, kv, dim, vdim, channelwise)
    o, s = run_delta(dev, data, (37,), H, kv, dim, vdim, channelwise, slots=(2, 0))
    eo, es = delta_oracle(data, channelwise)
    close(o, eo, 2e-5)
    close(s, es, 2e-5)


@pytest.mark.parametrize("channelwise", [False, True])
@pytest.mark.parametrize("cuts", [(1,) * 21, (2, 16, 3), (20, 1)])
def test_delta_rule_over_cuts(dev, channelwise, cuts):
    data = delta_data(1, 21, 4, 2, 24, 48, channelwise)
    o, s = run_delta(dev, data, cuts, 4, 2, 24, 48, channelwise)
    eo, es = delta_oracle(data, channelwise)
    close(o, eo, 2e-5)
    close(s, es, 2e-5)


@pytest.mark.parametrize("channelwise", [False, True])
@pytest.mark.parametrize("T", [1, 16, 17, 63, 64, 65, 200])
@pytest.mark.parametrize("H,kv,dim,vdim", [s for s in SIZES if s[2] <= 128] + [(2, 1, 36, 66)])
def test_delta_rule_in_chunks(dev, H, kv, dim, vdim, T, channelwise):
    data = delta_data(2, T, H, kv, dim, vdim, channelwise)
    o, s = run_delta(dev, data, (T,), H, kv, dim, vdim, channelwise, slots=(2, 0), chunk_from=1)
    eo, es = delta_oracle(data, channelwise)
    close(o, eo, 1e-3)
    close(s, es, 1e-3)


@pytest.mark.parametrize("channelwise", [False, True])
def test_chunks_and_single_tokens_carry_one_state(dev, channelwise):
    cuts = (1, 40, 2, 64, 1, 1, 70)
    data = delta_data(1, sum(cuts), 4, 2, 24, 48, channelwise)
    o, s = run_delta(dev, data, cuts, 4, 2, 24, 48, channelwise, chunk_from=24)
    eo, es = delta_oracle(data, channelwise)
    close(o, eo, 1e-3)
    close(s, es, 1e-3)


@pytest.mark.parametrize("channelwise", [False, True])
@pytest.mark.parametrize("kind", ["none", "total", "mixed"])
def test_chunks_with_extreme_decays(dev, kind, channelwise):
    """No decay at all, everything forgotten at every token, and both side by side: no exponent may overflow on the way."""
    H, dim, vdim, T = 2, 64, 64, 130
    q, k, v, a, b, a_log, dt = delta_data(1, T, H, 2, dim, vdim, channelwise)
    rng = rng_for(13)
    a = {"none": np.full_like(a, -60.0), "total": np.full_like(a, 60.0), "mixed": rng.choice([-60.0, 60.0, 0.0], a.shape)}[kind]
    data = (q, k, v, a, b, np.full(H, 3.0), dt)
    o, s = run_delta(dev, data, (T,), H, 2, dim, vdim, channelwise, chunk_from=1)
    eo, es = delta_oracle(data, channelwise)
    assert np.isfinite(o).all() and np.isfinite(s).all()
    close(o, eo, 2e-3)
    close(s, es, 2e-3)


@pytest.mark.parametrize("act,name", [(N.ACT_SILU, "silu"), (N.ACT_SIGMOID, "sigmoid")])
@pytest.mark.parametrize("vdim", [1, 20, 128, 200])
def test_gated_norm(dev, act, name, vdim):
    rows, H = 9, 3
    rng = rng_for(7, vdim)
    o, z, w = rng.standard_normal((rows, H, vdim)) * 0.01, rng.standard_normal((rows, H * vdim)) * 3, rng.standard_normal(vdim)
    do, dw = dev.from_numpy(o.astype(np.float32)), dev.from_numpy(w.astype(np.float32))
    src, ld = split_source(dev, np.concatenate([np.ones((rows, 5)), z], 1), 2)
    y_ld = (H * vdim + 7) // 8 * 8
    y = dev.from_numpy(np.full(rows * y_ld, 3, np.float32))
    N.call("ns_gated_norm", dev.handle, u(do.ptr), H * vdim, u(src.ptr), 2, N.NS_F32, ld, 5, act, u(dw.ptr), fl(1e-4), i64(rows), H, vdim, N.NS_F32, u(y.ptr), y_ld)
    dev.synchronize()
    want = F.rms_norm(o, w, 1e-4) * getattr(F, name)(z).reshape(rows, H, vdim)
    got = y.download((rows, y_ld))
    close(got[:, :H * vdim].reshape(rows, H, vdim), want, 1e-5)
    assert not got[:, H * vdim:].any()


# ------------------------------------------------------------------------------------------------ latent attention
def test_latent_rows_and_rotation(dev):
    B, T, qr, kr, rd, rot, H, dim, base, eps = 2, 5, 20, 28, 10, 8, 3, 12, 300.0, 1e-4
    rng = rng_for(8)
    x, qn, kn = rng.standard_normal((B * T, qr + kr + rd)), rng.standard_normal(qr), rng.standard_normal(kr)
    pos0, ring_len, ld = [7, 1000003], 9, 40
    st = Slots(dev, [1, 0], pos0)
    freq = dev.from_numpy((base ** (-2.0 * np.arange(rot // 2) / rot)).astype(np.float32))
    src, sld = split_source(dev, x, 2)
    dq, dk = dev.from_numpy(qn.astype(np.float32)), dev.from_numpy(kn.astype(np.float32))
    cq, ring = dev.empty(B * T * 24), dev.zeros(2 * ring_len * ld)
    N.call("ns_latent_append", dev.handle, u(src.ptr), 2, N.NS_F32, sld, qr, kr, rd, rot, u(dq.ptr), u(dk.ptr), fl(eps), u(freq.ptr), u(st.slots.ptr), u(st.pos.ptr),
           B, T, N.NS_F32, u(cq.ptr), 24, u(ring.ptr), i64(ring_len * ld), ring_len, ld)
    qs = rng.standard_normal((B * T, H * (dim + rd)))
    qsrc, qld = split_source(dev, qs, 1)
    plain, turned = dev.empty(B * T * H * dim), dev.empty(B * T * H * 16)
    N.call("ns_rotate_heads", dev.handle, u(qsrc.ptr), 1, N.NS_F32, qld, H, dim, rd, rot, u(freq.ptr), u(st.slots.ptr), u(st.pos.ptr), B, T, N.NS_F32, u(plain.ptr),
           i64(H * dim), dim, N.NS_F32, u(turned.ptr), i64(H * 16), 16)
    dev.synchronize()
    got_cq = cq.download((B * T, 24))
    close(got_cq[:, :qr], F.rms_norm(x[:, :qr], qn, eps), 1e-5)
    assert not got_cq[:, qr:].any()
    rows = ring.download((2, ring_len, ld))
    for b, slot in enumerate([1, 0]):
        p = pos0[b] + np.arange(T)
        part = x[b * T:(b + 1) * T]
        # the angle is a 32-bit product, so far positions are held to what that gives
        tol = 1e-5 if p[0] < 1000 else 0.3
        close(rows[slot, p % ring_len, :kr], F.rms_norm(part[:, qr:qr + kr], kn, eps), 1e-5)
        close(rows[slot, p % ring_len, kr:kr + rd], F.rotate(part[:, qr + kr:], p, base, rot), tol)
        want_q = F.rotate(qs[b * T:(b + 1) * T].reshape(T, H, dim + rd)[:, :, dim:], p, base, rot)
        close(turned.download((B, T, H, 16))[b, :, :, :rd], want_q, tol)
    close(plain.download((B * T, H, dim)), qs.reshape(B * T, H, dim + rd)[:, :, :dim], 1e-6)


@pytest.mark.parametrize("rows,H,k,n", [(1, 1, 16, 44), (5, 3, 20, 44), (70, 9, 48, 136), (130, 2, 128, 65)])
@pytest.mark.parametrize("transposed", [False, True])
def test_head_products(dev, rows, H, k, n, transposed):
    rng = rng_for(9, rows, k, n)
    x, w = rng.standard_normal((rows, H, k)).astype(np.float32), f32(bf16_bits(rng.standard_normal((H, n, k) if transposed else (H, k, n))))
    want = np.einsum("rhk,hnk->rhn" if transposed else "rhk,hkn->rhn", x.astype(np.float64), w.astype(np.float64))
    wk, wn = (1, k) if transposed else (n, 1)
    xb = f32(bf16_bits(x))
    want_b = np.einsum("rhk,hnk->rhn" if transposed else "rhk,hkn->rhn", xb.astype(np.float64), w.astype(np.float64))
    for xd, wd, yd in [(N.NS_F32, N.NS_F32, N.NS_F32), (N.NS_BF16, N.NS_BF16, N.NS_F32), (N.NS_F32, N.NS_BF16, N.NS_BF16)]:
        dx = dev.from_numpy(x if xd == N.NS_F32 else bf16_bits(x))
        dw = dev.from_numpy(w if wd == N.NS_F32 else bf16_bits(w))
        y = dev.empty(rows * H * n, yd)
        N.call("ns_head_matmul", dev.handle, xd, u(dx.ptr), i64(H * k), k, wd, u(dw.ptr), i64(k * n), i64(wk), i64(wn), yd, u(y.ptr), i64(H * n), n, rows, H, k, n)
        dev.synchronize()
        got = y.download((rows, H, n)) if yd == N.NS_F32 else f32(y.download((rows, H, n)))
        close(got, want if xd == N.NS_F32 else want_b, 2e-5 if yd == N.NS_F32 else 3e-2)


FORMS = {"f32": N.NS_F32, "f32_on_bf16_rows": N.NS_BF16, "tensor_cores": N.NS_BF16}


def attend(dev, q, ring_rows, window, pos, steps, rank, scale, form, ring_len):
    """q [B, steps, H, width]; ring_rows [B, pos + steps, width] by position."""
    dtype = FORMS[form]
    B, _, H, width = q.shape
    ld = (width + 7) // 8 * 8
    st = Slots(dev, list(range(B)), [pos] * B)
    ring = np.zeros((B, ring_len, ld), np.float32)
    for p in range(max(0, pos + steps - ring_len), pos + steps):
        ring[:, p % ring_len, :width] = ring_rows[:, p]
    dr = dev.from_numpy(ring if dtype == N.NS_F32 else bf16_bits(ring))
    tail = (u(dr.ptr), i64(ring_len * ld), ring_len, ld, rank, width, window, fl(scale), u(st.slots.ptr), u(st.pos.ptr), B, steps, H)
    if form == "tensor_cores":
        dq, o = dev.from_numpy(bf16_bits(q)), dev.empty(B * steps * H * rank, N.NS_BF16)
        N.call("ns_latent_decode", dev.handle, u(dq.ptr), *tail, u(o.ptr))
        dev.synchronize()
        return f32(o.download((B, steps, H, rank)))
    dq, o = dev.from_numpy(q.astype(np.float32)), dev.empty(B * steps * H * rank)
    N.call("ns_latent_attend", dev.handle, u(dq.ptr), dtype, *tail, u(o.ptr))
    dev.synchronize()
    return o.download((B, steps, H, rank))


def attend_oracle(q, rows, window, pos, rank, scale):
    B, steps, H, _ = q.shape
    out = np.zeros((B, steps, H, rank))
    for b in range(B):
        for i in range(steps):
            p = pos + i
            lo = max(0, p - window + 1)
            s = np.einsum("hw,jw->hj", q[b, i], rows[b, lo:p + 1]) * scale
            s = np.exp(s - s.max(1, keepdims=True))
            out[b, i] = (s / s.sum(1, keepdims=True)) @ rows[b, lo:p + 1, :rank]
    return out


@pytest.mark.parametrize("form", list(FORMS))
@pytest.mark.parametrize("H,rank,rd,window,pos,steps", [(1, 16, 2, 1, 0, 1), (3, 44, 12, 11, 5, 9), (9, 136, 16, 70, 300, 3), (16, 512, 64, 129, 1000, 2),
                                                       (5, 64, 8, 33, 31, 1), (5, 64, 8, 64, 0, 130), (40, 256, 32, 1000, 2000, 1), (2, 700, 20, 200, 90, 4)])
def test_latent_attention_over_the_ring(dev, form, H, rank, rd, window, pos, steps):
    rng = rng_for(10, H, rank, window)
    width = rank + rd
    rows = f32(bf16_bits(rng.standard_normal((2, pos + steps, width))))
    q = f32(bf16_bits(rng.standard_normal((2, steps, H, width))))
    scale = 1.5 / np.sqrt(width)
    got = attend(dev, q, rows, window, pos, steps, rank, scale, form, window - 1 + steps + 2)
    close(got, attend_oracle(q.astype(np.float64), rows.astype(np.float64), window, pos, rank, scale), 3e-2 if form == "tensor_cores" else 3e-5)


@pytest.mark.parametrize("form", list(FORMS))
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 64, 65, 100])
def test_a_standing_out_key_at_the_windows_edges(dev, form, window):
    """One key takes nearly all weight where it is seen, and none one token further."""
    H, rank, rd, pos, steps = 2, 32, 8, 150, 3
    width = rank + rd
    rng = rng_for(11, window)
    q = np.zeros((1, steps, H, width), np.float32)
    q[..., 0] = 1.0
    base = f32(bf16_bits(0.1 * rng.standard_normal((1, pos + steps, width))))
    base[..., 0] = 0.0
    for i in range(steps):
        for back, seen in ((window - 1, True), (window, False), (0, True)):
            j = pos + i - back
            rows = base.copy()
            rows[0, j, 0], rows[0, j, 1] = 30.0, 16.0
            got = attend(dev, q, rows, window, pos, steps, rank, 1.0, form, window - 1 + steps)[0, i]
            assert (abs(got[:, 1] - 16.0).max() < 0.05) if seen else (abs(got[:, 1]).max() < 1.0), (i, back)


@pytest.mark.parametrize("H,dim,rd,vdim,rank,window,pos,steps", [(2, 16, 2, 16, 16, 1, 0, 5), (3, 20, 12, 36, 44, 11, 0, 40), (3, 20, 12, 36, 44, 70, 31, 64),
                                                                (4, 48, 16, 80, 136, 65, 500, 130), (2, 128, 64, 128, 512, 128, 40, 200), (1, 64, 32, 200, 64, 300, 7, 65)])
def test_expanded_attention_of_a_portion(dev, H, dim, rd, vdim, rank, window, pos, steps):
    rng = rng_for(12, H, dim, window, steps)
    B, ld = 2, (rank + rd + 7) // 8 * 8
    poss = [pos, max(0, pos - 3)]
    past = min(window - 1, max(poss))
    ring_len = window - 1 + steps
    cached = f32(bf16_bits(rng.standard_normal((B, max(poss) + steps, rank + rd))))
    ring = np.full((B, ring_len, ld), 5.0, np.float32)
    for b in range(B):
        for p in range(max(0, poss[b] + steps - ring_len), poss[b] + steps):
            ring[b, p % ring_len] = 0.0
            ring[b, p % ring_len, :rank + rd] = cached[b, p]
    st, dr, keys = Slots(dev, [0, 1], poss), dev.from_numpy(bf16_bits(ring)), dev.empty(B * (past + steps) * ld, N.NS_BF16)
    nk = past + steps
    N.call("ns_latent_gather", dev.handle, u(dr.ptr), i64(ring_len * ld), ring_len, ld, past, u(st.slots.ptr), u(st.pos.ptr), B, nk, u(keys.ptr))
    dev.synchronize()
    got_keys = f32(keys.download((B, nk, ld)))
    for b in range(B):
        for j in range(nk):
            p = poss[b] - past + j
            assert np.array_equal(got_keys[b, j, :rank + rd], cached[b, p] if p >= 0 else np.zeros(rank + rd, np.float32))
    kv_ld = (H * (dim + vdim) + 7) // 8 * 8
    kv = f32(bf16_bits(rng.standard_normal((B, nk, kv_ld))))
    q = f32(bf16_bits(rng.standard_normal((B, steps, H, dim + rd))))
    o_ld = (H * vdim + 7) // 8 * 8
    dq, dkv, o = dev.from_numpy(bf16_bits(q)), dev.from_numpy(bf16_bits(kv)), dev.zeros(B * steps * o_ld, N.NS_BF16)
    scale = 1.5 / np.sqrt(dim + rd)
    N.call("ns_latent_prefill", dev.handle, u(dq.ptr), i64(H * (dim + rd)), u(dkv.ptr), i64(kv_ld), u(keys.ptr), i64(ld), rank, u(st.slots.ptr), u(st.pos.ptr), B, steps,
           H, dim, rd, vdim, past, window, fl(scale), u(o.ptr), i64(o_ld))
    dev.synchronize()
    got = f32(o.download((B, steps, o_ld)))[:, :, :H * vdim].reshape(B, steps, H, vdim)
    for b in range(B):
        k = kv[b, :, :H * dim].reshape(nk, H, dim)
        v = kv[b, :, H * dim:H * (dim + vdim)].reshape(nk, H, vdim)
        want = np.zeros((steps, H, vdim))
        for i in range(steps):
            lo, hi = max(i + past - window + 1, past - poss[b], 0), i + past + 1
            s = (np.einsum("hd,jhd->hj", q[b, i, :, :dim], k[lo:hi]) + np.einsum("hd,jd->hj", q[b, i, :, dim:], got_keys[b, lo:hi, rank:rank + rd])) * scale
            s = np.exp(s - s.max(1, keepdims=True))
            want[i] = np.einsum("hj,jhv->hv", s / s.sum(1, keepdims=True), v[lo:hi])
        close(got[b], want, 3e-2)
