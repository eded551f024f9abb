// Gated delta rule: short causal convolutions with carried history, the recurrence itself (one decay per head or one per head
// and key channel), and the normalised, gated read-out.
//
// Per head a state S [dim, vdim] in 32-bit floats lives in the sequence's slot.  Per token
//     S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// and since S after the write is the decayed state plus k u^T, the read-out is o = (decayed S)^T q + (k . q) u: one pass over
// the decayed state gives both S^T k and S^T q, and one barrier per token suffices.
//
// The reference has no recurrent layer on its cached path; conventions (device-side position, one launch per operator, error
// codes) are those of the cached attention beside it.
#include "ns_seq.cuh"

namespace {

// ---------------------------------------------------------------------------------------------
// short convolution + silu (+ unit length per head)
// ---------------------------------------------------------------------------------------------
constexpr int CONV_MAX_SEGMENTS = 4;
constexpr int CONV_CHUNK = 16;

struct ConvSegment {
    int col;              // first column of this tensor in the source
    int heads, hd;        // channels = heads * hd
    int taps;
    int unit;             // 1: every head becomes a unit vector, times scale
    float scale;
    const float* w;       // [channels, taps], the current token's weight last
    float* hist;          // slot 0's history [taps, channels], addressed by position modulo taps
    void* out;            // [rows, out_ld]
    int out_ld;
};
struct ConvArgs {
    NsSource src;
    ConvSegment seg[CONV_MAX_SEGMENTS];
    int segments;
    int64_t hist_slot_stride;
    const int32_t* slots;
    const int32_t* pos;
    int steps;
    int chunk;
};

// The raw inputs of the last taps - 1 tokens are the carried state.  They sit at position modulo taps: a step of one token
// writes the one place that none of the taps - 1 earlier inputs occupies.  Of a longer step the CTA of the first chunk both
// reads the history and, after a barrier, replaces it; no other CTA touches these channels' history.
// V neighbouring channels of a head per lane (32 * V covers the head), up to TAPS taps.  A warp takes CONV_WARP tokens of one head and
// slides over them with the last inputs in registers, so every input is read once plus taps - 1 at the seam.  `span` warps of a
// CTA share a head: 4 for prompts, 1 for the few tokens of a decoding step (the CTA then holds four heads).
constexpr int CONV_WARP = 8;

enum { CONV_ANY = 0, CONV_F32 = 1, CONV_BF16 = 2 };   // what the source is: anything, one float matrix, one bf16 matrix

template <int V, int SRC>
NS_DEVINL void conv_load(const NsSource& s, int64_t idx, float (&x)[V])
{
    if constexpr (SRC == CONV_F32 && V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(s.ptr) + idx);
        x[0] = t.x; x[1] = t.y; x[2] = t.z; x[3] = t.w;
    } else if constexpr (SRC == CONV_BF16 && V == 4) {
        const uint2 w = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(s.ptr) + idx);
        x[0] = __uint_as_float(w.x << 16); x[1] = __uint_as_float(w.x & 0xFFFF0000u);
        x[2] = __uint_as_float(w.y << 16); x[3] = __uint_as_float(w.y & 0xFFFF0000u);
    } else if constexpr (V == 4) {
        const float4 t = ns_source_at4(s, idx);
        x[0] = t.x; x[1] = t.y; x[2] = t.z; x[3] = t.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; i++) x[i] = ns_source_at(s, idx + i);
    }
}

template <typename T, int V, int TAPS, int SRC = CONV_ANY>
__global__ void __launch_bounds__(128) ns_short_conv_slide_kernel(const ConvArgs a, int span, int units, int pieces)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, b = blockIdx.z;
    int u = span == 4 ? (int)blockIdx.y : (int)blockIdx.y * 4 + warp, s = 0;
    const bool live = u < units;
    if (!live) u = 0;
    while (s + 1 < a.segments && u >= a.seg[s].heads) { u -= a.seg[s].heads; s++; }
    const ConvSegment& g = a.seg[s];
    const int slot = a.slots[b], pos0 = a.pos[slot];
    const int channels = g.heads * g.hd, taps = g.taps, c = lane * V, ch = u * g.hd + c;
    const bool mine = live && c < g.hd;
    float* hist = g.hist + (int64_t)slot * a.hist_slot_stride + ch;
    const int64_t src0 = (int64_t)b * a.steps * a.src.ld + g.col + ch;
    const int per = CONV_WARP * pieces;
    const int t0 = (span == 4 ? (int)blockIdx.x * 4 + warp : (int)blockIdx.x) * per, t1 = min(t0 + per, a.steps);
    float w[TAPS][V], x[TAPS][V];      // w[n]: weight of the input n tokens back; x[n]: that input
#pragma unroll
    for (int n = 0; n < TAPS; n++)
#pragma unroll
        for (int i = 0; i < V; i++) {
            w[n][i] = mine && n < taps ? __ldg(g.w + (int64_t)(ch + i) * taps + taps - 1 - n) : 0.0f;
            x[n][i] = 0.0f;
        }
    if (mine && t0 < t1) {
        // x[n - 1] becomes x[n] before the first token is loaded
#pragma unroll
        for (int n = 1; n < TAPS; n++) {
            const int tt = t0 - n;
            if (n >= taps || pos0 + tt < 0) continue;
            if (tt >= 0) {
                conv_load<V, SRC>(a.src, src0 + (int64_t)tt * a.src.ld, x[n - 1]);
            } else {
                const float* p = hist + (int64_t)((pos0 + tt) % taps) * channels;
#pragma unroll
                for (int i = 0; i < V; i++) x[n - 1][i] = p[i];
            }
        }
    }
    for (int tp = t0; tp < t1; tp += CONV_WARP) {
        // all inputs of a piece are on their way before the first is used
        float in[CONV_WARP][V];
#pragma unroll
        for (int j = 0; j < CONV_WARP; j++)
            if (mine && tp + j < t1) conv_load<V, SRC>(a.src, src0 + (int64_t)(tp + j) * a.src.ld, in[j]);
#pragma unroll
        for (int j = 0; j < CONV_WARP; j++) {
            const int t = tp + j;
            if (t >= t1) break;
#pragma unroll
            for (int n = TAPS - 1; n > 0; n--)
#pragma unroll
                for (int i = 0; i < V; i++) x[n][i] = x[n - 1][i];
#pragma unroll
            for (int i = 0; i < V; i++) x[0][i] = mine ? in[j][i] : 0.0f;
            float y[V], ss = 0.0f;
#pragma unroll
            for (int i = 0; i < V; i++) {
                float acc = 0.0f;
#pragma unroll
                for (int n = TAPS - 1; n >= 0; n--) acc = fmaf(x[n][i], w[n][i], acc);
                y[i] = mine ? __fdividef(acc, 1.0f + expf(-acc)) : 0.0f;
                ss = fmaf(y[i], y[i], ss);
            }
            float f = 1.0f;
            if (g.unit) f = g.scale / sqrtf(ns_warp_sum(ss) + 1e-6f);
            if (mine) {
                T* out = reinterpret_cast<T*>(g.out) + ((int64_t)b * a.steps + t) * g.out_ld + ch;
                if constexpr (V == 4) {
                    ns_store4(out, make_float4(y[0] * f, y[1] * f, y[2] * f, y[3] * f));
                } else {
#pragma unroll
                    for (int i = 0; i < V; i++) ns_store(out + i, y[i] * f);
                }
            }
        }
    }
    // the warps that read the history have their inputs: the first `span` warps' tokens come first in the step
    if (span == 4) __syncthreads();
    else __syncwarp();
    if (blockIdx.x != 0 || (span == 4 && warp != 0) || !mine || taps < 2) return;
    for (int t = max(0, a.steps - (taps - 1)); t < a.steps; t++) {
        float v[V];
        conv_load<V, SRC>(a.src, src0 + (int64_t)t * a.src.ld, v);
#pragma unroll
        for (int i = 0; i < V; i++) hist[(int64_t)((pos0 + t) % taps) * channels + i] = v[i];
    }
}

template <typename T, int NV>
__global__ void __launch_bounds__(128) ns_short_conv_kernel(const ConvArgs a)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    int u = blockIdx.y, s = 0;
    while (s + 1 < a.segments && u >= a.seg[s].heads) { u -= a.seg[s].heads; s++; }
    const ConvSegment& g = a.seg[s];
    const int b = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int slot = a.slots[b], pos0 = a.pos[slot];
    const int channels = g.heads * g.hd, c0 = u * g.hd, taps = g.taps;
    float* hist = g.hist + (int64_t)slot * a.hist_slot_stride;
    const int t_begin = blockIdx.x * a.chunk, t_end = min(t_begin + a.chunk, a.steps);
    for (int t = t_begin + warp; t < t_end; t += 4) {
        float v[NV];
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int c = j * 32 + lane;
            v[j] = 0.0f;
            if (c < g.hd) {
                float acc = 0.0f;
                for (int n = 0; n < taps; n++) {
                    const int back = taps - 1 - n, tt = t - back;
                    float x = 0.0f;
                    if (tt >= 0) x = ns_source_at(a.src, ((int64_t)b * a.steps + tt) * a.src.ld + g.col + c0 + c);
                    else if (pos0 + tt >= 0) x = hist[(int64_t)((pos0 + tt) % taps) * channels + c0 + c];
                    acc = fmaf(x, __ldg(g.w + (int64_t)(c0 + c) * taps + n), acc);
                }
                v[j] = ns_silu(acc);
                ss = fmaf(v[j], v[j], ss);
            }
        }
        float f = 1.0f;
        if (g.unit) f = g.scale / sqrtf(ns_warp_sum(ss) + 1e-6f);
        T* out = reinterpret_cast<T*>(g.out) + ((int64_t)b * a.steps + t) * g.out_ld + c0;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int c = j * 32 + lane;
            if (c < g.hd) ns_store(out + c, v[j] * f);
        }
    }
    if (blockIdx.x != 0 || taps < 2) return;
    __syncthreads();
    for (int t = max(0, a.steps - (taps - 1)); t < a.steps; t++)
        for (int c = threadIdx.x; c < g.hd; c += blockDim.x)
            hist[(int64_t)((pos0 + t) % taps) * channels + c0 + c] = ns_source_at(a.src, ((int64_t)b * a.steps + t) * a.src.ld + g.col + c0 + c);
}

// ---------------------------------------------------------------------------------------------
// the recurrence, token by token
// ---------------------------------------------------------------------------------------------
struct DeltaArgs {
    const float* q; int q_ld;      // [rows, kv_heads * dim], unit vectors (q scaled)
    const float* k; int k_ld;
    const float* v; int v_ld;      // [rows, heads * vdim]
    NsSource a; int a_col;         // decay projection: column a_col + head, or a_col + head * dim + channel
    NsSource b; int b_col;         // step size projection: column b_col + head
    const float* a_log;            // [heads]
    const float* dt_bias;          // [heads] or [heads * dim]
    float* state;                  // slot 0's [heads, dim, vdim]
    int64_t state_slot_stride;
    const int32_t* slots;
    int heads, kv_heads, dim, vdim, steps;
    float* o; int o_ld;            // [rows, heads * vdim]
};

NS_DEVINL float delta_decay(float a, float dt_bias, float rate) { return expf(-rate * ns_softplus(a + dt_bias)); }

// 8 warps; warp w holds state rows [w * RPW, (w + 1) * RPW), each lane V neighbouring columns of them, in registers.
template <int RPW, int V, bool CHANNEL>
__global__ void __launch_bounds__(256) ns_delta_recurrent_kernel(const DeltaArgs a)
{
    constexpr int DMAX = RPW * 8, VT = 32 * V, DI = (DMAX + 255) / 256;
    __shared__ float sq[3][DMAX], sk[3][DMAX], sg[3][CHANNEL ? DMAX : 1], sv[3][VT], sbeta[3];
    __shared__ float redk[2][8][VT], redq[2][8][VT], redkq[2][8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.x, b = blockIdx.y, v0 = blockIdx.z * VT;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int slot = a.slots[b], kv = head / (a.heads / a.kv_heads);
    const int dim = a.dim, vdim = a.vdim;
    float* S = a.state + (int64_t)slot * a.state_slot_stride + (int64_t)head * dim * vdim;
    const float rate = expf(a.a_log[head]);
    float dtb[DI];
#pragma unroll
    for (int j = 0; j < DI; j++) {
        const int c = j * 256 + tid;
        dtb[j] = CHANNEL ? (c < dim ? a.dt_bias[(int64_t)head * dim + c] : 0.0f) : a.dt_bias[head];
    }
    const int col = v0 + lane * V;
    float st[RPW][V];
    const bool whole = V == 4 && (vdim & 3) == 0;
#pragma unroll
    for (int i = 0; i < RPW; i++) {
        const int r = warp * RPW + i;
#pragma unroll
        for (int j = 0; j < V; j++) st[i][j] = 0.0f;
        if (r < dim && col < vdim) {
            const float* p = S + (int64_t)r * vdim + col;
            if constexpr (V == 4) {
                if (whole) {
                    const float4 t = *reinterpret_cast<const float4*>(p);
                    st[i][0] = t.x; st[i][1] = t.y; st[i][2] = t.z; st[i][3] = t.w;
                    continue;
                }
            }
#pragma unroll
            for (int j = 0; j < V; j++)
                if (col + j < vdim) st[i][j] = p[j];
        }
    }

    float pq[DI], pk[DI], pg[DI], pv = 0.0f, pb = 0.0f;
    auto fetch = [&](int t) {
        const int64_t row = (int64_t)b * a.steps + t;
#pragma unroll
        for (int j = 0; j < DI; j++) {
            const int c = j * 256 + tid;
            pq[j] = pk[j] = pg[j] = 0.0f;
            if (c < dim) {
                pq[j] = a.q[row * a.q_ld + kv * dim + c];
                pk[j] = a.k[row * a.k_ld + kv * dim + c];
                if (CHANNEL) pg[j] = ns_source_at(a.a, row * a.a.ld + a.a_col + head * dim + c);
            }
        }
        if (tid < VT) pv = v0 + tid < vdim ? a.v[row * a.v_ld + head * vdim + v0 + tid] : 0.0f;
        if (tid == 0) {
            pb = ns_source_at(a.b, row * a.b.ld + a.b_col + head);
            if (!CHANNEL) pg[0] = ns_source_at(a.a, row * a.a.ld + a.a_col + head);
        }
    };
    auto put = [&](int s) {
#pragma unroll
        for (int j = 0; j < DI; j++) {
            const int c = j * 256 + tid;
            if (c < DMAX) {
                sq[s][c] = pq[j];
                sk[s][c] = pk[j];
                if (CHANNEL) sg[s][c] = c < dim ? delta_decay(pg[j], dtb[j], rate) : 0.0f;
            }
        }
        if (tid < VT) sv[s][tid] = pv;
        if (tid == 0) {
            sbeta[s] = ns_sigmoid(pb);
            if (!CHANNEL) sg[s][0] = delta_decay(pg[0], dtb[0], rate);
        }
    };
    fetch(0);
    put(0);
    __syncthreads();
    for (int t = 0; t < a.steps; t++) {
        const int s = t % 3, par = t & 1;
        const bool more = t + 1 < a.steps;
        if (more) fetch(t + 1);
        float ak[V], aq[V], akq = 0.0f;
#pragma unroll
        for (int j = 0; j < V; j++) ak[j] = aq[j] = 0.0f;
        const float g1 = CHANNEL ? 0.0f : sg[s][0];
#pragma unroll
        for (int i = 0; i < RPW; i++) {
            const int r = warp * RPW + i;
            const float kk = sk[s][r], qq = sq[s][r], gg = CHANNEL ? sg[s][r] : g1;
            akq = fmaf(kk, qq, akq);
#pragma unroll
            for (int j = 0; j < V; j++) {
                st[i][j] *= gg;
                ak[j] = fmaf(st[i][j], kk, ak[j]);
                aq[j] = fmaf(st[i][j], qq, aq[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < V; j++) {
            redk[par][warp][lane * V + j] = ak[j];
            redq[par][warp][lane * V + j] = aq[j];
        }
        if (lane == 0) redkq[par][warp] = akq;
        if (more) put((t + 1) % 3);
        __syncthreads();
        const float beta = sbeta[s];
        float u[V];
#pragma unroll
        for (int j = 0; j < V; j++) {
            float x = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; w++) x += redk[par][w][lane * V + j];
            u[j] = beta * (sv[s][lane * V + j] - x);
        }
#pragma unroll
        for (int i = 0; i < RPW; i++) {
            const float kk = sk[s][warp * RPW + i];
#pragma unroll
            for (int j = 0; j < V; j++) st[i][j] = fmaf(kk, u[j], st[i][j]);
        }
        if (tid < VT && v0 + tid < vdim) {
            float x = 0.0f, y = 0.0f, kq = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; w++) { x += redk[par][w][tid]; y += redq[par][w][tid]; kq += redkq[par][w]; }
            a.o[((int64_t)b * a.steps + t) * a.o_ld + head * vdim + v0 + tid] = fmaf(beta * (sv[s][tid] - x), kq, y);
        }
    }
#pragma unroll
    for (int i = 0; i < RPW; i++) {
        const int r = warp * RPW + i;
        if (r < dim && col < vdim) {
            float* p = S + (int64_t)r * vdim + col;
            if constexpr (V == 4) {
                if (whole) {
                    *reinterpret_cast<float4*>(p) = make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
                    continue;
                }
            }
#pragma unroll
            for (int j = 0; j < V; j++)
                if (col + j < vdim) p[j] = st[i][j];
        }
    }
}

// ---------------------------------------------------------------------------------------------
// y = o / sqrt(mean(o^2) + eps) * w * act(gate), per row and head
// ---------------------------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ns_gated_norm_kernel(const float* __restrict__ o, int o_ld, const NsSource gate, int gate_col, int act,
                                                            const float* __restrict__ w, float eps, int64_t rows, int heads, int vdim, T* __restrict__ y,
                                                            int64_t y_ld)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int lane = threadIdx.x & 31;
    for (int64_t item = blockIdx.x * 8ll + (threadIdx.x >> 5); item < rows * heads; item += gridDim.x * 8ll) {
        const int64_t row = item / heads;
        const int head = (int)(item - row * heads);
        const float* x = o + row * o_ld + (int64_t)head * vdim;
        const int64_t gi = row * gate.ld + gate_col + head * vdim;
        T* out = y + row * y_ld + (int64_t)head * vdim;
        float ss = 0.0f;
        if (VEC) {
            // up to 128 values: four per lane
            const int c = lane * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f), z = v;
            if (c < vdim) {
                v = *reinterpret_cast<const float4*>(x + c);
                z = ns_source_at4(gate, gi + c);
                ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
            }
            const float inv = 1.0f / sqrtf(ns_warp_sum(ss) / (float)vdim + eps);
            if (c < vdim) {
                const float4 ww = __ldg(reinterpret_cast<const float4*>(w + c));
                const float4 r = act == NS_ACT_SILU ? make_float4(ns_silu(z.x), ns_silu(z.y), ns_silu(z.z), ns_silu(z.w))
                                                    : make_float4(ns_sigmoid(z.x), ns_sigmoid(z.y), ns_sigmoid(z.z), ns_sigmoid(z.w));
                ns_store4(out + c, make_float4(v.x * inv * ww.x * r.x, v.y * inv * ww.y * r.y, v.z * inv * ww.z * r.z, v.w * inv * ww.w * r.w));
            }
        } else {
            for (int c = lane; c < vdim; c += 32) ss = fmaf(x[c], x[c], ss);
            const float inv = 1.0f / sqrtf(ns_warp_sum(ss) / (float)vdim + eps);
            for (int c = lane; c < vdim; c += 32) {
                const float z = ns_source_at(gate, gi + c);
                ns_store(out + c, x[c] * inv * w[c] * (act == NS_ACT_SILU ? ns_silu(z) : ns_sigmoid(z)));
            }
        }
        if (head == heads - 1)
            for (int64_t c = (int64_t)heads * vdim + lane; c < y_ld; c += 32) ns_store(y + row * y_ld + c, 0.0f);
    }
}

// The same for one wide head (the whole row): a CTA per row, up to 8 groups of four values per thread in registers.
template <typename T, int Q>
__global__ void __launch_bounds__(256) ns_gated_norm_row_kernel(const float* __restrict__ o, int o_ld, const NsSource gate, int gate_col, int act,
                                                                const float* __restrict__ w, float eps, int n, T* __restrict__ y, int64_t y_ld)
{
    __shared__ float red[8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int64_t row = blockIdx.x;
    float4 v[Q], z[Q];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int c = (threadIdx.x + 256 * i) * 4;
        v[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= n) continue;
        v[i] = *reinterpret_cast<const float4*>(o + row * o_ld + c);
        z[i] = ns_source_at4(gate, row * gate.ld + gate_col + c);
    }
#pragma unroll
    for (int i = 0; i < Q; i++) { ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss); ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss); }
    const float inv = 1.0f / sqrtf(ns_cta_sum(ss, red) / (float)n + eps);
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int c = (threadIdx.x + 256 * i) * 4;
        if (c >= n) continue;
        const float4 ww = __ldg(reinterpret_cast<const float4*>(w + c));
        const float4 r = act == NS_ACT_SILU ? make_float4(ns_silu(z[i].x), ns_silu(z[i].y), ns_silu(z[i].z), ns_silu(z[i].w))
                                            : make_float4(ns_sigmoid(z[i].x), ns_sigmoid(z[i].y), ns_sigmoid(z[i].z), ns_sigmoid(z[i].w));
        ns_store4(y + row * y_ld + c, make_float4(v[i].x * inv * ww.x * r.x, v[i].y * inv * ww.y * r.y, v[i].z * inv * ww.z * r.z, v[i].w * inv * ww.w * r.w));
    }
    for (int c = n + threadIdx.x; c < y_ld; c += 256) ns_store(y + row * y_ld + c, 0.0f);
}

template <int RPW, int V>
int launch_recurrent(NsDevice* d, const DeltaArgs& a, int batch, bool channel)
{
    const dim3 grid((unsigned)a.heads, (unsigned)batch, (unsigned)((a.vdim + 32 * V - 1) / (32 * V)));
    auto k = channel ? ns_delta_recurrent_kernel<RPW, V, true> : ns_delta_recurrent_kernel<RPW, V, false>;
    NS_CUDA(ns_launch_plain(k, grid, dim3(256), 0, d->stream, a));
    return NS_OK;
}

template <int V>
int launch_recurrent_rows(NsDevice* d, const DeltaArgs& a, int batch, bool channel)
{
    if (a.dim <= 32) return launch_recurrent<4, V>(d, a, batch, channel);
    if (a.dim <= 64) return launch_recurrent<8, V>(d, a, batch, channel);
    if (a.dim <= 128) return launch_recurrent<16, V>(d, a, batch, channel);
    return launch_recurrent<32, V>(d, a, batch, channel);
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }

extern "C" int ns_short_conv(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int segments, const int64_t* fields, const float* scales,
                             int64_t hist_slot_stride, uint64_t slots, uint64_t pos, int batch, int steps, int out_dtype)
{
    NS_ENTER(h);
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype), NS_ERR_ARGUMENT, "ns_short_conv: bad source");
    NS_REQUIRE(fields && scales && slots && pos && batch > 0 && steps > 0 && segments >= 1 && segments <= CONV_MAX_SEGMENTS, NS_ERR_ARGUMENT,
               "ns_short_conv: bad argument");
    NS_REQUIRE(out_dtype == NS_F32 || out_dtype == NS_BF16, NS_ERR_ARGUMENT, "ns_short_conv: bad output type");
    ConvArgs a;
    a.src = ns_source(src, splits, src_dtype, (int64_t)batch * steps, src_ld);
    a.segments = segments;
    a.hist_slot_stride = hist_slot_stride;
    a.slots = reinterpret_cast<const int32_t*>(slots);
    a.pos = reinterpret_cast<const int32_t*>(pos);
    a.steps = steps;
    a.chunk = CONV_CHUNK;
    int units = 0, widest = 1;
    for (int i = 0; i < segments; i++) {
        const int64_t* f = fields + i * 9;
        ConvSegment& s = a.seg[i];
        s.col = (int)f[0]; s.heads = (int)f[1]; s.hd = (int)f[2]; s.taps = (int)f[3]; s.unit = (int)f[4];
        s.w = reinterpret_cast<const float*>(f[5]);
        s.hist = reinterpret_cast<float*>(f[6]);
        s.out = reinterpret_cast<void*>(f[7]);
        s.out_ld = (int)f[8];
        s.scale = scales[i];
        NS_REQUIRE(s.heads > 0 && s.hd > 0 && s.taps > 0 && s.w && s.out && (s.hist || s.taps == 1), NS_ERR_ARGUMENT, "ns_short_conv: bad segment %d", i);
        NS_REQUIRE(s.hd <= 512, NS_ERR_ARGUMENT, "ns_short_conv: heads of %d channels (at most 512)", s.hd);
        NS_REQUIRE(s.col >= 0 && s.col + s.heads * s.hd <= src_ld && s.out_ld >= s.heads * s.hd, NS_ERR_ARGUMENT, "ns_short_conv: segment %d does not fit", i);
        units += s.heads;
        if (s.hd > widest) widest = s.hd;
        // the first chunk is the one that reads the history
        if (s.taps - 1 > a.chunk) a.chunk = s.taps - 1;
    }
    const dim3 grid((unsigned)((steps + a.chunk - 1) / a.chunk), (unsigned)units, (unsigned)batch);
    auto launch = [&](auto k) -> int {
        NS_CUDA(ns_launch_plain(k, grid, dim3(128), 0, d->stream, a));
        return NS_OK;
    };
    // the sliding kernel: heads of up to 128 channels, up to 8 taps (its first chunk must hold all tokens that read the history)
    int most_taps = 1, v = widest <= 32 ? 1 : (widest <= 64 ? 2 : 4);
    for (int i = 0; i < segments; i++) {
        const ConvSegment& s = a.seg[i];
        if (s.taps > most_taps) most_taps = s.taps;
        if (s.hd % v != 0 || (v == 4 && ((s.col | s.out_ld) & 3) != 0)) v = 0;
        if (v == 4 && (reinterpret_cast<uintptr_t>(s.out) & 15) != 0) v = 0;
        if (v == 0) break;
    }
    if (v == 4 && ((src_ld & 3) != 0 || (src & 15) != 0)) v = 0;
    if (v != 0 && widest <= 128 && most_taps <= 8) {
        const int span = steps <= CONV_WARP ? 1 : 4;
        // a prompt's warps slide over four pieces: their weights and addresses are set up once
        const int pieces = steps >= 256 ? 4 : 1;
        const int per = span * CONV_WARP * pieces;
        const dim3 sgrid((unsigned)((steps + per - 1) / per), (unsigned)(span == 4 ? units : (units + 3) / 4), (unsigned)batch);
        auto slide = [&](auto k) -> int {
            NS_CUDA(ns_launch_plain(k, sgrid, dim3(128), 0, d->stream, a, span, units, pieces));
            return NS_OK;
        };
        auto pick = [&](auto zero) -> int {
            using T = decltype(zero);
            if (v == 4 && most_taps <= 4 && splits == 1 && steps > CONV_WARP)
                return src_dtype == NS_F32 ? slide(ns_short_conv_slide_kernel<T, 4, 4, CONV_F32>) : slide(ns_short_conv_slide_kernel<T, 4, 4, CONV_BF16>);
            if (most_taps <= 4)
                return v == 1 ? slide(ns_short_conv_slide_kernel<T, 1, 4>) : (v == 2 ? slide(ns_short_conv_slide_kernel<T, 2, 4>) : slide(ns_short_conv_slide_kernel<T, 4, 4>));
            return v == 1 ? slide(ns_short_conv_slide_kernel<T, 1, 8>) : (v == 2 ? slide(ns_short_conv_slide_kernel<T, 2, 8>) : slide(ns_short_conv_slide_kernel<T, 4, 8>));
        };
        return out_dtype == NS_F32 ? pick(float(0)) : pick(uint16_t(0));
    }
    if (out_dtype == NS_F32) {
        if (widest <= 64) return launch(ns_short_conv_kernel<float, 2>);
        if (widest <= 128) return launch(ns_short_conv_kernel<float, 4>);
        return launch(ns_short_conv_kernel<float, 16>);
    }
    if (widest <= 64) return launch(ns_short_conv_kernel<uint16_t, 2>);
    if (widest <= 128) return launch(ns_short_conv_kernel<uint16_t, 4>);
    return launch(ns_short_conv_kernel<uint16_t, 16>);
}

extern "C" int ns_delta_recurrent(ns_device_t h, uint64_t q, int q_ld, uint64_t k, int k_ld, uint64_t v, int v_ld, uint64_t a_src, int a_splits, int a_ld,
                                  int a_col, uint64_t b_src, int b_splits, int b_ld, int b_col, uint64_t a_log, uint64_t dt_bias, int per_channel,
                                  uint64_t state, int64_t state_slot_stride, uint64_t slots, int batch, int steps, int heads, int kv_heads, int dim, int vdim,
                                  uint64_t o, int o_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(q && k && v && a_log && dt_bias && state && slots && o && batch > 0 && steps > 0, NS_ERR_ARGUMENT, "ns_delta_recurrent: bad argument");
    NS_REQUIRE(ns_source_ok(a_src, a_splits, NS_F32) && ns_source_ok(b_src, b_splits, NS_F32), NS_ERR_ARGUMENT, "ns_delta_recurrent: bad source");
    NS_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0, NS_ERR_ARGUMENT, "ns_delta_recurrent: %d heads do not divide over %d key heads", heads, kv_heads);
    NS_REQUIRE(dim > 0 && dim <= 256 && vdim > 0, NS_ERR_ARGUMENT, "ns_delta_recurrent: key size %d (at most 256)", dim);
    NS_REQUIRE(batch <= 65535, NS_ERR_ARGUMENT, "ns_delta_recurrent: batch %d", batch);
    DeltaArgs a;
    const int64_t rows = (int64_t)batch * steps;
    a.q = reinterpret_cast<const float*>(q); a.q_ld = q_ld;
    a.k = reinterpret_cast<const float*>(k); a.k_ld = k_ld;
    a.v = reinterpret_cast<const float*>(v); a.v_ld = v_ld;
    a.a = ns_source(a_src, a_splits, NS_F32, rows, a_ld); a.a_col = a_col;
    a.b = ns_source(b_src, b_splits, NS_F32, rows, b_ld); a.b_col = b_col;
    a.a_log = reinterpret_cast<const float*>(a_log);
    a.dt_bias = reinterpret_cast<const float*>(dt_bias);
    a.state = reinterpret_cast<float*>(state);
    a.state_slot_stride = state_slot_stride;
    a.slots = reinterpret_cast<const int32_t*>(slots);
    a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim; a.steps = steps;
    a.o = reinterpret_cast<float*>(o); a.o_ld = o_ld;
    if (vdim <= 32) return launch_recurrent_rows<1>(d, a, batch, per_channel != 0);
    if (vdim <= 64) return launch_recurrent_rows<2>(d, a, batch, per_channel != 0);
    return launch_recurrent_rows<4>(d, a, batch, per_channel != 0);
}

extern "C" int ns_gated_norm(ns_device_t h, uint64_t o, int o_ld, uint64_t gate, int splits, int gate_dtype, int gate_ld, int gate_col, int act, uint64_t w,
                             float eps, int64_t rows, int heads, int vdim, int out_dtype, uint64_t y, int y_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(o && w && y && rows > 0 && heads > 0 && vdim > 0 && o_ld >= heads * vdim && y_ld >= heads * vdim, NS_ERR_ARGUMENT, "ns_gated_norm: bad argument");
    NS_REQUIRE(ns_source_ok(gate, splits, gate_dtype) && gate_col >= 0 && gate_ld >= gate_col + heads * vdim, NS_ERR_ARGUMENT, "ns_gated_norm: bad gate");
    NS_REQUIRE(act == NS_ACT_SILU || act == NS_ACT_SIGMOID, NS_ERR_ARGUMENT, "ns_gated_norm: unknown activation %d", act);
    NS_REQUIRE(out_dtype == NS_F32 || out_dtype == NS_BF16, NS_ERR_ARGUMENT, "ns_gated_norm: bad output type");
    const NsSource g = ns_source(gate, splits, gate_dtype, rows, gate_ld);
    const bool aligned = ((vdim | o_ld | gate_ld | gate_col | y_ld) & 3) == 0 && ((o | gate | w | y) & 15) == 0 && (g.slab & 3) == 0, vec = aligned && vdim <= 128;
    if (aligned && heads == 1 && vdim > 128 && vdim <= 8192) {
        auto row = [&](auto zero, auto kernel) -> int {
            using T = decltype(zero);
            NS_CUDA(ns_launch_plain(kernel, dim3((unsigned)rows), dim3(256), 0, d->stream, reinterpret_cast<const float*>(o), o_ld, g, gate_col, act,
                                    reinterpret_cast<const float*>(w), eps, vdim, reinterpret_cast<T*>(y), (int64_t)y_ld));
            return NS_OK;
        };
        auto pick = [&](auto zero) -> int {
            using T = decltype(zero);
            if (vdim <= 2048) return row(zero, ns_gated_norm_row_kernel<T, 2>);
            if (vdim <= 4096) return row(zero, ns_gated_norm_row_kernel<T, 4>);
            return row(zero, ns_gated_norm_row_kernel<T, 8>);
        };
        return out_dtype == NS_F32 ? pick(float(0)) : pick(uint16_t(0));
    }
    const int64_t blocks = (rows * heads + 7) / 8, most = (int64_t)d->sm_count * 32;
    const dim3 grid((unsigned)(blocks < most ? blocks : most));
    if (out_dtype == NS_F32) {
        auto k = vec ? ns_gated_norm_kernel<float, true> : ns_gated_norm_kernel<float, false>;
        NS_CUDA(ns_launch_plain(k, grid, dim3(256), 0, d->stream, reinterpret_cast<const float*>(o), o_ld, g, gate_col, act, reinterpret_cast<const float*>(w), eps,
                                rows, heads, vdim, reinterpret_cast<float*>(y), (int64_t)y_ld));
    } else {
        auto k = vec ? ns_gated_norm_kernel<uint16_t, true> : ns_gated_norm_kernel<uint16_t, false>;
        NS_CUDA(ns_launch_plain(k, grid, dim3(256), 0, d->stream, reinterpret_cast<const float*>(o), o_ld, g, gate_col, act, reinterpret_cast<const float*>(w), eps,
                                rows, heads, vdim, reinterpret_cast<uint16_t*>(y), (int64_t)y_ld));
    }
    return NS_OK;
}
