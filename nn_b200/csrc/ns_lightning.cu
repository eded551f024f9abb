// Linear attention with a fixed decay per head: S_t = d S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, with q, k and v read straight from
// one product (the activation is applied here) and the state S [dim, vdim] in 32-bit floats in the sequence's slot.
//
//   ns_lightning_recurrent  token by token, for the few tokens of a decoding step and for float32 models
//   ns_lightning_chunked    a prompt's portion, 64 tokens at a time on the tensor cores
//
// In a chunk of n tokens with the state S before it
//     o_i = d^(i+1) S^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j,      S <- d^n S + sum_j d^(n-1-j) k_j v_j^T,
// so no power is ever formed with a negative exponent.  q, k and v are bf16 there (activations); what is made from the decays and
// the state is split into two bf16 halves (16 mantissa bits) against them, with 32-bit sums.
//
// When a pass has few sequences, its tokens are cut into segments that run side by side: one kernel sums every segment's own
// writes, a second carries the state through them, a third does the work above from each segment's state.
#include <math.h>

#include "ns_mma.cuh"
#include "ns_seq.cuh"

namespace {

struct LightningArgs {
    NsSource src;                  // [rows, ld]: q, k, v before the activation
    int q_col, k_col, v_col;       // element (row, head, c) at column col + head * size + c
    const float* decay;            // [heads]
    const float* decay_log2;       // [heads], finite
    float* state;                  // slot 0's [heads, dim, vdim]
    int64_t state_slot_stride;
    const int32_t* slots;
    int heads, dim, vdim, steps;
    float* o; int o_ld;            // [rows, heads * vdim]
    // segments of `seg_len` tokens (a multiple of the chunk) when segs > 1
    int segs, seg_len;
    float* seg_state;              // [batch, segs, heads, dim, vdim]: a segment's own writes, then the state before it
};

// ---------------------------------------------------------------------------------------------
// token by token: 8 warps; warp w holds state rows [w * RPW, (w + 1) * RPW), each lane V neighbouring columns of them
// ---------------------------------------------------------------------------------------------
template <int RPW, int V>
__global__ void __launch_bounds__(256) ns_lightning_recurrent_kernel(const LightningArgs a)
{
    constexpr int DMAX = RPW * 8, VT = 32 * V;
    __shared__ float sq[2][DMAX], sk[2][DMAX], sv[2][VT], red[2][8][VT];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.x, b = blockIdx.y, v0 = blockIdx.z * VT;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dim = a.dim, vdim = a.vdim, col = v0 + lane * V;
    const float d = a.decay[head];
    float* S = a.state + (int64_t)a.slots[b] * a.state_slot_stride + (int64_t)head * dim * vdim;
    const bool whole = V == 4 && (vdim & 3) == 0;

    // one element of q, k and v of a token per thread
    float pq = 0.0f, pk = 0.0f, pv = 0.0f;
    auto fetch = [&](int t) {
        const int64_t at = ((int64_t)b * a.steps + t) * a.src.ld;
        if (tid < dim) {
            pq = ns_source_at(a.src, at + a.q_col + head * dim + tid);
            pk = ns_source_at(a.src, at + a.k_col + head * dim + tid);
        }
        if (tid < VT && v0 + tid < vdim) pv = ns_source_at(a.src, at + a.v_col + head * vdim + v0 + tid);
    };
    auto put = [&](int s) {
        if (tid < DMAX) {
            sq[s][tid] = tid < dim ? ns_silu(pq) : 0.0f;
            sk[s][tid] = tid < dim ? ns_silu(pk) : 0.0f;
        }
        if (tid < VT) sv[s][tid] = v0 + tid < vdim ? ns_silu(pv) : 0.0f;
    };
    fetch(0);
    float st[RPW][V];
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
    put(0);
    __syncthreads();
    for (int t = 0; t < a.steps; t++) {
        const int s = t & 1;
        const bool more = t + 1 < a.steps;
        if (more) fetch(t + 1);
        float v[V], acc[V];
#pragma unroll
        for (int j = 0; j < V; j++) { v[j] = sv[s][lane * V + j]; acc[j] = 0.0f; }
#pragma unroll
        for (int i = 0; i < RPW; i++) {
            const float kk = sk[s][warp * RPW + i], qq = sq[s][warp * RPW + i];
#pragma unroll
            for (int j = 0; j < V; j++) {
                st[i][j] = fmaf(st[i][j], d, kk * v[j]);
                acc[j] = fmaf(st[i][j], qq, acc[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < V; j++) red[s][warp][lane * V + j] = acc[j];
        if (more) put(s ^ 1);
        __syncthreads();
        if (tid < VT && v0 + tid < vdim) {
            float x = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; w++) x += red[s][w][tid];
            a.o[((int64_t)b * a.steps + t) * a.o_ld + head * vdim + v0 + tid] = x;
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
// chunks of 64 tokens
// ---------------------------------------------------------------------------------------------
constexpr int LC = 64;        // tokens per chunk
constexpr int LDV = 64;       // value columns per CTA

template <int DK>
struct LightningSmem {
    static constexpr int LK = DK + 8, LV = LDV + 8;                   // row lengths that keep ldmatrix free of bank conflicts
    static constexpr int Q = 0, K = Q + LC * LK * 2, V = K + LC * LK * 2, VH = V + LC * LV * 2, VL = VH + LC * LV * 2, SH = VL + LC * LV * 2,
                         SL = SH + DK * LV * 2, TOTAL = SL + DK * LV * 2;
};

// the bf16 halves of two values: x = hi + lo up to 2^-17 of x
NS_DEVINL void halves(float x, float y, uint32_t& hi, uint32_t& lo)
{
    hi = ns_pack_bf16x2(x, y);
    lo = ns_pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}
NS_DEVINL void st_shared_v2(uint32_t addr, uint32_t a, uint32_t b) { asm volatile("st.shared.v2.b32 [%0], {%1, %2};" ::"r"(addr), "r"(a), "r"(b) : "memory"); }
NS_DEVINL void st_shared_1(uint32_t addr, uint32_t a) { asm volatile("st.shared.b32 [%0], %1;" ::"r"(addr), "r"(a) : "memory"); }
// z / (1 + e^-z); what it makes is rounded to bf16
NS_DEVINL float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// Up to N groups of four neighbouring channels of the tile [64, width] at column `col` of a row, activated, as bf16 pairs.  Group x of a
// thread is element tid + 256 x.  Rows past n and channels past size are zero.
template <int WIDTH, int N>
NS_DEVINL void load_silu(const NsSource& s, int64_t row0, int n, int col, int first, int size, bool vec, int tid, uint2 (&out)[N])
{
    constexpr int QUADS = WIDTH / 4;
    float4 x[N];
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int e = tid + 256 * i, t = e / QUADS, c = first + (e % QUADS) * 4;
        x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < n && c < size) {
            const int64_t at = (row0 + t) * s.ld + col + c;
            if (vec) {
                x[i] = ns_source_at4(s, at);
            } else {
                x[i].x = ns_source_at(s, at);
                if (c + 1 < size) x[i].y = ns_source_at(s, at + 1);
                if (c + 2 < size) x[i].z = ns_source_at(s, at + 2);
                if (c + 3 < size) x[i].w = ns_source_at(s, at + 3);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < N; i++)
        out[i] = make_uint2(ns_pack_bf16x2(silu_fast(x[i].x), silu_fast(x[i].y)), ns_pack_bf16x2(silu_fast(x[i].z), silu_fast(x[i].w)));
}

// WRITES_ONLY: a segment's own writes (no queries, no outputs), left in seg_state.
template <int DK, bool WRITES_ONLY>
__global__ void __launch_bounds__(256, 2) ns_lightning_chunk_kernel(const LightningArgs a, int vec)
{
    using L = LightningSmem<DK>;
    constexpr int ROW_TILES = DK / 16, COL_PARTS = 8 / ROW_TILES, NS = LDV / 8 / COL_PARTS;     // state tile of a warp: 16 rows, NS x 8 columns
    extern __shared__ __align__(16) uint8_t lc_smem[];
    const uint32_t base = ns_smem_u32(lc_smem), sQ = base + L::Q, sK = base + L::K, sV = base + L::V, sVH = base + L::VH, sVL = base + L::VL,
                   sSH = base + L::SH, sSL = base + L::SL;
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.x, b = blockIdx.y, seg = blockIdx.z % a.segs, v0 = (blockIdx.z / a.segs) * LDV;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int dim = a.dim, vdim = a.vdim;
    const float ld2 = a.decay_log2[head];
    const int64_t per_head = (int64_t)dim * vdim;
    float* S = a.segs > 1 ? a.seg_state + (((int64_t)b * a.segs + seg) * a.heads + head) * per_head
                          : a.state + (int64_t)a.slots[b] * a.state_slot_stride + head * per_head;
    const int begin = seg * a.seg_len, end = min(a.steps, begin + a.seg_len);
    const int sr = (warp % ROW_TILES) * 16, sc = (warp / ROW_TILES) * NS * 8;

    float st[NS][4];
#pragma unroll
    for (int j = 0; j < NS; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g + (e >> 1) * 8, c = v0 + sc + j * 8 + t4 * 2 + (e & 1);
            st[j][e] = !WRITES_ONLY && r < dim && c < vdim ? S[(int64_t)r * vdim + c] : 0.0f;
        }

    for (int c0 = begin; c0 < end; c0 += LC) {
        const int n = min(LC, end - c0);
        const int64_t row0 = (int64_t)b * a.steps + c0;
        {
            constexpr int NQ = LC * DK / 1024, NVG = LC * LDV / 1024;
            uint2 kx[NQ], qx[WRITES_ONLY ? 1 : NQ], vx[NVG];
            load_silu<DK, NQ>(a.src, row0, n, a.k_col + head * dim, 0, dim, vec, tid, kx);
            if constexpr (!WRITES_ONLY) load_silu<DK, NQ>(a.src, row0, n, a.q_col + head * dim, 0, dim, vec, tid, qx);
            load_silu<LDV, NVG>(a.src, row0, n, a.v_col + head * vdim, v0, vdim, vec, tid, vx);
#pragma unroll
            for (int i = 0; i < NQ; i++) {
                const int e = tid + 256 * i, t = e / (DK / 4), c = (e % (DK / 4)) * 4;
                st_shared_v2(sK + (t * L::LK + c) * 2, kx[i].x, kx[i].y);
                if constexpr (!WRITES_ONLY) st_shared_v2(sQ + (t * L::LK + c) * 2, qx[i].x, qx[i].y);
            }
#pragma unroll
            for (int i = 0; i < NVG; i++) {
                const int e = tid + 256 * i, t = e / (LDV / 4), c = (e % (LDV / 4)) * 4;
                const uint32_t at = (t * L::LV + c) * 2;
                if constexpr (!WRITES_ONLY) st_shared_v2(sV + at, vx[i].x, vx[i].y);
                // the values as the state at the chunk's end sees them
                const float w = t < n ? ns_exp2((float)(n - 1 - t) * ld2) : 0.0f;
                uint32_t h0, l0, h1, l1;
                halves(__uint_as_float(vx[i].x << 16) * w, __uint_as_float(vx[i].x & 0xFFFF0000u) * w, h0, l0);
                halves(__uint_as_float(vx[i].y << 16) * w, __uint_as_float(vx[i].y & 0xFFFF0000u) * w, h1, l1);
                st_shared_v2(sVH + at, h0, h1);
                st_shared_v2(sVL + at, l0, l1);
            }
            if constexpr (!WRITES_ONLY) {
#pragma unroll
                for (int j = 0; j < NS; j++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        uint32_t hi, lo;
                        halves(st[j][2 * h], st[j][2 * h + 1], hi, lo);
                        const uint32_t at = ((sr + g + h * 8) * L::LV + sc + j * 8 + t4 * 2) * 2;
                        st_shared_1(sSH + at, hi);
                        st_shared_1(sSL + at, lo);
                    }
            }
        }
        __syncthreads();
        if constexpr (!WRITES_ONLY) {
            // 16 rows x 32 value columns per warp
            const int r0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;
            float acc[4][4];
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[j][e] = 0.0f;
            uint32_t qf[DK / 16][4];
#pragma unroll
            for (int k = 0; k < DK / 16; k++) {
                ns_ldsm4(qf[k], ns_addr_a(sQ, L::LK, r0, k * 16, lane));
                uint32_t bh[2][4], bl[2][4];
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    ns_ldsm4_t(bh[j], ns_addr_bt(sSH, L::LV, k * 16, n0 + j * 16, lane));
                    ns_ldsm4_t(bl[j], ns_addr_bt(sSL, L::LV, k * 16, n0 + j * 16, lane));
                }
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], qf[k], bh[j >> 1][2 * (j & 1)], bh[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], qf[k], bl[j >> 1][2 * (j & 1)], bl[j >> 1][2 * (j & 1) + 1]);
            }
            const float f0 = ns_exp2((float)(r0 + g + 1) * ld2), f1 = ns_exp2((float)(r0 + g + 9) * ld2);
#pragma unroll
            for (int j = 0; j < 4; j++) { acc[j][0] *= f0; acc[j][1] *= f0; acc[j][2] *= f1; acc[j][3] *= f1; }
            for (int kb = 0; kb <= r0; kb += 16) {
                float s[2][4];
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[j][e] = 0.0f;
#pragma unroll
                for (int k = 0; k < DK / 16; k++) {
                    uint32_t bf[4];
                    ns_ldsm4(bf, ns_addr_b(sK, L::LK, kb, k * 16, lane));
                    ns_mma_bf16(s[0], qf[k], bf[0], bf[1]);
                    ns_mma_bf16(s[1], qf[k], bf[2], bf[3]);
                }
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int back = r0 + g + (e >> 1) * 8 - (kb + j * 8 + t4 * 2 + (e & 1));
                        s[j][e] = back >= 0 ? s[j][e] * ns_exp2((float)back * ld2) : 0.0f;
                    }
                uint32_t ph[4], pl[4];
                halves(s[0][0], s[0][1], ph[0], pl[0]);
                halves(s[0][2], s[0][3], ph[1], pl[1]);
                halves(s[1][0], s[1][1], ph[2], pl[2]);
                halves(s[1][2], s[1][3], ph[3], pl[3]);
                uint32_t vf[2][4];
#pragma unroll
                for (int j = 0; j < 2; j++) ns_ldsm4_t(vf[j], ns_addr_bt(sV, L::LV, kb, n0 + j * 16, lane));
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], ph, vf[j >> 1][2 * (j & 1)], vf[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], pl, vf[j >> 1][2 * (j & 1)], vf[j >> 1][2 * (j & 1) + 1]);
            }
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int r = r0 + g + h * 8;
                if (r >= n) continue;
                float* o = a.o + (row0 + r) * a.o_ld + (int64_t)head * vdim;
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int c = v0 + n0 + j * 8 + t4 * 2;
                    if ((vdim & 1) == 0 && (a.o_ld & 1) == 0) {
                        if (c < vdim) *reinterpret_cast<float2*>(o + c) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
                    } else {
                        if (c < vdim) o[c] = acc[j][2 * h];
                        if (c + 1 < vdim) o[c + 1] = acc[j][2 * h + 1];
                    }
                }
            }
        }
        // the state after the chunk
        const float fn = ns_exp2((float)n * ld2);
#pragma unroll
        for (int j = 0; j < NS; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) st[j][e] *= fn;
#pragma unroll
        for (int k = 0; k < LC; k += 16) {
            uint32_t af[4];
            ns_ldsm4_t(af, ns_addr_at(sK, L::LK, sr, k, lane));
#pragma unroll
            for (int j = 0; j < NS; j += 2) {
                uint32_t bh[4], bl[4];
                ns_ldsm4_t(bh, ns_addr_bt(sVH, L::LV, k, sc + j * 8, lane));
                ns_ldsm4_t(bl, ns_addr_bt(sVL, L::LV, k, sc + j * 8, lane));
                ns_mma_bf16(st[j], af, bh[0], bh[1]);
                ns_mma_bf16(st[j + 1], af, bh[2], bh[3]);
                ns_mma_bf16(st[j], af, bl[0], bl[1]);
                ns_mma_bf16(st[j + 1], af, bl[2], bl[3]);
            }
        }
        __syncthreads();
    }
    if (!WRITES_ONLY && a.segs > 1) return;          // the states at the segments' ends are known already
#pragma unroll
    for (int j = 0; j < NS; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = sr + g + (e >> 1) * 8, c = v0 + sc + j * 8 + t4 * 2 + (e & 1);
            if (r < dim && c < vdim) S[(int64_t)r * vdim + c] = st[j][e];
        }
}

// the segments' writes become the states before them; the state after the last goes to the slot
__global__ void __launch_bounds__(256) ns_lightning_carry_kernel(const LightningArgs a)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.y, b = blockIdx.z;
    const int64_t per_head = (int64_t)a.dim * a.vdim, i = (int64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= per_head) return;
    float* S = a.state + (int64_t)a.slots[b] * a.state_slot_stride + head * per_head + i;
    float x = *S;
    for (int s = 0; s < a.segs; s++) {
        float* p = a.seg_state + (((int64_t)b * a.segs + s) * a.heads + head) * per_head + i;
        const int len = min(a.steps, (s + 1) * a.seg_len) - s * a.seg_len;
        const float own = *p;
        *p = x;
        x = fmaf(x, exp2f((float)len * a.decay_log2[head]), own);
    }
    *S = x;
}

template <int RPW, int V>
int launch_recurrent(NsDevice* d, const LightningArgs& a, int batch)
{
    const dim3 grid((unsigned)a.heads, (unsigned)batch, (unsigned)((a.vdim + 32 * V - 1) / (32 * V)));
    NS_CUDA(ns_launch_plain(ns_lightning_recurrent_kernel<RPW, V>, grid, dim3(256), 0, d->stream, a));
    return NS_OK;
}
template <int V>
int launch_recurrent_rows(NsDevice* d, const LightningArgs& a, int batch)
{
    if (a.dim <= 32) return launch_recurrent<4, V>(d, a, batch);
    if (a.dim <= 64) return launch_recurrent<8, V>(d, a, batch);
    if (a.dim <= 128) return launch_recurrent<16, V>(d, a, batch);
    return launch_recurrent<32, V>(d, a, batch);
}

template <int DK, bool WRITES_ONLY>
int launch_chunk_kernel(NsDevice* d, const LightningArgs& a, int batch, int vec)
{
    constexpr int smem = LightningSmem<DK>::TOTAL;
    auto k = ns_lightning_chunk_kernel<DK, WRITES_ONLY>;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    const dim3 grid((unsigned)a.heads, (unsigned)batch, (unsigned)((a.vdim + LDV - 1) / LDV * a.segs));
    NS_CUDA(ns_launch_plain(k, grid, dim3(256), (size_t)smem, d->stream, a, vec));
    return NS_OK;
}

template <int DK>
int launch_chunked(NsDevice* d, const LightningArgs& a, int batch, int vec)
{
    if (a.segs > 1) {
        int rc = launch_chunk_kernel<DK, true>(d, a, batch, vec);
        if (rc != NS_OK) return rc;
        const dim3 grid((unsigned)(((int64_t)a.dim * a.vdim + 255) / 256), (unsigned)a.heads, (unsigned)batch);
        NS_CUDA(ns_launch_plain(ns_lightning_carry_kernel, grid, dim3(256), 0, d->stream, a));
    }
    return launch_chunk_kernel<DK, false>(d, a, batch, vec);
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }

static int lightning_args(LightningArgs& a, const char* who, uint64_t src, int splits, int src_dtype, int src_ld, int q_col, int k_col, int v_col, uint64_t decay,
                          uint64_t decay_log2, uint64_t state, int64_t state_slot_stride, uint64_t slots, int batch, int steps, int heads, int dim, int vdim,
                          uint64_t o, int o_ld)
{
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype), NS_ERR_ARGUMENT, "%s: bad source", who);
    NS_REQUIRE(decay && decay_log2 && state && slots && o && batch > 0 && batch <= 65535 && steps > 0, NS_ERR_ARGUMENT, "%s: bad argument", who);
    NS_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && o_ld >= heads * vdim, NS_ERR_ARGUMENT, "%s: bad sizes", who);
    NS_REQUIRE(q_col >= 0 && k_col >= 0 && v_col >= 0 && q_col + heads * dim <= src_ld && k_col + heads * dim <= src_ld && v_col + heads * vdim <= src_ld,
               NS_ERR_ARGUMENT, "%s: the source has too few columns", who);
    a.src = ns_source(src, splits, src_dtype, (int64_t)batch * steps, src_ld);
    a.q_col = q_col; a.k_col = k_col; a.v_col = v_col;
    a.decay = reinterpret_cast<const float*>(decay);
    a.decay_log2 = reinterpret_cast<const float*>(decay_log2);
    a.state = reinterpret_cast<float*>(state);
    a.state_slot_stride = state_slot_stride;
    a.slots = reinterpret_cast<const int32_t*>(slots);
    a.heads = heads; a.dim = dim; a.vdim = vdim; a.steps = steps;
    a.o = reinterpret_cast<float*>(o);
    a.o_ld = o_ld;
    a.segs = 1; a.seg_len = (steps + LC - 1) / LC * LC;
    a.seg_state = nullptr;
    return NS_OK;
}

extern "C" int ns_lightning_recurrent(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int q_col, int k_col, int v_col, uint64_t decay,
                                      uint64_t decay_log2, uint64_t state, int64_t state_slot_stride, uint64_t slots, int batch, int steps, int heads, int dim,
                                      int vdim, uint64_t o, int o_ld)
{
    NS_ENTER(h);
    LightningArgs a;
    int rc = lightning_args(a, "ns_lightning_recurrent", src, splits, src_dtype, src_ld, q_col, k_col, v_col, decay, decay_log2, state, state_slot_stride, slots,
                            batch, steps, heads, dim, vdim, o, o_ld);
    if (rc != NS_OK) return rc;
    NS_REQUIRE(dim <= 256, NS_ERR_ARGUMENT, "ns_lightning_recurrent: key size %d (at most 256)", dim);
    if (vdim <= 32) return launch_recurrent_rows<1>(d, a, batch);
    if (vdim <= 64) return launch_recurrent_rows<2>(d, a, batch);
    return launch_recurrent_rows<4>(d, a, batch);
}

extern "C" int ns_lightning_chunked(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int q_col, int k_col, int v_col, uint64_t decay,
                                    uint64_t decay_log2, uint64_t state, int64_t state_slot_stride, uint64_t slots, int batch, int steps, int heads, int dim,
                                    int vdim, uint64_t o, int o_ld, int segments)
{
    NS_ENTER(h);
    LightningArgs a;
    int rc = lightning_args(a, "ns_lightning_chunked", src, splits, src_dtype, src_ld, q_col, k_col, v_col, decay, decay_log2, state, state_slot_stride, slots, batch,
                            steps, heads, dim, vdim, o, o_ld);
    if (rc != NS_OK) return rc;
    NS_REQUIRE(dim <= 128, NS_ERR_ARGUMENT, "ns_lightning_chunked: key size %d (at most 128)", dim);
    NS_REQUIRE(segments >= 0, NS_ERR_ARGUMENT, "ns_lightning_chunked: %d segments", segments);
    // Segments when one CTA per (head, sequence, value columns) leaves SMs empty; at least two chunks each.  A source that is one
    // bf16 matrix lies outside the device object's scratch block, which then holds the segments' states.
    const int chunks = (steps + LC - 1) / LC;
    const int64_t ctas = (int64_t)heads * batch * ((vdim + LDV - 1) / LDV);
    int64_t segs = segments > 0 ? segments : (2 * d->sm_count) / ctas;
    if (segments == 0 && segs > chunks / 2) segs = chunks / 2;
    if (segs > chunks) segs = chunks;
    if (segs > 1 && src_dtype == NS_BF16) {
        a.seg_len = (int)((chunks + segs - 1) / segs) * LC;
        a.segs = (steps + a.seg_len - 1) / a.seg_len;
        if (a.segs > 1) {
            void* block = nullptr;
            rc = ns_scratch_reserve(d, (size_t)batch * a.segs * heads * dim * vdim * 4, &block);
            if (rc != NS_OK) return rc;
            a.seg_state = reinterpret_cast<float*>(block);
        }
    }
    const int vec = ((dim | vdim | q_col | k_col | v_col | src_ld) & 3) == 0 && (src & 15) == 0 && (a.src.slab & 3) == 0;
    if (dim <= 32) return launch_chunked<32>(d, a, batch, vec);
    if (dim <= 64) return launch_chunked<64>(d, a, batch, vec);
    return launch_chunked<128>(d, a, batch, vec);
}
