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
    fetch(0);
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

// A CTA handles up to DV value columns with DV * 4 threads: 16 rows x 32 columns of a chunk's outputs per warp.
template <int DK, int DV>
struct LightningShape {
    static constexpr int THREADS = DV * 4, WARPS = DV / 8;
    // rows that keep ldmatrix free of bank conflicts, in elements
    static constexpr int LK = DK + 8, LV = DV + 8, LP = LC + 8;
    // shared memory: queries, keys, values (two chunks), values as the chunk's end sees them, the state, weighted scores (two chunks); the
    // last three as two halves each
    static constexpr int K_BYTES = LC * LK * 2, V_BYTES = LC * LV * 2, S_BYTES = DK * LV * 2, P_BYTES = LC * LP * 2;
    static constexpr int Q = 0, K = Q + K_BYTES, V = K + K_BYTES, W = V + 2 * V_BYTES, S = W + 2 * V_BYTES, P = S + 2 * S_BYTES, TOTAL = P + 4 * P_BYTES;
    // state tile of a warp: MT x 16 rows, NT x 8 columns
    static constexpr int MT = DK >= 128 ? 2 : 1, ROW_GROUPS = DK / (16 * MT), NT = DV / 8 / (WARPS / ROW_GROUPS);
    static_assert(TOTAL <= 227 * 1024 && NT % 2 == 0, "a CTA's shared memory");
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
NS_DEVINL float silu_fast(float z)
{
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + ns_exp2(z * -1.4426950408889634f)));
    return z * r;
}

// A tile [64, WIDTH] of the source from column `col` on, activated, as bf16 pairs: groups of four neighbouring channels, or of eight where the
// source is one bf16 matrix (BF16).  Group x of a thread is element tid + THREADS x.  Rows past n and channels from `size` on are zero.
// All loads are on their way before the first is used.
template <int WIDTH, int THREADS, bool BF16>
struct Tile {
    static constexpr int PER = BF16 ? 8 : 4, GROUPS = WIDTH / PER, N = LC * GROUPS / THREADS > 0 ? LC * GROUPS / THREADS : 1;
    uint32_t x[N][PER / 2];

    NS_DEVINL static int row(int i, int tid) { return (tid + THREADS * i) / GROUPS; }
    NS_DEVINL static int column(int i, int tid) { return (tid + THREADS * i) % GROUPS * PER; }

    NS_DEVINL void load(const NsSource& s, int64_t row0, int n, int col, int size, bool vec, int tid)
    {
        if constexpr (BF16) {
            const uint16_t* p = reinterpret_cast<const uint16_t*>(s.ptr) + row0 * s.ld + col;
#pragma unroll
            for (int i = 0; i < N; i++) {
                const int t = row(i, tid), c = column(i, tid);
                uint4 v = make_uint4(0, 0, 0, 0);
                if (t < n && t < LC && c < size) v = *reinterpret_cast<const uint4*>(p + (int64_t)t * s.ld + c);
                x[i][0] = v.x; x[i][1] = v.y; x[i][2] = v.z; x[i][3] = v.w;
            }
        } else {
            float4 f[N];
#pragma unroll
            for (int i = 0; i < N; i++) {
                const int t = row(i, tid), c = column(i, tid);
                f[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t >= n || t >= LC || c >= size) continue;
                const int64_t at = (row0 + t) * s.ld + col + c;
                if (vec) {
                    f[i] = ns_source_at4(s, at);
                } else {
                    f[i].x = ns_source_at(s, at);
                    if (c + 1 < size) f[i].y = ns_source_at(s, at + 1);
                    if (c + 2 < size) f[i].z = ns_source_at(s, at + 2);
                    if (c + 3 < size) f[i].w = ns_source_at(s, at + 3);
                }
            }
#pragma unroll
            for (int i = 0; i < N; i++) {
                x[i][0] = ns_pack_bf16x2(silu_fast(f[i].x), silu_fast(f[i].y));
                x[i][1] = ns_pack_bf16x2(silu_fast(f[i].z), silu_fast(f[i].w));
            }
        }
    }
    NS_DEVINL void activate()
    {
        if constexpr (BF16) {
#pragma unroll
            for (int i = 0; i < N; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) x[i][j] = ns_pack_bf16x2(silu_fast(__uint_as_float(x[i][j] << 16)), silu_fast(__uint_as_float(x[i][j] & 0xFFFF0000u)));
        }
    }
    NS_DEVINL void store(uint32_t dst, int ld, int tid) const
    {
#pragma unroll
        for (int i = 0; i < N; i++) {
            if (row(i, tid) >= LC) continue;
            const uint32_t at = dst + (row(i, tid) * ld + column(i, tid)) * 2;
            if constexpr (BF16) ns_st_shared_v4(at, x[i][0], x[i][1], x[i][2], x[i][3]);
            else st_shared_v2(at, x[i][0], x[i][1]);
        }
    }
};

// WRITES_ONLY: a segment's own writes (no queries, no outputs), left in seg_state.  BF16: the source is one bf16 matrix and every
// tensor's columns start and end on multiples of eight; the next chunk's rows are then on their way while this one is computed.
//
// Between the first barrier of a chunk (its tiles and the state are in shared memory) and the second one, ten of the warps' 16 x 16
// blocks of scores are made, weighted and left in shared memory, every warp reads the state out for its rows and takes the
// chunk's writes into its piece of the state; after the second barrier the weighted scores meet the values.
template <int DK, int DV, bool WRITES_ONLY, bool BF16>
__global__ void __launch_bounds__(DV * 4, LightningShape<DK, DV>::TOTAL <= 113 * 1024 ? 2 : 1) ns_lightning_chunk_kernel(const LightningArgs a, int vec)
{
    using L = LightningShape<DK, DV>;
    constexpr int MT = L::MT, NT = L::NT, T = L::THREADS;
    extern __shared__ __align__(16) uint8_t lc_smem[];
    const uint32_t base = ns_smem_u32(lc_smem), sQ = base + L::Q, sK = base + L::K, sWH = base + L::W, sWL = sWH + L::V_BYTES, sSH = base + L::S, sSL = sSH + L::S_BYTES;
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.x, b = blockIdx.y, seg = blockIdx.z % a.segs, v0 = (blockIdx.z / a.segs) * DV;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int dim = a.dim, vdim = a.vdim;
    const float ld2 = a.decay_log2[head];
    const int64_t per_head = (int64_t)dim * vdim;
    float* S = a.segs > 1 ? a.seg_state + (((int64_t)b * a.segs + seg) * a.heads + head) * per_head
                          : a.state + (int64_t)a.slots[b] * a.state_slot_stride + head * per_head;
    const int begin = seg * a.seg_len, end = min(a.steps, begin + a.seg_len);
    const int sr = (warp % L::ROW_GROUPS) * MT * 16, sc = (warp / L::ROW_GROUPS) * NT * 8;

    Tile<DK, T, BF16> kt, qt;
    Tile<DV, T, BF16> vt;
    auto load_tiles = [&](int c0) {
        const int n = min(LC, end - c0);
        const int64_t row0 = (int64_t)b * a.steps + c0;
        kt.load(a.src, row0, n, a.k_col + head * dim, dim, vec, tid);
        if constexpr (!WRITES_ONLY) qt.load(a.src, row0, n, a.q_col + head * dim, dim, vec, tid);
        vt.load(a.src, row0, n, a.v_col + head * vdim + v0, vdim - v0, vec, tid);
    };
    load_tiles(begin);

    float st[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = sr + i * 16 + g + (e >> 1) * 8, c = v0 + sc + j * 8 + t4 * 2 + (e & 1);
                st[i][j][e] = !WRITES_ONLY && r < dim && c < vdim ? S[(int64_t)r * vdim + c] : 0.0f;
            }

    for (int c0 = begin, turn = 0; c0 < end; c0 += LC, turn ^= 1) {
        const int n = min(LC, end - c0);
        const uint32_t sV = base + L::V + turn * L::V_BYTES, sPH = base + L::P + turn * 2 * L::P_BYTES, sPL = sPH + L::P_BYTES;
        if (!BF16 && c0 > begin) load_tiles(c0);
        kt.activate();
        kt.store(sK, L::LK, tid);
        if constexpr (!WRITES_ONLY) {
            qt.activate();
            qt.store(sQ, L::LK, tid);
        }
        vt.activate();
        if constexpr (!WRITES_ONLY) vt.store(sV, L::LV, tid);
        // the values as the state at the chunk's end sees them
        using VT = Tile<DV, T, BF16>;
#pragma unroll
        for (int i = 0; i < VT::N; i++) {
            const int t = VT::row(i, tid);
            const float w = t < n ? ns_exp2((float)(n - 1 - t) * ld2) : 0.0f;
            uint32_t hi[VT::PER / 2], lo[VT::PER / 2];
#pragma unroll
            for (int j = 0; j < VT::PER / 2; j++) halves(__uint_as_float(vt.x[i][j] << 16) * w, __uint_as_float(vt.x[i][j] & 0xFFFF0000u) * w, hi[j], lo[j]);
            const uint32_t at = (t * L::LV + VT::column(i, tid)) * 2;
            if constexpr (BF16) {
                ns_st_shared_v4(sWH + at, hi[0], hi[1], hi[2], hi[3]);
                ns_st_shared_v4(sWL + at, lo[0], lo[1], lo[2], lo[3]);
            } else {
                st_shared_v2(sWH + at, hi[0], hi[1]);
                st_shared_v2(sWL + at, lo[0], lo[1]);
            }
        }
        if constexpr (!WRITES_ONLY) {
#pragma unroll
            for (int i = 0; i < MT; i++)
#pragma unroll
                for (int j = 0; j < NT; j++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        uint32_t hi, lo;
                        halves(st[i][j][2 * h], st[i][j][2 * h + 1], hi, lo);
                        const uint32_t at = ((sr + i * 16 + g + h * 8) * L::LV + sc + j * 8 + t4 * 2) * 2;
                        st_shared_1(sSH + at, hi);
                        st_shared_1(sSL + at, lo);
                    }
        }
        __syncthreads();
        if (BF16 && c0 + LC < end) load_tiles(c0 + LC);
        const int r0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;       // this warp's outputs
        float acc[4][4];
        if constexpr (!WRITES_ONLY) {
            // blocks (0, 0), (1, 0), (1, 1), (2, 0), ... of the scores
            for (int block = warp; block < 10; block += L::WARPS) {
                const int qb = block < 1 ? 0 : (block < 3 ? 1 : (block < 6 ? 2 : 3)), kb = block - qb * (qb + 1) / 2;
                float s[2][4];
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[j][e] = 0.0f;
#pragma unroll
                for (int k = 0; k < DK / 16; k++) {
                    uint32_t af[4], bf[4];
                    ns_ldsm4(af, ns_addr_a(sQ, L::LK, qb * 16, k * 16, lane));
                    ns_ldsm4(bf, ns_addr_b(sK, L::LK, kb * 16, k * 16, lane));
                    ns_mma_bf16(s[0], af, bf[0], bf[1]);
                    ns_mma_bf16(s[1], af, bf[2], bf[3]);
                }
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        const int r = qb * 16 + g + h * 8, c = kb * 16 + j * 8 + t4 * 2;
                        const float x = r >= c ? s[j][2 * h] * ns_exp2((float)(r - c) * ld2) : 0.0f;
                        const float y = r >= c + 1 ? s[j][2 * h + 1] * ns_exp2((float)(r - c - 1) * ld2) : 0.0f;
                        uint32_t hi, lo;
                        halves(x, y, hi, lo);
                        st_shared_1(sPH + (r * L::LP + c) * 2, hi);
                        st_shared_1(sPL + (r * L::LP + c) * 2, lo);
                    }
            }
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[j][e] = 0.0f;
#pragma unroll
            for (int k = 0; k < DK / 16; k++) {
                uint32_t af[4], bh[2][4], bl[2][4];
                ns_ldsm4(af, ns_addr_a(sQ, L::LK, r0, k * 16, lane));
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    ns_ldsm4_t(bh[j], ns_addr_bt(sSH, L::LV, k * 16, n0 + j * 16, lane));
                    ns_ldsm4_t(bl[j], ns_addr_bt(sSL, L::LV, k * 16, n0 + j * 16, lane));
                }
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], af, bh[j >> 1][2 * (j & 1)], bh[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
                for (int j = 0; j < 4; j++) ns_mma_bf16(acc[j], af, bl[j >> 1][2 * (j & 1)], bl[j >> 1][2 * (j & 1) + 1]);
            }
            const float f0 = ns_exp2((float)(r0 + g + 1) * ld2), f1 = ns_exp2((float)(r0 + g + 9) * ld2);
#pragma unroll
            for (int j = 0; j < 4; j++) { acc[j][0] *= f0; acc[j][1] *= f0; acc[j][2] *= f1; acc[j][3] *= f1; }
        }
        // the state after the chunk
        const float fn = ns_exp2((float)n * ld2);
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) st[i][j][e] *= fn;
#pragma unroll
        for (int k = 0; k < LC; k += 16) {
            uint32_t af[MT][4];
#pragma unroll
            for (int i = 0; i < MT; i++) ns_ldsm4_t(af[i], ns_addr_at(sK, L::LK, sr + i * 16, k, lane));
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t bh[4], bl[4];
                ns_ldsm4_t(bh, ns_addr_bt(sWH, L::LV, k, sc + j * 8, lane));
                ns_ldsm4_t(bl, ns_addr_bt(sWL, L::LV, k, sc + j * 8, lane));
#pragma unroll
                for (int i = 0; i < MT; i++) {
                    ns_mma_bf16(st[i][j], af[i], bh[0], bh[1]);
                    ns_mma_bf16(st[i][j + 1], af[i], bh[2], bh[3]);
                }
#pragma unroll
                for (int i = 0; i < MT; i++) {
                    ns_mma_bf16(st[i][j], af[i], bl[0], bl[1]);
                    ns_mma_bf16(st[i][j + 1], af[i], bl[2], bl[3]);
                }
            }
        }
        __syncthreads();
        if constexpr (!WRITES_ONLY) {
            for (int kb = 0; kb <= r0; kb += 16) {
                uint32_t ph[4], pl[4], vf[2][4];
                ns_ldsm4(ph, ns_addr_a(sPH, L::LP, r0, kb, lane));
                ns_ldsm4(pl, ns_addr_a(sPL, L::LP, r0, kb, lane));
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
                float* o = a.o + ((int64_t)b * a.steps + c0 + r) * a.o_ld + (int64_t)head * vdim;
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
    }
    if (!WRITES_ONLY && a.segs > 1) return;          // the states at the segments' ends are known already
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = sr + i * 16 + g + (e >> 1) * 8, c = v0 + sc + j * 8 + t4 * 2 + (e & 1);
                if (r < dim && c < vdim) S[(int64_t)r * vdim + c] = st[i][j][e];
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

template <int DK, int DV, bool WRITES_ONLY, bool BF16>
int launch_chunk_kernel(NsDevice* d, const LightningArgs& a, int batch, int vec)
{
    using L = LightningShape<DK, DV>;
    auto k = ns_lightning_chunk_kernel<DK, DV, WRITES_ONLY, BF16>;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
    const dim3 grid((unsigned)a.heads, (unsigned)batch, (unsigned)((a.vdim + DV - 1) / DV * a.segs));
    NS_CUDA(ns_launch_plain(k, grid, dim3(L::THREADS), (size_t)L::TOTAL, d->stream, a, vec));
    return NS_OK;
}

template <int DK, int DV, bool BF16>
int launch_chunked(NsDevice* d, const LightningArgs& a, int batch, int vec)
{
    if (a.segs > 1) {
        int rc = launch_chunk_kernel<DK, DV, true, BF16>(d, a, batch, vec);
        if (rc != NS_OK) return rc;
        const dim3 grid((unsigned)(((int64_t)a.dim * a.vdim + 255) / 256), (unsigned)a.heads, (unsigned)batch);
        NS_CUDA(ns_launch_plain(ns_lightning_carry_kernel, grid, dim3(256), 0, d->stream, a));
    }
    return launch_chunk_kernel<DK, DV, false, BF16>(d, a, batch, vec);
}

template <int DV, bool BF16>
int dispatch_chunked(NsDevice* d, const LightningArgs& a, int batch, int vec)
{
    if (a.dim <= 32) return launch_chunked<32, DV, BF16>(d, a, batch, vec);
    return a.dim <= 64 ? launch_chunked<64, DV, BF16>(d, a, batch, vec) : launch_chunked<128, DV, BF16>(d, a, batch, vec);
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
    const int64_t ctas = (int64_t)heads * batch * (vdim <= 64 ? 1 : (vdim + 127) / 128);
    int64_t segs = segments > 0 ? segments : (vdim <= 64 ? 2 : 1) * d->sm_count / ctas;
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
    const bool eights = src_dtype == NS_BF16 && ((dim | vdim | q_col | k_col | v_col | src_ld) & 7) == 0 && (src & 15) == 0;
    if (vdim <= 64) return eights ? dispatch_chunked<64, true>(d, a, batch, vec) : dispatch_chunked<64, false>(d, a, batch, vec);
    return eights ? dispatch_chunked<128, true>(d, a, batch, vec) : dispatch_chunked<128, false>(d, a, batch, vec);
}
