// The gated delta rule over a prompt's portion, 64 tokens at a time on the tensor cores (ns_delta.cu has the token-by-token form
// and the recurrence's definition).
//
// With G_t the running sum of the log decays inside a chunk (per head, or per head and key channel), S the state before it and
//     A[i, j] = beta_i sum_c k_i k_j exp(G_i - G_j)  (j < i),     P[i, j] = sum_c q_i k_j exp(G_i - G_j)  (j <= i),
// the writes of the chunk solve a unit lower-triangular system and everything else is products:
//     (I + A) U = beta (V - (K e^G) S),   O = (Q e^G) S + P U,   S <- e^(G_end) S + (K e^(G_end - G))^T U.
// Every exponent that is formed is <= 0: inside a 16-token block the pairs are summed one by one, and between blocks both sides
// are scaled relative to the row block's beginning.
//
// The recurrence is a 32-bit one, so each product's operands are split into two bf16 halves (x = hi + lo, 16 mantissa bits) and
// multiplied as hi hi + hi lo + lo hi into 32-bit accumulators; the state stays in 32-bit registers from chunk to chunk.
//
// One CTA of 8 warps walks the chunks of one (sequence, head, up to 128 value columns).
#include "ns_mma.cuh"
#include "ns_seq.cuh"

namespace {

constexpr int CH = 64;                       // tokens per chunk
constexpr float LOG2E = 1.4426950408889634f;
// A token's decay is taken as at least 2^-48.  What a stronger one would leave of the state is far below the rounding of anything
// that is added to it, and the running sums of a chunk stay small enough that their differences keep the weak decays' digits.
constexpr float WEAKEST = -48.0f;

struct ChunkArgs {
    const float* q; int q_ld;
    const float* k; int k_ld;
    const float* v; int v_ld;
    NsSource a; int a_col;
    NsSource b; int b_col;
    const float* a_log;
    const float* dt_bias;
    float* state;
    int64_t state_slot_stride;
    const int32_t* slots;
    int heads, kv_heads, dim, vdim, steps;
    float* o; int o_ld;
};

// bf16 halves of two values, packed: x = hi + lo up to 2^-17 of x
NS_DEVINL void split2(float x, float y, uint32_t& hi, uint32_t& lo)
{
    hi = ns_pack_bf16x2(x, y);
    lo = ns_pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}
NS_DEVINL void st32(uint32_t addr, uint32_t v) { asm volatile("st.shared.b32 [%0], %1;" ::"r"(addr), "r"(v) : "memory"); }
// c[i][j] += (A_i hi + lo) (B_j hi + lo) without the lo lo term, for M row tiles and N pairs of column tiles.  One term after the other over
// all accumulators, so that products which depend on one another are as far apart as the tile allows.
template <int M, int N, int NC>
NS_DEVINL void mma3(float (&c)[M][NC][4], int j0, const uint32_t (&ah)[M][4], const uint32_t (&al)[M][4], const uint32_t (&bh)[N][4], const uint32_t (&bl)[N][4])
{
#pragma unroll
    for (int term = 0; term < 3; term++)
#pragma unroll
        for (int j = 0; j < N; j++)
#pragma unroll
            for (int i = 0; i < M; i++)
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const uint32_t(&x)[4] = term == 2 ? al[i] : ah[i];
                    const uint32_t(&y)[4] = term == 1 ? bl[j] : bh[j];
                    ns_mma_bf16(c[i][2 * (j0 + j) + h], x, y[2 * h], y[2 * h + 1]);
                }
}
// four neighbouring channels of a row, zero beyond dim
NS_DEVINL float4 row4(const float* p, int c, int dim) { return c < dim ? *reinterpret_cast<const float4*>(p + c) : make_float4(0.f, 0.f, 0.f, 0.f); }
NS_DEVINL float4 times(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
NS_DEVINL float4 exp2_of(float4 a, float4 b)      // 2^(a - b)
{
    return make_float4(ns_exp2(a.x - b.x), ns_exp2(a.y - b.y), ns_exp2(a.z - b.z), ns_exp2(a.w - b.w));
}
// four values as halves at `hi` and `lo`
NS_DEVINL void st_split4(uint32_t hi, uint32_t lo, float4 v)
{
    uint32_t h0, l0, h1, l1;
    split2(v.x, v.y, h0, l0);
    split2(v.z, v.w, h1, l1);
    asm volatile("st.shared.v2.b32 [%0], {%1, %2};" ::"r"(hi), "r"(h0), "r"(h1) : "memory");
    asm volatile("st.shared.v2.b32 [%0], {%1, %2};" ::"r"(lo), "r"(l0), "r"(l1) : "memory");
}

// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z| in (0, 1]; log(1 + e) / e by its Chebyshev interpolant of degree 9 on [0, 1]
// (within 1.6e-7 of the value, evaluated in 32-bit), so that small e keep their digits and no lane branches.
NS_DEVINL float softplus(float z)
{
    const float e = ns_exp2(-fabsf(z) * LOG2E);
    float p = -0.00317605701f;
    p = fmaf(p, e, 0.0195425283f);
    p = fmaf(p, e, -0.0563736148f);
    p = fmaf(p, e, 0.105436236f);
    p = fmaf(p, e, -0.152696669f);
    p = fmaf(p, e, 0.196632743f);
    p = fmaf(p, e, -0.249516159f);
    p = fmaf(p, e, 0.333297104f);
    p = fmaf(p, e, -0.499998927f);
    p = fmaf(p, e, 1.0f);
    return fmaf(e, p, fmaxf(z, 0.0f));
}

template <int DK, int DV>
struct ChunkSmem {
    static constexpr int LK = DK + 8, LV = DV + 8, LT = CH + 8, LG = DK + 4, LA = CH + 1;
    static constexpr int KMAT = CH * LK * 2, VMAT = CH * LV * 2, TMAT = CH * LT * 2;      // bytes of one half
    // U also holds the keys as they are while A and P are made
    static constexpr int U_BYTES = 2 * VMAT > CH * LG * 4 ? 2 * VMAT : CH * LG * 4;
    static constexpr int KT = 0, QT = KT + 2 * KMAT, KB = QT + 2 * KMAT, U = KB + 2 * KMAT, T = U + U_BYTES, X = T + 2 * TMAT;
    static constexpr int S_BYTES = 2 * DK * LV * 2, G_BYTES = CH * LG * 4, A_BYTES = CH * LA * 4;
    static constexpr int X_BYTES = S_BYTES > G_BYTES + 2 * A_BYTES ? S_BYTES : G_BYTES + 2 * A_BYTES;
    static constexpr int SMALL = X + X_BYTES;                                              // beta, gamma, end decay
    static constexpr int TOTAL = SMALL + (2 * CH + DK) * 4;
    static_assert(2 * VMAT >= 2 * 32 * 33 * 4, "work space of the inversion");
    static_assert(2 * TMAT >= 2 * 32 * LK * 2, "scaled keys of the third block row");
    static_assert(TOTAL <= 227 * 1024, "a CTA's shared memory");
};

template <int DK, int DV, bool CHANNEL>
__global__ void __launch_bounds__(256, 1) ns_delta_chunk_kernel(const ChunkArgs a)
{
    using L = ChunkSmem<DK, DV>;
    extern __shared__ __align__(16) uint8_t ch_smem[];
    const uint32_t base = ns_smem_u32(ch_smem);
    float* sG = reinterpret_cast<float*>(ch_smem + L::X);                       // running log2 decays [CH][LG]; scalar mode: unused
    float* sA = reinterpret_cast<float*>(ch_smem + L::X + L::G_BYTES);          // A, then its inverse
    float* sP = sA + CH * L::LA;
    float* sW = reinterpret_cast<float*>(ch_smem + L::U);
    float* sK = sW;
    float* sBeta = reinterpret_cast<float*>(ch_smem + L::SMALL);
    float* sGam = sBeta + CH;                                                   // running log2 decay per token (scalar mode)
    float* sEnd = sGam + CH;                                                    // decay of a state row over the chunk
    constexpr int MS = DK / 64, NS = DV / 16;                                   // state tile of a warp: MS x 16 rows, NS x 8 columns

    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.x, b = blockIdx.y, v0 = blockIdx.z * DV;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int slot = a.slots[b], kvh = head / (a.heads / a.kv_heads), dim = a.dim, vdim = a.vdim;
    const int64_t row_base = (int64_t)b * a.steps;
    float* S = a.state + (int64_t)slot * a.state_slot_stride + (int64_t)head * dim * vdim;
    const float rate2 = expf(a.a_log[head]) * LOG2E;
    const int sr0 = (warp >> 1) * (DK / 4), sc0 = (warp & 1) * (DV / 2);        // this warp's state tile

    float st[MS][NS][4];
#pragma unroll
    for (int i = 0; i < MS; i++)
#pragma unroll
        for (int j = 0; j < NS; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = sr0 + i * 16 + g + (e >> 1) * 8, c = v0 + sc0 + j * 8 + t4 * 2 + (e & 1);
                st[i][j][e] = r < dim && c < vdim ? S[(int64_t)r * vdim + c] : 0.0f;
            }

    const float* qh = a.q + (int64_t)kvh * dim;
    const float* kh = a.k + (int64_t)kvh * dim;
    const float* vh = a.v + (int64_t)head * vdim + v0;

    for (int c0 = 0; c0 < a.steps; c0 += CH) {
        const int n = min(CH, a.steps - c0);
        const int64_t row0 = row_base + c0;
        // the next chunk's rows towards L2 (one line per thread and tensor covers 64 rows of 128 floats)
        if (c0 + CH < a.steps) {
            const int r = tid >> 2, c = (tid & 3) * 32;
            if (c0 + CH + r < a.steps) {
                if (c < dim) {
                    asm volatile("prefetch.global.L2 [%0];" ::"l"(kh + (row0 + CH + r) * a.k_ld + c));
                    asm volatile("prefetch.global.L2 [%0];" ::"l"(qh + (row0 + CH + r) * a.q_ld + c));
                }
                if (v0 + c < vdim && c < DV) asm volatile("prefetch.global.L2 [%0];" ::"l"(vh + (row0 + CH + r) * a.v_ld + c));
            }
        }
        constexpr int QUADS = DK / 4;      // a thread takes four channels of a row
        // keys and queries of elements e0, e0 + stride, ... (four of them), all loaded before the caller stores any
        auto load_rows = [&](int e0, int stride, float4 (&k4)[4], float4 (&q4)[4]) {
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int e = e0 + stride * x, t = e / QUADS, c = (e % QUADS) * 4;
                k4[x] = q4[x] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t < n) {
                    k4[x] = row4(kh + (row0 + t) * a.k_ld, c, dim);
                    q4[x] = row4(qh + (row0 + t) * a.q_ld, c, dim);
                }
            }
        };
        // ------------------------------------------------------------ step sizes, running decays
        if (tid < CH) sBeta[tid] = tid < n ? ns_sigmoid(ns_source_at(a.b, (row0 + tid) * a.b.ld + a.b_col + head)) : 0.0f;
        if (CHANNEL) {
            const int c = (tid % QUADS) * 4;
            const float4 dt = row4(a.dt_bias + (int64_t)head * dim, c, dim);
#pragma unroll 8
            for (int t = tid / QUADS; t < CH; t += 256 / QUADS) {
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t < n && c < dim) {
                    const int64_t at = (row0 + t) * a.a.ld + a.a_col + head * dim + c;
                    x = ns_source_at4(a.a, at);
                    x = make_float4(fmaxf(-rate2 * softplus(x.x + dt.x), WEAKEST), fmaxf(-rate2 * softplus(x.y + dt.y), WEAKEST),
                                    fmaxf(-rate2 * softplus(x.z + dt.z), WEAKEST), fmaxf(-rate2 * softplus(x.w + dt.w), WEAKEST));
                }
                *reinterpret_cast<float4*>(sG + t * L::LG + c) = x;
            }
            __syncthreads();
            if (tid < DK) {
                float s = 0.0f;
#pragma unroll 8
                for (int t = 0; t < CH; t++) { s += sG[t * L::LG + tid]; sG[t * L::LG + tid] = s; }
                sEnd[tid] = ns_exp2(s);
            }
        } else if (tid < 32) {
            const float dt = a.dt_bias[head];
            float x[2];
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int t = 2 * lane + i;
                x[i] = t < n ? fmaxf(-rate2 * softplus(ns_source_at(a.a, (row0 + t) * a.a.ld + a.a_col + head) + dt), WEAKEST) : 0.0f;
            }
            float s = x[0] + x[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float y = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += y;
            }
            sGam[2 * lane] = s - x[1];
            sGam[2 * lane + 1] = s;
        }
        __syncthreads();

        // ------------------------------------------------------------ A and P
        if (!CHANNEL) {
            const float end = sGam[CH - 1];
            for (int e0 = tid; e0 < CH * QUADS; e0 += 1024) {
                float4 k4[4], q4[4];
                load_rows(e0, 256, k4, q4);
#pragma unroll
                for (int x = 0; x < 4; x++) {
                    const int e = e0 + 256 * x, t = e / QUADS, c = (e % QUADS) * 4;
                    const uint32_t at = base + (t * L::LK + c) * 2;
                    st_split4(at + L::KT, at + L::KT + L::KMAT, k4[x]);
                    st_split4(at + L::QT, at + L::QT + L::KMAT, q4[x]);
                    const float f = ns_exp2(end - sGam[t]);
                    st_split4(at + L::KB, at + L::KB + L::KMAT, make_float4(k4[x].x * f, k4[x].y * f, k4[x].z * f, k4[x].w * f));
                }
            }
            __syncthreads();
            // warps 0..3: k rows, warps 4..7: q rows, 16 each, against all k
            float acc[1][8][4];
#pragma unroll
            for (int j = 0; j < 8; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[0][j][e] = 0.0f;
            const uint32_t am = base + (warp < 4 ? L::KT : L::QT), bm = base + L::KT;
            const int mr = (warp & 3) * 16;
#pragma unroll 1
            for (int k = 0; k < DK; k += 16) {
                uint32_t ah[1][4], al[1][4], bh[2][4], bl[2][4];
                ns_ldsm4(ah[0], ns_addr_a(am, L::LK, mr, k, lane));
                ns_ldsm4(al[0], ns_addr_a(am + L::KMAT, L::LK, mr, k, lane));
#pragma unroll
                for (int j = 0; j < 4; j += 2) {
                    if (j * 16 > mr) continue;
#pragma unroll
                    for (int x = 0; x < 2; x++) {
                        ns_ldsm4(bh[x], ns_addr_b(bm, L::LK, (j + x) * 16, k, lane));
                        ns_ldsm4(bl[x], ns_addr_b(bm + L::KMAT, L::LK, (j + x) * 16, k, lane));
                    }
                    mma3(acc, j, ah, al, bh, bl);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int r = mr + g + (e >> 1) * 8, c = j * 8 + t4 * 2 + (e & 1);
                    const float f = c <= r ? ns_exp2(sGam[r] - sGam[c]) : 0.0f;
                    if (warp < 4) sA[r * L::LA + c] = c < r ? acc[0][j][e] * f * sBeta[r] : 0.0f;
                    else sP[r * L::LA + c] = acc[0][j][e] * f;
                }
            for (int c = tid; c < DK; c += 256) sEnd[c] = ns_exp2(end);
        } else {
            // rows of block I relative to the block's beginning (in KT, QT), columns before it likewise: block 1 in KB rows 0..15,
            // block 3 in KB rows 16..63, block 2 in the T area
            for (int e0 = tid; e0 < CH * QUADS; e0 += 1024) {
                float4 k4[4], q4[4];
                load_rows(e0, 256, k4, q4);
#pragma unroll
                for (int x = 0; x < 4; x++) {
                    const int e = e0 + 256 * x, t = e / QUADS, c = (e % QUADS) * 4, blk = t >> 4;
                    const float4 G = *reinterpret_cast<const float4*>(sG + t * L::LG + c);
                    *reinterpret_cast<float4*>(sK + t * L::LG + c) = k4[x];
                    if (blk > 0) {
                        const float4 f = exp2_of(G, *reinterpret_cast<const float4*>(sG + (blk * 16 - 1) * L::LG + c));
                        const uint32_t at = base + (t * L::LK + c) * 2;
                        st_split4(at + L::KT, at + L::KT + L::KMAT, times(k4[x], f));
                        st_split4(at + L::QT, at + L::QT + L::KMAT, times(q4[x], f));
                    }
#pragma unroll
                    for (int I = 1; I < 4; I++) {
                        if (blk >= I) continue;
                        const float4 f = exp2_of(*reinterpret_cast<const float4*>(sG + (I * 16 - 1) * L::LG + c), G);
                        const uint32_t at = I == 2 ? base + L::T + (t * L::LK + c) * 2 : base + L::KB + (((I == 3 ? 16 : 0) + t) * L::LK + c) * 2;
                        st_split4(at, at + (I == 2 ? 32 * L::LK * 2 : L::KMAT), times(k4[x], f));
                    }
                }
            }
            __syncthreads();
            if (warp < 6) {
                // warps (0, 1), (2, 3), (4, 5): block rows 3, 2, 1; k rows and q rows
                const int I = 3 - (warp >> 1), which = warp & 1;
                const uint32_t am = base + (which ? L::QT : L::KT);
                const uint32_t bh_m = I == 2 ? base + L::T : base + L::KB + (I == 3 ? 16 * L::LK * 2 : 0);
                const uint32_t bl_m = bh_m + (I == 2 ? 32 * L::LK * 2 : L::KMAT);
                float acc[1][6][4];
#pragma unroll
                for (int j = 0; j < 6; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) acc[0][j][e] = 0.0f;
#pragma unroll 1
                for (int k = 0; k < DK; k += 16) {
                    uint32_t ah[1][4], al[1][4], bh[3][4], bl[3][4];
                    ns_ldsm4(ah[0], ns_addr_a(am, L::LK, I * 16, k, lane));
                    ns_ldsm4(al[0], ns_addr_a(am + L::KMAT, L::LK, I * 16, k, lane));
#pragma unroll
                    for (int j = 0; j < 3; j++) {
                        // (blocks 1 and 2 multiply some rows that are not theirs; those columns are dropped below)
                        const int n0 = j < I ? j * 16 : 0;
                        ns_ldsm4(bh[j], ns_addr_b(bh_m, L::LK, n0, k, lane));
                        ns_ldsm4(bl[j], ns_addr_b(bl_m, L::LK, n0, k, lane));
                    }
                    mma3(acc, 0, ah, al, bh, bl);
                }
#pragma unroll
                for (int j = 0; j < 6; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int r = I * 16 + g + (e >> 1) * 8, c = j * 8 + t4 * 2 + (e & 1);
                        if (c >= I * 16) continue;
                        if (which) sP[r * L::LA + c] = acc[0][j][e];
                        else sA[r * L::LA + c] = acc[0][j][e] * sBeta[r];
                    }
            }
            // the 16 x 16 blocks on the diagonal, pair by pair: 16 lanes share a row, each a sixteenth of the channels
            constexpr int CPL = DK / 16;
            const int hl = lane & 15;
            for (int task = (warp + 2) & 7; task < CH / 2; task += 8) {
                const int blk = task >> 3, ii = (lane >> 4) ? 15 - (task & 7) : (task & 7), i = blk * 16 + ii;
                const int ch = hl * 4;      // channels ch + 64 y: 16 lanes read 256 neighbouring bytes
                float ki[CPL], qi[CPL], gi[CPL];
#pragma unroll
                for (int x = 0; x < CPL; x += 4) {
                    const float4 k4 = *reinterpret_cast<const float4*>(sK + i * L::LG + ch + 16 * x);
                    const float4 q4 = i < n ? row4(qh + (row0 + i) * a.q_ld, ch + 16 * x, dim) : make_float4(0.f, 0.f, 0.f, 0.f);
                    const float4 G = *reinterpret_cast<const float4*>(sG + i * L::LG + ch + 16 * x);
                    ki[x] = k4.x; ki[x + 1] = k4.y; ki[x + 2] = k4.z; ki[x + 3] = k4.w;
                    qi[x] = q4.x; qi[x + 1] = q4.y; qi[x + 2] = q4.z; qi[x + 3] = q4.w;
                    gi[x] = G.x; gi[x + 1] = G.y; gi[x + 2] = G.z; gi[x + 3] = G.w;
                }
                // columns in groups of four; what lies right of the diagonal is dropped afterwards
                const int groups = (max(task & 7, 15 - (task & 7)) >> 2) + 1;
#pragma unroll 1
                for (int j0 = 0; j0 < groups * 4; j0 += 4) {
                    const int t0 = blk * 16 + j0;
                    float v[8];
#pragma unroll
                    for (int x = 0; x < 4; x++) {
                        float kk = 0.0f, qk = 0.0f;
#pragma unroll
                        for (int y = 0; y < CPL / 4; y++) {
                            const float4 G = *reinterpret_cast<const float4*>(sG + (t0 + x) * L::LG + ch + 64 * y);
                            const float4 k4 = *reinterpret_cast<const float4*>(sK + (t0 + x) * L::LG + ch + 64 * y);
                            const float w0 = k4.x * ns_exp2(fminf(gi[4 * y] - G.x, 0.0f)), w1 = k4.y * ns_exp2(fminf(gi[4 * y + 1] - G.y, 0.0f));
                            const float w2 = k4.z * ns_exp2(fminf(gi[4 * y + 2] - G.z, 0.0f)), w3 = k4.w * ns_exp2(fminf(gi[4 * y + 3] - G.w, 0.0f));
                            kk = fmaf(ki[4 * y], w0, fmaf(ki[4 * y + 1], w1, fmaf(ki[4 * y + 2], w2, fmaf(ki[4 * y + 3], w3, kk))));
                            qk = fmaf(qi[4 * y], w0, fmaf(qi[4 * y + 1], w1, fmaf(qi[4 * y + 2], w2, fmaf(qi[4 * y + 3], w3, qk))));
                        }
                        v[x] = kk;
                        v[4 + x] = qk;
                    }
                    // sums over the 16 lanes; two lanes end up with the same one of the eight values
#pragma unroll
                    for (int m = 8, half = 4; m >= 2; m >>= 1, half >>= 1) {
                        const bool up = (lane & m) != 0;
#pragma unroll
                        for (int x = 0; x < half; x++) {
                            const float give = up ? v[x] : v[x + half], keep = up ? v[x + half] : v[x];
                            v[x] = keep + __shfl_xor_sync(0xffffffffu, give, m);
                        }
                    }
                    v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
                    const int j = j0 + ((lane >> 1) & 1) + ((lane >> 1) & 2);
                    if ((lane & 1) == 0) {
                        if (lane & 8) sP[i * L::LA + blk * 16 + j] = j <= ii ? v[0] : 0.0f;
                        else sA[i * L::LA + blk * 16 + j] = j < ii ? v[0] * sBeta[i] : 0.0f;
                    }
                }
                for (int j = groups * 4 + hl; j < 16; j += 16) sA[i * L::LA + blk * 16 + j] = sP[i * L::LA + blk * 16 + j] = 0.0f;
                // right of the diagonal block
                for (int c = (blk + 1) * 16 + hl; c < CH; c += 16) sA[i * L::LA + c] = sP[i * L::LA + c] = 0.0f;
            }
        }
        __syncthreads();

        // ------------------------------------------------------------ (I + A)^-1, and the operands relative to the chunk
        if (tid < 64) {
            // inverse of a diagonal block, a column per thread
            float* blk = sA + (tid >> 4) * 16 * (L::LA + 1);
            const int col = tid & 15;
            float x[16];
#pragma unroll
            for (int i = 0; i < 16; i++) {
                float s = i == col ? 1.0f : 0.0f;
#pragma unroll
                for (int j = 0; j < i; j++) s = fmaf(-blk[i * L::LA + j], x[j], s);
                x[i] = s;
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < 16; i++) blk[i * L::LA + col] = x[i];
        } else if (CHANNEL) {
            for (int e0 = tid - 64; e0 < CH * QUADS; e0 += 768) {
                float4 k4[4], q4[4];
                load_rows(e0, 192, k4, q4);
#pragma unroll
                for (int x = 0; x < 4; x++) {
                    const int e = e0 + 192 * x, t = e / QUADS, c = (e % QUADS) * 4;
                    if (e >= CH * QUADS) break;
                    const float4 G = *reinterpret_cast<const float4*>(sG + t * L::LG + c), f = exp2_of(G, make_float4(0.f, 0.f, 0.f, 0.f));
                    const uint32_t at = base + (t * L::LK + c) * 2;
                    st_split4(at + L::KT, at + L::KT + L::KMAT, times(k4[x], f));
                    st_split4(at + L::QT, at + L::QT + L::KMAT, times(q4[x], f));
                    st_split4(at + L::KB, at + L::KB + L::KMAT, times(k4[x], exp2_of(*reinterpret_cast<const float4*>(sG + (CH - 1) * L::LG + c), G)));
                }
            }
        }
        __syncthreads();
        {
            // 32 x 32 blocks: lower left = -T11 A10 T00; threads 0..127 the upper, 128..255 the lower block, two outputs each
            float* m = sA + (tid >> 7) * 32 * (L::LA + 1);
            float* w = sW + (tid >> 7) * 16 * 17;
            const int t = tid & 127, r = t >> 3, c = (t & 7) * 2;
            float x0 = 0.0f, x1 = 0.0f;
#pragma unroll
            for (int k = 0; k < 16; k++) {
                const float y = m[(16 + r) * L::LA + k];
                x0 = fmaf(y, m[k * L::LA + c], x0);
                x1 = fmaf(y, m[k * L::LA + c + 1], x1);
            }
            w[r * 17 + c] = x0;
            w[r * 17 + c + 1] = x1;
            __syncthreads();
            x0 = x1 = 0.0f;
#pragma unroll
            for (int k = 0; k < 16; k++) {
                const float y = m[(16 + r) * L::LA + 16 + k];
                x0 = fmaf(y, w[k * 17 + c], x0);
                x1 = fmaf(y, w[k * 17 + c + 1], x1);
            }
            m[(16 + r) * L::LA + c] = -x0;
            m[(16 + r) * L::LA + c + 1] = -x1;
            __syncthreads();
            // the whole: a thread takes one row and four columns of the lower left 32 x 32 block
            const int R = tid >> 3, C = (tid & 7) * 4;
            float y[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 8
            for (int k = 0; k < 32; k++) {
                const float z = sA[(32 + R) * L::LA + k];
#pragma unroll
                for (int i = 0; i < 4; i++) y[i] = fmaf(z, sA[k * L::LA + C + i], y[i]);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) sW[R * 33 + C + i] = y[i];
            __syncthreads();
#pragma unroll
            for (int i = 0; i < 4; i++) y[i] = 0.0f;
#pragma unroll 8
            for (int k = 0; k < 32; k++) {
                const float z = sA[(32 + R) * L::LA + 32 + k];
#pragma unroll
                for (int i = 0; i < 4; i++) y[i] = fmaf(z, sW[k * 33 + C + i], y[i]);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) sA[(32 + R) * L::LA + C + i] = -y[i];
            __syncthreads();
        }
        // the inverse as operand; P waits in registers until the inverse has been used
        float pr[16];
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int e = tid + 256 * i, r = e >> 5, c = (e & 31) * 2;
            uint32_t hi, lo;
            split2(c <= r ? sA[r * L::LA + c] : 0.0f, c + 1 <= r ? sA[r * L::LA + c + 1] : 0.0f, hi, lo);
            const uint32_t at = base + L::T + (r * L::LT + c) * 2;
            st32(at, hi); st32(at + L::TMAT, lo);
            pr[2 * i] = sP[r * L::LA + c];
            pr[2 * i + 1] = sP[r * L::LA + c + 1];
        }
        __syncthreads();
        // ------------------------------------------------------------ the state as operand
#pragma unroll
        for (int i = 0; i < MS; i++)
#pragma unroll
            for (int j = 0; j < NS; j++)
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    uint32_t hi, lo;
                    split2(st[i][j][2 * h], st[i][j][2 * h + 1], hi, lo);
                    const uint32_t at = base + L::X + ((sr0 + i * 16 + g + h * 8) * L::LV + sc0 + j * 8 + t4 * 2) * 2;
                    st32(at, hi); st32(at + DK * L::LV * 2, lo);
                }
        __syncthreads();
        // ------------------------------------------------------------ (K e^G) S by warps 0..3, (Q e^G) S by warps 4..7
        const bool kside = warp < 4;
        const int xr = ((warp >> 1) & 1) * 32;      // rows xr .. xr + 31, columns sc0 .. sc0 + DV / 2 - 1
        float acc[2][NS][4];
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int j = 0; j < NS; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[i][j][e] = 0.0f;
        {
            const uint32_t am = base + (kside ? L::KT : L::QT), bm = base + L::X;
#pragma unroll 1
            for (int k = 0; k < DK; k += 16) {
                uint32_t ah[2][4], al[2][4];
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    ns_ldsm4(ah[i], ns_addr_a(am, L::LK, xr + i * 16, k, lane));
                    ns_ldsm4(al[i], ns_addr_a(am + L::KMAT, L::LK, xr + i * 16, k, lane));
                }
#pragma unroll
                for (int j = 0; j < NS / 2; j += 2) {
                    uint32_t bh[2][4], bl[2][4];
#pragma unroll
                    for (int x = 0; x < 2; x++) {
                        ns_ldsm4_t(bh[x], ns_addr_bt(bm, L::LV, k, sc0 + (j + x) * 16, lane));
                        ns_ldsm4_t(bl[x], ns_addr_bt(bm + DK * L::LV * 2, L::LV, k, sc0 + (j + x) * 16, lane));
                    }
                    mma3(acc, j, ah, al, bh, bl);
                }
            }
        }
        if (kside) {
            // right-hand side beta (v - decayed read); the values of 16 rows are loaded before any is used
#pragma unroll
            for (int i = 0; i < 2; i++) {
                float2 y[2][NS];
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int r = xr + i * 16 + g + h * 8;
                    const float* vp = vh + (row0 + r) * a.v_ld;
#pragma unroll
                    for (int j = 0; j < NS; j++) {
                        const int c = sc0 + j * 8 + t4 * 2;
                        y[h][j] = make_float2(0.0f, 0.0f);
                        if (r >= n) continue;
                        if (v0 + c < vdim) y[h][j] = *reinterpret_cast<const float2*>(vp + c);
                    }
                }
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int r = xr + i * 16 + g + h * 8;
                    const float beta = sBeta[r], f = CHANNEL ? 1.0f : ns_exp2(sGam[r]);
#pragma unroll
                    for (int j = 0; j < NS; j++) {
                        uint32_t hi, lo;
                        split2(beta * fmaf(-f, acc[i][j][2 * h], y[h][j].x), beta * fmaf(-f, acc[i][j][2 * h + 1], y[h][j].y), hi, lo);
                        const uint32_t at = base + L::U + (r * L::LV + sc0 + j * 8 + t4 * 2) * 2;
                        st32(at, hi); st32(at + L::VMAT, lo);
                    }
                }
            }
        }
        __syncthreads();
        // ------------------------------------------------------------ U = T (right-hand side)
        {
            constexpr int NU = DV / 32;              // n-tiles of a warp: 32 rows x DV / 4 columns
            const int ur = (warp >> 2) * 32, uc = (warp & 3) * (DV / 4);
            float ua[2][NU][4];
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int j = 0; j < NU; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) ua[i][j][e] = 0.0f;
#pragma unroll
            for (int k = 0; k < CH; k += 16) {
                if (k >= ur + 32) continue;          // above the diagonal
                uint32_t ah[2][4], al[2][4];
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    ns_ldsm4(ah[i], ns_addr_a(base + L::T, L::LT, ur + i * 16, k, lane));
                    ns_ldsm4(al[i], ns_addr_a(base + L::T + L::TMAT, L::LT, ur + i * 16, k, lane));
                }
                uint32_t bh[NU / 2][4], bl[NU / 2][4];
#pragma unroll
                for (int j = 0; j < NU / 2; j++) {
                    ns_ldsm4_t(bh[j], ns_addr_bt(base + L::U, L::LV, k, uc + j * 16, lane));
                    ns_ldsm4_t(bl[j], ns_addr_bt(base + L::U + L::VMAT, L::LV, k, uc + j * 16, lane));
                }
                mma3(ua, 0, ah, al, bh, bl);
            }
            __syncthreads();
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int j = 0; j < NU; j++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        uint32_t hi, lo;
                        split2(ua[i][j][2 * h], ua[i][j][2 * h + 1], hi, lo);
                        const uint32_t at = base + L::U + ((ur + i * 16 + g + h * 8) * L::LV + uc + j * 8 + t4 * 2) * 2;
                        st32(at, hi); st32(at + L::VMAT, lo);
                    }
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const int e = tid + 256 * i, r = e >> 5, c = (e & 31) * 2;
                uint32_t hi, lo;
                split2(pr[2 * i], pr[2 * i + 1], hi, lo);
                const uint32_t at = base + L::T + (r * L::LT + c) * 2;
                st32(at, hi); st32(at + L::TMAT, lo);
            }
        }
        __syncthreads();
        // ------------------------------------------------------------ O = (Q e^G) S + P U
        if (!kside) {
            if (!CHANNEL) {
#pragma unroll
                for (int i = 0; i < 2; i++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        const float f = ns_exp2(sGam[xr + i * 16 + g + h * 8]);
#pragma unroll
                        for (int j = 0; j < NS; j++) { acc[i][j][2 * h] *= f; acc[i][j][2 * h + 1] *= f; }
                    }
            }
#pragma unroll 1
            for (int k = 0; k < xr + 32; k += 16) {
                uint32_t ah[2][4], al[2][4];
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    ns_ldsm4(ah[i], ns_addr_a(base + L::T, L::LT, xr + i * 16, k, lane));
                    ns_ldsm4(al[i], ns_addr_a(base + L::T + L::TMAT, L::LT, xr + i * 16, k, lane));
                }
#pragma unroll
                for (int j = 0; j < NS / 2; j += 2) {
                    uint32_t bh[2][4], bl[2][4];
#pragma unroll
                    for (int x = 0; x < 2; x++) {
                        ns_ldsm4_t(bh[x], ns_addr_bt(base + L::U, L::LV, k, sc0 + (j + x) * 16, lane));
                        ns_ldsm4_t(bl[x], ns_addr_bt(base + L::U + L::VMAT, L::LV, k, sc0 + (j + x) * 16, lane));
                    }
                    mma3(acc, j, ah, al, bh, bl);
                }
            }
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int r = xr + i * 16 + g + h * 8;
                    if (r >= n) continue;
                    float* op = a.o + (row0 + r) * a.o_ld + (int64_t)head * vdim + v0;
#pragma unroll
                    for (int j = 0; j < NS; j++) {
                        const int c = sc0 + j * 8 + t4 * 2;
                        if (v0 + c < vdim) *reinterpret_cast<float2*>(op + c) = make_float2(acc[i][j][2 * h], acc[i][j][2 * h + 1]);
                    }
                }
        }
        // ------------------------------------------------------------ S <- e^(G_end) S + (K e^(G_end - G))^T U
#pragma unroll
        for (int i = 0; i < MS; i++)
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const float f = sEnd[sr0 + i * 16 + g + h * 8];
#pragma unroll
                for (int j = 0; j < NS; j++) { st[i][j][2 * h] *= f; st[i][j][2 * h + 1] *= f; }
            }
#pragma unroll 1
        for (int k = 0; k < CH; k += 16) {
            uint32_t ah[MS][4], al[MS][4];
#pragma unroll
            for (int i = 0; i < MS; i++) {
                ns_ldsm4_t(ah[i], ns_addr_at(base + L::KB, L::LK, sr0 + i * 16, k, lane));
                ns_ldsm4_t(al[i], ns_addr_at(base + L::KB + L::KMAT, L::LK, sr0 + i * 16, k, lane));
            }
#pragma unroll
            for (int j = 0; j < NS / 2; j += 2) {
                uint32_t bh[2][4], bl[2][4];
#pragma unroll
                for (int x = 0; x < 2; x++) {
                    ns_ldsm4_t(bh[x], ns_addr_bt(base + L::U, L::LV, k, sc0 + (j + x) * 16, lane));
                    ns_ldsm4_t(bl[x], ns_addr_bt(base + L::U + L::VMAT, L::LV, k, sc0 + (j + x) * 16, lane));
                }
                mma3(st, j, ah, al, bh, bl);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < MS; i++)
#pragma unroll
        for (int j = 0; j < NS; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = sr0 + i * 16 + g + (e >> 1) * 8, c = v0 + sc0 + j * 8 + t4 * 2 + (e & 1);
                if (r < dim && c < vdim) S[(int64_t)r * vdim + c] = st[i][j][e];
            }
}

template <int DK, int DV, bool CHANNEL>
int launch_chunk(NsDevice* d, const ChunkArgs& a, int batch)
{
    auto k = ns_delta_chunk_kernel<DK, DV, CHANNEL>;
    constexpr int smem = ChunkSmem<DK, DV>::TOTAL;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    NS_CUDA(ns_launch_plain(k, dim3((unsigned)a.heads, (unsigned)batch, (unsigned)((a.vdim + DV - 1) / DV)), dim3(256), smem, d->stream, a));
    return NS_OK;
}

}  // namespace

extern "C" int ns_delta_chunked(ns_device_t h, uint64_t q, int q_ld, uint64_t k, int k_ld, uint64_t v, int v_ld, uint64_t a_src, int a_splits, int a_ld,
                                int a_col, uint64_t b_src, int b_splits, int b_ld, int b_col, uint64_t a_log, uint64_t dt_bias, int per_channel,
                                uint64_t state, int64_t state_slot_stride, uint64_t slots, int batch, int steps, int heads, int kv_heads, int dim, int vdim,
                                uint64_t o, int o_ld)
{
    NsDevice* d = ns_dev(h);
    int rc = ns_device_make_current(d);
    if (rc != NS_OK) return rc;
    NS_REQUIRE(q && k && v && a_log && dt_bias && state && slots && o && batch > 0 && batch <= 65535 && steps > 0, NS_ERR_ARGUMENT, "ns_delta_chunked: bad argument");
    NS_REQUIRE(ns_source_ok(a_src, a_splits, NS_F32) && ns_source_ok(b_src, b_splits, NS_F32), NS_ERR_ARGUMENT, "ns_delta_chunked: bad source");
    NS_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0, NS_ERR_ARGUMENT, "ns_delta_chunked: %d heads do not divide over %d key heads", heads, kv_heads);
    NS_REQUIRE(dim > 0 && dim <= 128 && vdim > 0, NS_ERR_ARGUMENT, "ns_delta_chunked: key size %d (at most 128)", dim);
    NS_REQUIRE(((dim | q_ld | k_ld) & 3) == 0 && ((q | k | dt_bias) & 15) == 0 && ((vdim | v_ld | o_ld) & 1) == 0 && ((v | o) & 7) == 0, NS_ERR_ARGUMENT,
               "ns_delta_chunked: keys of %d and values of %d channels (multiples of 4 and 2, aligned)", dim, vdim);
    NS_REQUIRE(!per_channel || (((a_ld | a_col) & 3) == 0 && (a_src & 15) == 0), NS_ERR_ARGUMENT, "ns_delta_chunked: decay projection not aligned");
    ChunkArgs a;
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
    const bool wide = vdim > 64;
    if (dim <= 64) {
        if (per_channel) return wide ? launch_chunk<64, 128, true>(d, a, batch) : launch_chunk<64, 64, true>(d, a, batch);
        return wide ? launch_chunk<64, 128, false>(d, a, batch) : launch_chunk<64, 64, false>(d, a, batch);
    }
    if (per_channel) return wide ? launch_chunk<128, 128, true>(d, a, batch) : launch_chunk<128, 64, true>(d, a, batch);
    return wide ? launch_chunk<128, 128, false>(d, a, batch) : launch_chunk<128, 64, false>(d, a, batch);
}
