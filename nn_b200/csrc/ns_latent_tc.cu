// Latent attention in bf16 on the tensor cores (the float32 forms are in ns_latent.cu).
//
//   ns_latent_gather   cached rows of a step's window, ring order -> position order, one block per sequence
//   ns_latent_prefill  a prompt's portion: keys and values already expanded per head, windowed causal attention over 64-row
//                      query tiles and 64-key tiles, one warp per 16 query rows
//   ns_latent_decode   few tokens: attention over the cached latents themselves; all heads of a sequence share the cached rows,
//                      so a tile of 32 rows is read once for 16 or 32 (token, head) rows
//   ns_head_matmul_tc  the per-head products around it
//
// Scores, maxima, sums and accumulators are 32-bit; the operands of the two products (queries, keys, values, softmax weights) are
// bf16 as in the full-attention kernels.
#include <string.h>

#include "ns_mma.cuh"
#include "ns_seq.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

NS_DEVINL void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar)
{
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// ---------------------------------------------------------------------------------------------
// gather
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) ns_latent_gather_kernel(const uint16_t* __restrict__ ring, int64_t slot_stride, int ring_len, int ld, int past,
                                                               const int32_t* __restrict__ slots, const int32_t* __restrict__ pos, int rows, uint16_t* __restrict__ keys)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slot = slots[b];
    for (int j = blockIdx.x * 4 + warp; j < rows; j += gridDim.x * 4) {
        const int p = pos[slot] - past + j;
        uint4* dst = reinterpret_cast<uint4*>(keys + ((int64_t)b * rows + j) * ld);
        const uint4* src = reinterpret_cast<const uint4*>(ring + (int64_t)slot * slot_stride + (int64_t)(p >= 0 ? p % ring_len : 0) * ld);
        for (int c = lane; c < ld / 8; c += 32) dst[c] = p >= 0 ? src[c] : make_uint4(0, 0, 0, 0);
    }
}

// ---------------------------------------------------------------------------------------------
// prefill
// ---------------------------------------------------------------------------------------------
struct PrefillArgs {
    const uint16_t* q; int64_t q_ld;         // [rows, heads * (dim + rot)], rotated
    const uint16_t* kv; int64_t kv_ld;       // [batch * nk, heads * dim | heads * vdim]
    const uint16_t* keys; int64_t keys_ld;   // [batch * nk, rank | rot]
    int rank;
    uint16_t* o; int64_t o_ld;               // [rows, heads * vdim]
    const int32_t* slots;
    const int32_t* pos;
    int steps, heads, dim, rot, vdim, past, nk, window;
    float scale2;                            // scale * log2(e)
    int vec;
    int dim_boxes;                           // TMA: boxes of the unrotated part
    int* status;
};
struct PrefillMaps {
    CUtensorMap kv, keys;                    // boxes of 64 columns x 64 rows
};

constexpr int PF_ROWS = 64, PF_KEYS = 64;
constexpr uint32_t PF_BOX = 64 * 128;       // bytes

// NV: value n-tiles of 8.  KS: 16-wide k-steps of the scores whose query fragments stay in registers.
// TMA: key and value tiles arrive as boxes of 64 columns x 64 rows (128-byte swizzle), the unrotated and the rotated part of the
// heads each padded to whole boxes.  What a box holds beyond its part meets zeros of the query, or columns that are not stored.
// Otherwise (sizes that are not multiples of 8) rows are copied piece by piece.
template <int NV, int KS, bool TMA>
__global__ void __launch_bounds__(128) ns_latent_prefill_kernel(const __grid_constant__ PrefillMaps maps, const PrefillArgs a)
{
    extern __shared__ __align__(1024) uint16_t pf_smem[];
    constexpr int VLD = NV * 8 + 8, DKP = KS * 16, KLD = DKP + 8;
    constexpr int KB = KS / 4, VB = (NV + 7) / 8;        // boxes of a key and of a value tile
    constexpr uint32_t K_BYTES = TMA ? KB * PF_BOX : PF_KEYS * KLD * 2, V_BYTES = TMA ? VB * PF_BOX : PF_KEYS * VLD * 2;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t raw = ns_smem_u32(pf_smem), sK = TMA ? (raw + 1023u) & ~1023u : raw, sV = sK + 2 * K_BYTES;
    const uint32_t sQ = TMA ? sV : sK + K_BYTES;         // a place that is filled after the query fragments have been read
    __shared__ __align__(8) uint64_t full[2];
    __shared__ int abort_flag;
    const uint32_t bars = ns_smem_u32(full);
    if (TMA && tid == 0) {
        abort_flag = 0;
        ns_mbar_init(bars, 1);
        ns_mbar_init(bars + 8, 1);
        ns_fence_barrier_init();
        ns_fence_proxy_async();
    }
    ns_pdl_wait();
    ns_pdl_trigger();
    const int tiles_q = (a.steps + PF_ROWS - 1) / PF_ROWS;
    const int q0 = (tiles_q - 1 - (int)blockIdx.x) * PF_ROWS, head = blockIdx.y, b = blockIdx.z;
    const int pos0 = a.pos[a.slots[b]];
    const int dk = a.dim + a.rot;

    // a warp per row, a lane per 16 bytes
    for (int r = warp; r < PF_ROWS; r += 4) {
        const bool in = q0 + r < a.steps;
        const uint16_t* src = a.q + ((int64_t)b * a.steps + (in ? q0 + r : 0)) * a.q_ld + (int64_t)head * dk;
        for (int c = lane * 8; c < DKP; c += 256) {
            int at = c, left = dk - c;                   // column of the head and how many follow it in its part
            if (TMA) {
                const bool plain = c < a.dim_boxes * 64;
                at = plain ? c : a.dim + c - a.dim_boxes * 64;
                left = plain ? a.dim - c : dk - at;
            }
            ns_copy8(sQ + (r * KLD + c) * 2, src + (in && left > 0 ? at : 0), in ? left : 0, a.vec);
        }
    }
    auto load_tile = [&](int kt, int stage) {
        const int k0 = kt * PF_KEYS;
        if (TMA) {
            if (tid == 0) {
                const uint32_t bar = bars + 8 * stage, dk_s = sK + stage * K_BYTES, dv_s = sV + stage * V_BYTES;
                const int y = b * a.nk + k0;
                ns_mbar_expect_tx(bar, K_BYTES + V_BYTES);
                for (int i = 0; i < KB; i++) {
                    if (i < a.dim_boxes) ns_tma_load_2d(dk_s + i * PF_BOX, &maps.kv, bar, head * a.dim + i * 64, y);
                    else ns_tma_load_2d(dk_s + i * PF_BOX, &maps.keys, bar, a.rank + (i - a.dim_boxes) * 64, y);
                }
                for (int i = 0; i < VB; i++) ns_tma_load_2d(dv_s + i * PF_BOX, &maps.kv, bar, a.heads * a.dim + head * a.vdim + i * 64, y);
            }
            return;
        }
        const uint32_t dk_s = sK + stage * PF_KEYS * KLD * 2, dv_s = sV + stage * PF_KEYS * VLD * 2;
        for (int r = warp; r < PF_KEYS; r += 4) {
            const bool in = k0 + r < a.nk;
            const int64_t row = (int64_t)b * a.nk + (in ? k0 + r : 0);
            const uint16_t* kp = a.kv + row * a.kv_ld + (int64_t)head * a.dim;
            const uint16_t* rp = a.keys + row * a.keys_ld + a.rank;
            for (int c = lane * 8; c < DKP; c += 256) {
                const uint32_t dst = dk_s + (r * KLD + c) * 2;
                if (a.vec) {
                    const uint16_t* src = c < a.dim ? kp + c : rp + (c < dk ? c - a.dim : 0);
                    ns_copy8(dst, src, in ? dk - c : 0, true);
                } else {
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        uint32_t h2[2];
#pragma unroll
                        for (int s = 0; s < 2; s++) {
                            const int cc = c + 2 * i + s;
                            h2[s] = !in || cc >= dk ? 0u : (cc < a.dim ? kp[cc] : rp[cc - a.dim]);
                        }
                        w[i] = h2[0] | (h2[1] << 16);
                    }
                    ns_st_shared_v4(dst, w[0], w[1], w[2], w[3]);
                }
            }
        }
        for (int e = tid; e < PF_KEYS * NV; e += 128) {
            const int r = e / NV, c = (e - r * NV) * 8;
            const bool in = k0 + r < a.nk;
            const int64_t row = (int64_t)b * a.nk + (in ? k0 + r : 0);
            ns_copy8(dv_s + (r * VLD + c) * 2, a.kv + row * a.kv_ld + (int64_t)a.heads * a.dim + (int64_t)head * a.vdim + (c < a.vdim ? c : 0),
                     in ? a.vdim - c : 0, a.vec);
        }
        ns_cp_commit();
    };

    // visible keys of query row i, as indexes of the gathered block: (i + past - window, i + past]
    int lo = max(0, a.past - pos0);
    if (a.window > 0) lo = max(lo, q0 + a.past - a.window + 1);
    const int hi = min(q0 + PF_ROWS, a.steps) - 1 + a.past;
    const int t_first = lo / PF_KEYS, t_last = hi / PF_KEYS;

    float acc[NV][4];
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[j][i] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    const int r0 = q0 + warp * 16 + g;       // query rows r0 and r0 + 8

    if (TMA) ns_cp_commit();
    else load_tile(t_first, 0);
    ns_cp_wait<0>();
    __syncthreads();
    uint32_t qf[KS][4];
#pragma unroll
    for (int k = 0; k < KS; k++) ns_ldsm4(qf[k], ns_addr_a(sQ, KLD, warp * 16, k * 16, lane));
    __syncthreads();
    if (TMA) {
        ns_fence_proxy_async();          // the query's place was written and read by the generic proxy
        load_tile(t_first, 0);
    }
    bool gave_up = false;
    for (int kt = t_first; kt <= t_last; kt++) {
        const int stage = (kt - t_first) & 1;
        if (kt < t_last) load_tile(kt + 1, stage ^ 1);
        if (TMA) {
            const bool ok = ns_mbar_wait(bars + 8 * stage, ((kt - t_first) >> 1) & 1, &abort_flag, a.status, 710);
            if (__syncthreads_or(!ok)) {
                gave_up = true;
                break;
            }
        } else {
            if (kt < t_last) ns_cp_wait<1>();
            else ns_cp_wait<0>();
            __syncthreads();
        }
        const uint32_t tK = sK + stage * K_BYTES, tV = sV + stage * V_BYTES;
        // ldmatrix addresses of 16 keys x 16 columns, and of 16 keys x 16 value columns (transposed)
        auto key_addr = [&](int n, int k) -> uint32_t {
            if (TMA) return tK + (k >> 6) * PF_BOX + (n + (lane & 7) + (lane >> 4) * 8) * 128 + (((((k & 63) >> 3) + ((lane >> 3) & 1)) ^ (lane & 7)) * 16);
            return ns_addr_b(tK, KLD, n, k, lane);
        };
        auto value_addr = [&](int k, int n) -> uint32_t {
            if (TMA) return tV + (n >> 6) * PF_BOX + (k + (lane & 7) + ((lane >> 3) & 1) * 8) * 128 + (((((n & 63) >> 3) + (lane >> 4)) ^ (lane & 7)) * 16);
            return ns_addr_bt(tV, VLD, k, n, lane);
        };
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[j][i] = 0.0f;
        // the next k-step's key fragments are on their way while this one is multiplied
        uint32_t bf[2][4][4];
#pragma unroll
        for (int j = 0; j < 4; j++) ns_ldsm4(bf[0][j], key_addr(j * 16, 0));
#pragma unroll
        for (int k = 0; k < KS; k++) {
            if (k + 1 < KS)
#pragma unroll
                for (int j = 0; j < 4; j++) ns_ldsm4(bf[(k + 1) & 1][j], key_addr(j * 16, (k + 1) * 16));
#pragma unroll
            for (int j = 0; j < 4; j++) {
                ns_mma_bf16(s[2 * j], qf[k], bf[k & 1][j][0], bf[k & 1][j][1]);
                ns_mma_bf16(s[2 * j + 1], qf[k], bf[k & 1][j][2], bf[k & 1][j][3]);
            }
        }
        const int k0 = kt * PF_KEYS;
        // every key of the tile visible to every row of the warp?
        const int wr = q0 + warp * 16;
        const bool inner = k0 >= lo && k0 + PF_KEYS - 1 <= wr + a.past && (a.window <= 0 || k0 > wr + 15 + a.past - a.window);
        if (!inner) {
#pragma unroll
            for (int j = 0; j < 8; j++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int row = r0 + (i >> 1) * 8, key = k0 + j * 8 + t4 * 2 + (i & 1);
                    const bool see = key <= row + a.past && key >= a.past - pos0 && (a.window <= 0 || key > row + a.past - a.window);
                    if (!see) s[j][i] = -INFINITY;
                }
        }
        float f[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            float mt = -INFINITY;
#pragma unroll
            for (int j = 0; j < 8; j++) mt = fmaxf(mt, fmaxf(s[j][2 * h], s[j][2 * h + 1]));
            mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 1));
            mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 2));
            const float mn = fmaxf(m[h], mt * a.scale2);
            const float base = mn == -INFINITY ? 0.0f : mn;
            f[h] = ns_exp2(m[h] - base);
            m[h] = mn;
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < 8; j++)
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const float p = ns_exp2(fmaf(s[j][2 * h + i], a.scale2, -base));
                    s[j][2 * h + i] = p;
                    sum += p;
                }
            l[h] = fmaf(l[h], f[h], sum);
        }
#pragma unroll
        for (int j = 0; j < NV; j++) {
            acc[j][0] *= f[0]; acc[j][1] *= f[0]; acc[j][2] *= f[1]; acc[j][3] *= f[1];
        }
        constexpr int GV = NV >= 8 ? 4 : NV / 2, NG = NV / 2 / GV;      // value fragments in groups of GV, one group ahead
        uint32_t vf[2][GV][4];
#pragma unroll
        for (int j = 0; j < GV; j++) ns_ldsm4_t(vf[0][j], value_addr(0, j * 16));
#pragma unroll
        for (int k = 0; k < 4; k++) {
            const uint32_t pf[4] = {ns_pack_bf16x2(s[2 * k][0], s[2 * k][1]), ns_pack_bf16x2(s[2 * k][2], s[2 * k][3]),
                                    ns_pack_bf16x2(s[2 * k + 1][0], s[2 * k + 1][1]), ns_pack_bf16x2(s[2 * k + 1][2], s[2 * k + 1][3])};
#pragma unroll
            for (int q = 0; q < NG; q++) {
                const int at = k * NG + q, nx = at + 1;
                if (nx < 4 * NG)
#pragma unroll
                    for (int j = 0; j < GV; j++) ns_ldsm4_t(vf[nx & 1][j], value_addr((nx / NG) * 16, ((nx % NG) * GV + j) * 16));
#pragma unroll
                for (int j = 0; j < GV; j++) {
                    ns_mma_bf16(acc[2 * (q * GV + j)], pf, vf[at & 1][j][0], vf[at & 1][j][1]);
                    ns_mma_bf16(acc[2 * (q * GV + j) + 1], pf, vf[at & 1][j][2], vf[at & 1][j][3]);
                }
            }
        }
        __syncthreads();
    }
    if (gave_up) {                       // copies of this CTA may still be in flight: leave them time to land
        const long long t0 = clock64();
        while (clock64() - t0 < 400000) { }
        return;
    }
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const int row = r0 + h * 8;
        if (row >= a.steps) continue;
        const float inv = 1.0f / l[h];
        uint16_t* o = a.o + ((int64_t)b * a.steps + row) * a.o_ld + (int64_t)head * a.vdim;
        const bool pair = (((uintptr_t)o) & 3) == 0;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int c = j * 8 + t4 * 2;
            const float v0 = acc[j][2 * h] * inv, v1 = acc[j][2 * h + 1] * inv;
            if (pair && c + 1 < a.vdim) {
                *reinterpret_cast<uint32_t*>(o + c) = ns_pack_bf16x2(v0, v1);
            } else {
                if (c < a.vdim) o[c] = ns_f32_to_bf16_bits(v0);
                if (c + 1 < a.vdim) o[c + 1] = ns_f32_to_bf16_bits(v1);
            }
        }
    }
}

// ---------------------------------------------------------------------------------------------
// decode
// ---------------------------------------------------------------------------------------------
struct DecodeArgs {
    const uint16_t* q;         // [batch, steps * heads, width]
    const uint16_t* ring;
    int64_t ring_slot_stride;
    int ring_len, ring_ld;
    int rank, width, wp;       // wp: width rounded up to 32
    int window;
    float scale2;
    const int32_t* slots;
    const int32_t* pos;
    int steps, heads, rows;    // rows = steps * heads
    uint16_t* o;               // [batch, rows, rank]; splits == 1
    float* part;               // [batch, rows, splits, rank + 2]: weighted sum, maximum, sum
    int splits;
    int* status;
};

constexpr int DC_KEYS = 32;

// MT: 16-row tiles per CTA; NW: value n-tiles of 8 per warp (8 warps side by side over the latent)
template <int MT, int NW>
__global__ void __launch_bounds__(256, MT == 1 && NW <= 8 ? 2 : 1) ns_latent_decode_kernel(const DecodeArgs a)
{
    extern __shared__ __align__(16) uint16_t dc_smem[];
    constexpr int R = MT * 16, SLD = DC_KEYS + 4, PLD = DC_KEYS + 8;
    const int ld = a.wp + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t sQ = ns_smem_u32(dc_smem), sC = sQ + R * ld * 2, sP = sC + 2 * DC_KEYS * ld * 2;
    float* sS = reinterpret_cast<float*>(dc_smem + (size_t)(R + 2 * DC_KEYS) * ld + R * PLD);
    float* sF = sS + 2 * R * SLD;             // rescale factor of a row, then its 1 / sum
    __shared__ __align__(8) uint64_t full[2];
    __shared__ int abort_flag;
    const uint32_t bars = ns_smem_u32(full);
    if (tid == 0) {
        abort_flag = 0;
        ns_mbar_init(bars, 1);
        ns_mbar_init(bars + 8, 1);
        ns_fence_barrier_init();
        ns_fence_proxy_async();
    }
    __syncthreads();
    ns_pdl_wait();
    ns_pdl_trigger();
    const int b = blockIdx.z, row0 = blockIdx.y * R, split = blockIdx.x;
    const int slot = a.slots[b], pos0 = a.pos[slot];
    const uint16_t* ring = a.ring + (int64_t)slot * a.ring_slot_stride;
    const int first = a.window > 0 ? max(0, pos0 - a.window + 1) : 0, last = pos0 + a.steps - 1;
    const int tiles = (last - first) / DC_KEYS + 1, per = (tiles + a.splits - 1) / a.splits;
    const int tb = split * per, te = min(tiles, tb + per);

    // Warp 0 orders the rows of a tile as one bulk copy each; rows past the last position become zero.
    auto load_tile = [&](int t, int stage) {
        const int p0 = first + t * DC_KEYS, count = min(DC_KEYS, last - p0 + 1);
        if (warp == 0) {
            const uint32_t bar = bars + 8 * stage, bytes = a.ring_ld * 2;
            if (lane == 0) ns_mbar_expect_tx(bar, count * bytes);
            __syncwarp();
            for (int r = lane; r < count; r += 32)
                bulk_load(sC + (stage * DC_KEYS + r) * ld * 2, ring + (int64_t)((p0 + r) % a.ring_len) * a.ring_ld, bytes, bar);
        } else if (count < DC_KEYS) {
            for (int r = count + warp - 1; r < DC_KEYS; r += 7)
                for (int c = lane * 8; c < a.ring_ld; c += 256) ns_st_shared_v4(sC + ((stage * DC_KEYS + r) * ld + c) * 2, 0, 0, 0, 0);
        }
    };
    if (tb < te) load_tile(tb, 0);

    for (int r = warp; r < R; r += 8) {
        const bool in = row0 + r < a.rows;
        const uint16_t* src = a.q + ((int64_t)b * a.rows + (in ? row0 + r : 0)) * a.width;
        for (int c = lane * 8; c < a.wp; c += 256) ns_copy8(sQ + (r * ld + c) * 2, src + (c < a.width ? c : 0), in ? a.width - c : 0, (a.width & 7) == 0);
    }
    // columns past the cached row stay zero
    for (int r = warp; r < 2 * DC_KEYS; r += 8)
        for (int c = a.ring_ld + lane * 8; c < a.wp; c += 256) ns_st_shared_v4(sC + (r * ld + c) * 2, 0, 0, 0, 0);
    ns_cp_commit();
    ns_cp_wait<0>();
    __syncthreads();

    float acc[MT][NW][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int j = 0; j < NW; j++)
#pragma unroll
            for (int k = 0; k < 4; k++) acc[i][j][k] = 0.0f;
    // warp w keeps maximum and sum of rows w * 2 * MT .. of the tile
    float m[2 * MT], l[2 * MT];
#pragma unroll
    for (int i = 0; i < 2 * MT; i++) { m[i] = -INFINITY; l[i] = 0.0f; }

    for (int t = tb; t < te; t++) {
        const int stage = (t - tb) & 1;
        if (t + 1 < te) load_tile(t + 1, stage ^ 1);
        const bool ok = ns_mbar_wait(bars + 8 * stage, ((t - tb) >> 1) & 1, &abort_flag, a.status, 700);
        if (__syncthreads_or(!ok)) break;
        const uint32_t tC = sC + stage * DC_KEYS * ld * 2;
        // scores: four warps share the keys, 8 each, for the first half of the columns, four for the second
        const int kq = (warp & 3) * 8, half = warp >> 2, k_mid = (a.wp / 32 + 1) / 2 * 32;
        float s[MT][4], s2[MT][4];
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) s[i][k] = s2[i][k] = 0.0f;
#pragma unroll 4
        for (int k = half ? k_mid : 0; k < (half ? a.wp : k_mid); k += 32) {
            uint32_t bf[4];
            ns_ldsm4(bf, tC + ((kq + (lane & 7)) * ld + k + (lane >> 3) * 8) * 2);
#pragma unroll
            for (int i = 0; i < MT; i++) {
                uint32_t af[4], ag[4];
                ns_ldsm4(af, ns_addr_a(sQ, ld, i * 16, k, lane));
                ns_ldsm4(ag, ns_addr_a(sQ, ld, i * 16, k + 16, lane));
                ns_mma_bf16(s[i], af, bf[0], bf[1]);
                ns_mma_bf16(s2[i], ag, bf[2], bf[3]);
            }
        }
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) sS[(half * R + i * 16 + g + (k >> 1) * 8) * SLD + kq + t4 * 2 + (k & 1)] = s[i][k] + s2[i][k];
        __syncthreads();
        const int key = first + t * DC_KEYS + lane;
#pragma unroll
        for (int i = 0; i < 2 * MT; i++) {
            const int r = warp * 2 * MT + i, at = pos0 + (row0 + r) / a.heads;
            const bool see = key <= at && (a.window <= 0 || key > at - a.window);
            const float s0 = see ? (sS[r * SLD + lane] + sS[(R + r) * SLD + lane]) * a.scale2 : -INFINITY;
            float mt = s0;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
            const float mn = fmaxf(m[i], mt), base = mn == -INFINITY ? 0.0f : mn;
            const float f = ns_exp2(m[i] - base), e0 = ns_exp2(s0 - base);
            l[i] = fmaf(l[i], f, ns_warp_sum(e0));
            m[i] = mn;
            asm volatile("st.shared.b16 [%0], %1;" ::"r"(sP + (r * PLD + lane) * 2), "h"(ns_f32_to_bf16_bits(e0)) : "memory");
            if (lane == 0) sF[r] = f;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const float f0 = sF[i * 16 + g], f1 = sF[i * 16 + g + 8];
#pragma unroll
            for (int j = 0; j < NW; j++) { acc[i][j][0] *= f0; acc[i][j][1] *= f0; acc[i][j][2] *= f1; acc[i][j][3] *= f1; }
        }
#pragma unroll
        for (int k = 0; k < DC_KEYS / 16; k++) {
            uint32_t pf[MT][4];
#pragma unroll
            for (int i = 0; i < MT; i++) ns_ldsm4(pf[i], ns_addr_a(sP, PLD, i * 16, k * 16, lane));
#pragma unroll
            for (int j = 0; j < NW / 2; j++) {
                const int n = warp * NW * 8 + j * 16;
                if (n >= a.wp) continue;          // columns past the cached row: nothing is stored from them
                uint32_t bf[4];
                ns_ldsm4_t(bf, ns_addr_bt(tC, ld, k * 16, n, lane));
#pragma unroll
                for (int i = 0; i < MT; i++) {
                    ns_mma_bf16(acc[i][2 * j], pf[i], bf[0], bf[1]);
                    ns_mma_bf16(acc[i][2 * j + 1], pf[i], bf[2], bf[3]);
                }
            }
        }
        __syncthreads();
    }

    if (abort_flag != 0) {                    // copies of this CTA may still be in flight: leave them time to land
        const long long t0 = clock64();
        while (clock64() - t0 < 400000) { }
    }
    if (a.splits == 1) {
#pragma unroll
        for (int i = 0; i < 2 * MT; i++)
            if (lane == 0) sF[warp * 2 * MT + i] = 1.0f / l[i];
        __syncthreads();
    } else {
#pragma unroll
        for (int i = 0; i < 2 * MT; i++) {
            const int r = row0 + warp * 2 * MT + i;
            if (lane == 0 && r < a.rows) {
                float* p = a.part + (((int64_t)b * a.rows + r) * a.splits + split) * (a.rank + 2) + a.rank;
                p[0] = m[i];
                p[1] = l[i];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int rr = i * 16 + g + h * 8, r = row0 + rr;
            if (r >= a.rows) continue;
            const float inv = a.splits == 1 ? sF[rr] : 1.0f;
#pragma unroll
            for (int j = 0; j < NW; j++)
#pragma unroll
                for (int k = 0; k < 2; k++) {
                    const int c = warp * NW * 8 + j * 8 + t4 * 2 + k;
                    if (c >= a.rank) continue;
                    const float v = acc[i][j][2 * h + k] * inv;
                    if (a.splits == 1) a.o[((int64_t)b * a.rows + r) * a.rank + c] = ns_f32_to_bf16_bits(v);
                    else a.part[(((int64_t)b * a.rows + r) * a.splits + split) * (a.rank + 2) + c] = v;
                }
        }
}

// the splits of a row, in split order
__global__ void __launch_bounds__(128) ns_latent_combine_kernel(const float* __restrict__ part, int splits, int rank, uint16_t* __restrict__ o)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const float* p = part + (int64_t)blockIdx.x * splits * (rank + 2);
    float m = -INFINITY, l = 0.0f;
    for (int s = 0; s < splits; s++) m = fmaxf(m, p[s * (rank + 2) + rank]);
    for (int s = 0; s < splits; s++) l = fmaf(p[s * (rank + 2) + rank + 1], ns_exp2(p[s * (rank + 2) + rank] - m), l);
    const float inv = 1.0f / l;
    for (int c = threadIdx.x; c < rank; c += 128) {
        float v = 0.0f;
        for (int s = 0; s < splits; s++) v = fmaf(p[s * (rank + 2) + c], ns_exp2(p[s * (rank + 2) + rank] - m), v);
        o[(int64_t)blockIdx.x * rank + c] = ns_f32_to_bf16_bits(v * inv);
    }
}

// ---------------------------------------------------------------------------------------------
// per-head product, 64 x 64 tiles, k in pieces of 64
// ---------------------------------------------------------------------------------------------
struct HeadTcArgs {
    const uint16_t* x; int64_t x_ld; int x_head;
    const uint16_t* w; int64_t w_head, w_ld;     // [n, k] rows (KN = false) or [k, n] rows (KN = true) of w_ld elements
    void* y; int64_t y_ld; int y_head;
    int rows, k, n, vec_x, vec_w;
};

template <bool KN, typename TY>
__global__ void __launch_bounds__(128) ns_head_matmul_tc_kernel(const HeadTcArgs a)
{
    constexpr int LD = 72;
    __shared__ __align__(16) uint16_t xs[2][64 * LD], ws[2][64 * LD];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int head = blockIdx.z, r0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const uint16_t* x = a.x + (int64_t)head * a.x_head;
    const uint16_t* w = a.w + (int64_t)head * a.w_head;
    auto load = [&](int k0, int s) {
        for (int e = tid; e < 512; e += 128) {
            const int r = e >> 3, c = (e & 7) * 8;
            const bool in = r0 + r < a.rows && k0 + c < a.k;
            ns_copy8(ns_smem_u32(&xs[s][r * LD + c]), x + (in ? (int64_t)(r0 + r) * a.x_ld + k0 + c : 0), in ? a.k - k0 - c : 0, a.vec_x);
            const int wr = KN ? k0 + r : n0 + r, wc = KN ? n0 + c : k0 + c;
            const bool win = wr < (KN ? a.k : a.n) && wc < (KN ? a.n : a.k);
            ns_copy8(ns_smem_u32(&ws[s][r * LD + c]), w + (win ? (int64_t)wr * a.w_ld + wc : 0), win ? (KN ? a.n : a.k) - wc : 0, a.vec_w);
        }
        ns_cp_commit();
    };
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[j][i] = 0.0f;
    const int pieces = (a.k + 63) / 64;
    load(0, 0);
    for (int p = 0; p < pieces; p++) {
        if (p + 1 < pieces) {
            load((p + 1) * 64, (p + 1) & 1);
            ns_cp_wait<1>();
        } else {
            ns_cp_wait<0>();
        }
        __syncthreads();
        const uint32_t tx = ns_smem_u32(xs[p & 1]), tw = ns_smem_u32(ws[p & 1]);
#pragma unroll
        for (int k = 0; k < 64; k += 16) {
            uint32_t af[4];
            ns_ldsm4(af, ns_addr_a(tx, LD, warp * 16, k, lane));
#pragma unroll
            for (int j = 0; j < 4; j++) {
                uint32_t bf[4];
                if (KN) ns_ldsm4_t(bf, ns_addr_bt(tw, LD, k, j * 16, lane));
                else ns_ldsm4(bf, ns_addr_b(tw, LD, j * 16, k, lane));
                ns_mma_bf16(acc[2 * j], af, bf[0], bf[1]);
                ns_mma_bf16(acc[2 * j + 1], af, bf[2], bf[3]);
            }
        }
        __syncthreads();
    }
    TY* y = reinterpret_cast<TY*>(a.y) + (int64_t)head * a.y_head;
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int r = r0 + warp * 16 + g + (i >> 1) * 8, c = n0 + j * 8 + t4 * 2 + (i & 1);
            if (r < a.rows && c < a.n) ns_store(y + (int64_t)r * a.y_ld + c, acc[j][i]);
        }
}

template <int NV, int KS, bool TMA>
int launch_prefill(NsDevice* d, const PrefillMaps& maps, const PrefillArgs& a, int batch)
{
    constexpr size_t rows = ((size_t)2 * PF_KEYS * (KS * 16 + 8) + 2 * PF_KEYS * (NV * 8 + 8)) * 2;
    constexpr size_t boxes = 1024 + 2 * ((size_t)KS / 4 + (NV + 7) / 8) * PF_BOX, q_end = 1024 + 2 * (size_t)(KS / 4) * PF_BOX + PF_ROWS * (KS * 16 + 8) * 2;
    constexpr size_t smem = TMA ? (boxes > q_end ? boxes : q_end) : rows;
    static_assert(smem <= 227 * 1024, "tiles do not fit shared memory");
    auto k = ns_latent_prefill_kernel<NV, KS, TMA>;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    NS_CUDA(ns_launch_plain(k, dim3((a.steps + PF_ROWS - 1) / PF_ROWS, a.heads, batch), dim3(128), smem, d->stream, maps, a));
    return NS_OK;
}

template <int NV>
int dispatch_prefill(NsDevice* d, const PrefillMaps& maps, const PrefillArgs& a, int batch, int boxes)
{
    if (boxes == 0) {
        const int dk = a.dim + a.rot;
        if (dk <= 64) return launch_prefill<NV, 4, false>(d, maps, a, batch);
        if (dk <= 128) return launch_prefill<NV, 8, false>(d, maps, a, batch);
        if (dk <= 192) return launch_prefill<NV, 12, false>(d, maps, a, batch);
        return launch_prefill<NV, 16, false>(d, maps, a, batch);
    }
    if (boxes == 1) return launch_prefill<NV, 4, true>(d, maps, a, batch);
    if (boxes == 2) return launch_prefill<NV, 8, true>(d, maps, a, batch);
    if (boxes == 3) return launch_prefill<NV, 12, true>(d, maps, a, batch);
    return launch_prefill<NV, 16, true>(d, maps, a, batch);
}

template <int MT, int NW>
int launch_decode(NsDevice* d, const DecodeArgs& a, int batch)
{
    constexpr int R = MT * 16;
    const size_t smem = ((size_t)(R + 2 * DC_KEYS) * (a.wp + 8) + R * (DC_KEYS + 8)) * 2 + (size_t)(2 * R * (DC_KEYS + 4) + R) * 4;
    NS_REQUIRE(smem <= 227 * 1024, NS_ERR_ARGUMENT, "ns_latent_decode: cached rows of %d values do not fit shared memory", a.width);
    auto k = ns_latent_decode_kernel<MT, NW>;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    NS_CUDA(ns_launch_plain(k, dim3(a.splits, (a.rows + R - 1) / R, batch), dim3(256), smem, d->stream, a));
    return NS_OK;
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }
#define I32P(x) reinterpret_cast<const int32_t*>(x)
#define U16P(x) reinterpret_cast<const uint16_t*>(x)

extern "C" int ns_latent_gather(ns_device_t h, uint64_t ring, int64_t ring_slot_stride, int ring_len, int ring_ld, int past, uint64_t slots, uint64_t pos, int batch,
                                int rows, uint64_t keys)
{
    NS_ENTER(h);
    NS_REQUIRE(ring && slots && pos && keys && batch > 0 && batch <= 65535 && rows > 0 && past >= 0 && rows <= ring_len, NS_ERR_ARGUMENT, "ns_latent_gather: bad argument");
    NS_REQUIRE(ring_ld % 8 == 0 && ring_slot_stride % 8 == 0 && ((ring | keys) & 15) == 0, NS_ERR_ARGUMENT, "ns_latent_gather: rows are not multiples of 16 bytes");
    const int blocks = (rows + 3) / 4;
    NS_CUDA(ns_launch_plain(ns_latent_gather_kernel, dim3(blocks < 256 ? blocks : 256, batch), dim3(128), 0, d->stream, U16P(ring), ring_slot_stride, ring_len, ring_ld,
                            past, I32P(slots), I32P(pos), rows, reinterpret_cast<uint16_t*>(keys)));
    return NS_OK;
}

extern "C" int ns_latent_prefill(ns_device_t h, uint64_t q, int64_t q_ld, uint64_t kv, int64_t kv_ld, uint64_t keys, int64_t keys_ld, int rank, uint64_t slots,
                                 uint64_t pos, int batch, int steps, int heads, int dim, int rot_dim, int vdim, int past, int window, float scale, uint64_t o,
                                 int64_t o_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(q && kv && keys && slots && pos && o && batch > 0 && batch <= 65535 && steps > 0 && heads > 0 && heads <= 65535, NS_ERR_ARGUMENT,
               "ns_latent_prefill: bad argument");
    NS_REQUIRE(dim > 0 && rot_dim >= 0 && dim + rot_dim <= 256 && vdim > 0 && vdim <= 256 && rank > 0 && past >= 0 && window >= 0, NS_ERR_ARGUMENT, "ns_latent_prefill: bad sizes");
    NS_REQUIRE(kv_ld >= (int64_t)heads * (dim + vdim) && q_ld >= (int64_t)heads * (dim + rot_dim) && keys_ld >= rank + rot_dim && o_ld >= (int64_t)heads * vdim,
               NS_ERR_ARGUMENT, "ns_latent_prefill: rows too short");
    PrefillArgs a;
    a.q = U16P(q); a.q_ld = q_ld; a.kv = U16P(kv); a.kv_ld = kv_ld; a.keys = U16P(keys); a.keys_ld = keys_ld; a.rank = rank;
    a.o = reinterpret_cast<uint16_t*>(o); a.o_ld = o_ld; a.slots = I32P(slots); a.pos = I32P(pos);
    a.steps = steps; a.heads = heads; a.dim = dim; a.rot = rot_dim; a.vdim = vdim; a.past = past; a.nk = past + steps; a.window = window;
    a.scale2 = scale * LOG2E;
    a.vec = ((dim | rot_dim | vdim | rank | (int)q_ld | (int)kv_ld | (int)keys_ld) & 7) == 0 && ((q | kv | keys) & 15) == 0;
    a.status = d->status_dev;
    a.dim_boxes = (dim + 63) / 64;
    const int boxes = a.dim_boxes + (rot_dim + 63) / 64;
    const bool tma = a.vec && boxes <= 4 && (int64_t)batch * a.nk < (1ll << 31);
    PrefillMaps maps;
    memset(&maps, 0, sizeof(maps));
    if (tma) {
        const uint64_t rows = (uint64_t)batch * a.nk;
        const uint32_t box[2] = {64, 64};
        const uint64_t kv_dims[2] = {(uint64_t)kv_ld, rows}, kv_strides[1] = {(uint64_t)kv_ld * 2};
        const uint64_t key_dims[2] = {(uint64_t)keys_ld, rows}, key_strides[1] = {(uint64_t)keys_ld * 2};
        int rc = ns_make_tensor_map(&maps.kv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.kv, kv_dims, kv_strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
        if (rc == NS_OK) rc = ns_make_tensor_map(&maps.keys, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.keys, key_dims, key_strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
        if (rc != NS_OK) return rc;
    }
    const int n = tma ? boxes : 0;
    if (vdim <= 32) return dispatch_prefill<4>(d, maps, a, batch, n);
    if (vdim <= 64) return dispatch_prefill<8>(d, maps, a, batch, n);
    if (vdim <= 128) return dispatch_prefill<16>(d, maps, a, batch, n);
    return dispatch_prefill<32>(d, maps, a, batch, n);
}

extern "C" int ns_latent_decode(ns_device_t h, uint64_t q, uint64_t ring, int64_t ring_slot_stride, int ring_len, int ring_ld, int rank, int width, int window,
                                float scale, uint64_t slots, uint64_t pos, int batch, int steps, int heads, uint64_t o)
{
    NS_ENTER(h);
    NS_REQUIRE(q && ring && slots && pos && o && batch > 0 && batch <= 65535 && steps > 0 && heads > 0, NS_ERR_ARGUMENT, "ns_latent_decode: bad argument");
    NS_REQUIRE(rank > 0 && rank <= 1024 && width >= rank && ring_ld >= width && ring_ld % 8 == 0 && ring_slot_stride % 8 == 0 && window >= 0 && ((ring | q) & 15) == 0,
               NS_ERR_ARGUMENT, "ns_latent_decode: bad sizes");
    NS_REQUIRE(window == 0 || window - 1 + steps <= ring_len, NS_ERR_ARGUMENT, "ns_latent_decode: a window of %d and %d tokens need more than %d ring rows", window,
               steps, ring_len);
    DecodeArgs a;
    a.q = U16P(q); a.ring = U16P(ring); a.ring_slot_stride = ring_slot_stride; a.ring_len = ring_len; a.ring_ld = ring_ld;
    a.rank = rank; a.width = width; a.wp = (width + 31) / 32 * 32; a.window = window; a.scale2 = scale * LOG2E;
    a.slots = I32P(slots); a.pos = I32P(pos); a.steps = steps; a.heads = heads; a.rows = steps * heads;
    a.o = reinterpret_cast<uint16_t*>(o);
    a.part = nullptr;
    a.status = d->status_dev;
    const bool two = a.rows > 16 && rank <= 512;
    const int R = two ? 32 : 16;
    const int64_t ctas = (int64_t)batch * ((a.rows + R - 1) / R);
    NS_REQUIRE((a.rows + R - 1) / R <= 65535, NS_ERR_ARGUMENT, "ns_latent_decode: too many rows");
    // about two CTAs per SM, at least two tiles of keys each
    const int span = window > 0 ? window - 1 + steps : ring_len;
    int splits = (int)(2 * d->sm_count / ctas);
    const int most = (span / DC_KEYS + 1) / 2;
    if (splits > most) splits = most;
    if (splits > 16) splits = 16;
    a.splits = splits < 1 ? 1 : splits;
    if (a.splits > 1) {
        void* block = nullptr;
        int rc = ns_scratch_reserve(d, (size_t)batch * a.rows * a.splits * (rank + 2) * 4, &block);
        if (rc != NS_OK) return rc;
        a.part = reinterpret_cast<float*>(block);
    }
    int rc;
    if (rank <= 128) rc = two ? launch_decode<2, 2>(d, a, batch) : launch_decode<1, 2>(d, a, batch);
    else if (rank <= 256) rc = two ? launch_decode<2, 4>(d, a, batch) : launch_decode<1, 4>(d, a, batch);
    else if (rank <= 512) rc = two ? launch_decode<2, 8>(d, a, batch) : launch_decode<1, 8>(d, a, batch);
    else rc = launch_decode<1, 16>(d, a, batch);
    if (rc != NS_OK || a.splits == 1) return rc;
    NS_CUDA(ns_launch_plain(ns_latent_combine_kernel, dim3((unsigned)(batch * a.rows)), dim3(128), 0, d->stream, a.part, a.splits, rank, a.o));
    return NS_OK;
}

// bf16 operands on the tensor cores; w rows contiguous along k (w_k == 1) or n (w_n == 1)
int ns_head_matmul_tc(NsDevice* d, uint64_t x, int64_t x_ld, int x_head, uint64_t w, int64_t w_head, int64_t w_k, int64_t w_n, int y_dtype, uint64_t y, int64_t y_ld,
                      int y_head, int rows, int heads, int k, int n)
{
    HeadTcArgs a;
    a.x = U16P(x); a.x_ld = x_ld; a.x_head = x_head; a.w = U16P(w); a.w_head = w_head;
    const bool kn = w_n == 1;
    a.w_ld = kn ? w_k : w_n;
    a.y = reinterpret_cast<void*>(y); a.y_ld = y_ld; a.y_head = y_head; a.rows = rows; a.k = k; a.n = n;
    a.vec_x = ((x_ld | x_head) & 7) == 0 && (x & 15) == 0;
    a.vec_w = ((w_head | a.w_ld) & 7) == 0 && (w & 15) == 0;
    const dim3 grid((n + 63) / 64, (rows + 63) / 64, heads);
    auto go = [&](auto kern) -> int {
        NS_CUDA(ns_launch_plain(kern, grid, dim3(128), 0, d->stream, a));
        return NS_OK;
    };
    if (y_dtype == NS_F32) return kn ? go(ns_head_matmul_tc_kernel<true, float>) : go(ns_head_matmul_tc_kernel<false, float>);
    return kn ? go(ns_head_matmul_tc_kernel<true, uint16_t>) : go(ns_head_matmul_tc_kernel<false, uint16_t>);
}
