// Grouped-query attention over a sliding window, with optional parts: normalised queries and keys, a learned sink in the
// softmax's denominator, one gate per head on the output.
//
// The cache of a sequence is two rings per key/value head, keys [ring_len, k_ld] and values [ring_len, v_ld], addressed by position
// modulo ring_len.  ring_len is a multiple of 128, so a tile of up to 128 positions that starts at a multiple of its own
// length is contiguous: every kernel walks such tiles in place and masks what lies outside the window by position.
// Columns that pad a row stay zero, and rings are cleared when a sequence opens, so a masked row holds finite numbers.
//
//   ns_window_append   [queries | keys | values | gates] of a row -> normalised queries, ring rows, sigmoid gates
//   ns_window_attend   32-bit throughout, a warp per row and head (float32 models)
//   ns_window_decode   few tokens, bf16 on the tensor cores: the rows of all query heads of a key/value head share a tile's read
// A prompt's portion in bf16 goes through ns_window_prefill (ns_attention_prefill.cu).
//
// The reference's cached attention (MultiHeadAttention.ForwardCached, src/NeuralSharp/Layers/Attention.cs:98-118) sees every
// earlier position and has none of the optional parts.
#include <math.h>

#include "ns_mma.cuh"
#include "ns_seq.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

struct Rings {
    void* k;                       // slot 0's [kv_heads, ring_len, k_ld]
    void* v;                       // slot 0's [kv_heads, ring_len, v_ld]
    int64_t k_slot_stride, v_slot_stride;
    int ring_len, k_ld, v_ld;
};

// ---------------------------------------------------------------------------------------------
// append
// ---------------------------------------------------------------------------------------------
struct AppendArgs {
    NsSource src;
    int q_col, k_col, v_col, g_col;
    int heads, kv_heads, dim, vdim;
    const float* q_norm;           // [heads * dim] or null
    const float* k_norm;           // [kv_heads * dim] or null
    float eps;
    const int32_t* slots;
    const int32_t* pos;
    int steps;
    void* q;                       // [rows, heads, k_ld]
    float* gate;                   // [rows, heads] or null
    Rings r;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ns_window_append_kernel(const AppendArgs a)
{
    extern __shared__ float4 wa_smem[];
    float* x = reinterpret_cast<float*>(wa_smem);              // queries, then keys
    __shared__ float red[2][8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, tid = threadIdx.x;
    const int slot = a.slots[b], at = (a.pos[slot] + row % a.steps) % a.r.ring_len;
    const int64_t base = (int64_t)row * a.src.ld;
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    T* q = reinterpret_cast<T*>(a.q) + (int64_t)row * a.heads * a.r.k_ld;
    T* k = reinterpret_cast<T*>(a.r.k) + (int64_t)slot * a.r.k_slot_stride + (int64_t)at * a.r.k_ld;
    T* v = reinterpret_cast<T*>(a.r.v) + (int64_t)slot * a.r.v_slot_stride + (int64_t)at * a.r.v_ld;
    const int64_t k_head = (int64_t)a.r.ring_len * a.r.k_ld, v_head = (int64_t)a.r.ring_len * a.r.v_ld;
    float sq = 0.0f, sk = 0.0f;
    if (VEC) {
        for (int c = tid * 4; c < nq + nk; c += 1024) {
            const bool query = c < nq;
            const float4 t = ns_source_at4(a.src, base + (query ? a.q_col + c : a.k_col + c - nq));
            *reinterpret_cast<float4*>(x + c) = t;
            const float s = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, t.w * t.w)));
            if (query) sq += s;
            else sk += s;
        }
        for (int c = tid * 4; c < nv; c += 1024) {
            const int head = c / a.vdim;
            ns_store4(v + head * v_head + c - head * a.vdim, ns_source_at4(a.src, base + a.v_col + c));
        }
    } else {
        for (int c = tid; c < nq + nk; c += 256) {
            const bool query = c < nq;
            const float t = ns_source_at(a.src, base + (query ? a.q_col + c : a.k_col + c - nq));
            x[c] = t;
            if (query) sq = fmaf(t, t, sq);
            else sk = fmaf(t, t, sk);
        }
        for (int c = tid; c < nv; c += 256) {
            const int head = c / a.vdim;
            ns_store(v + head * v_head + c - head * a.vdim, ns_source_at(a.src, base + a.v_col + c));
        }
    }
    if (a.gate != nullptr)
        for (int c = tid; c < a.heads; c += 256) a.gate[(int64_t)row * a.heads + c] = ns_sigmoid(ns_source_at(a.src, base + a.g_col + c));
    const float fq = 1.0f / sqrtf(ns_cta_sum(sq, red[0]) / (float)nq + a.eps);
    const float fk = 1.0f / sqrtf(ns_cta_sum(sk, red[1]) / (float)nk + a.eps);
    if (VEC) {
        for (int c = tid * 4; c < nq + nk; c += 1024) {
            float4 t = *reinterpret_cast<const float4*>(x + c);
            const bool query = c < nq;
            const int cc = query ? c : c - nq, head = cc / a.dim;
            const float* w = query ? a.q_norm : a.k_norm;
            if (w != nullptr) {
                const float4 g = __ldg(reinterpret_cast<const float4*>(w + cc));
                const float f = query ? fq : fk;
                t = make_float4(t.x * f * g.x, t.y * f * g.y, t.z * f * g.z, t.w * f * g.w);
            }
            T* dst = query ? q + head * a.r.k_ld : k + head * k_head;
            ns_store4(dst + cc - head * a.dim, t);
        }
    } else {
        for (int c = tid; c < nq + nk; c += 256) {
            const bool query = c < nq;
            const int cc = query ? c : c - nq, head = cc / a.dim;
            const float* w = query ? a.q_norm : a.k_norm;
            T* dst = query ? q + head * a.r.k_ld : k + head * k_head;
            ns_store(dst + cc - head * a.dim, w != nullptr ? x[c] * (query ? fq : fk) * w[cc] : x[c]);
        }
    }
    const int pad = a.r.k_ld - a.dim;
    for (int c = tid; c < a.heads * pad; c += 256) ns_store(q + (c / pad) * a.r.k_ld + a.dim + c % pad, 0.0f);
}

// The same from one bf16 matrix whose columns come in eights (a prompt's portion): Q groups of eight query or key values of a row per
// thread in registers, values moved as they are.  k_magic, v_magic: group index -> head, head = index * magic >> 32.
template <int Q>
__global__ void __launch_bounds__(256) ns_window_append_rows_kernel(const AppendArgs a, uint32_t k_magic, uint32_t v_magic)
{
    __shared__ float2 red[8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, tid = threadIdx.x;
    const int slot = a.slots[b], at = (a.pos[slot] + row - b * a.steps) % a.r.ring_len;
    const uint16_t* src = reinterpret_cast<const uint16_t*>(a.src.ptr) + (int64_t)row * a.src.ld;
    const int per_k = a.dim / 8, per_v = a.vdim / 8, nq = a.heads * per_k, n = nq + a.kv_heads * per_k, nv = a.kv_heads * per_v;
    uint4 x[Q];
    float sq = 0.0f, sk = 0.0f;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int p = tid + 256 * i;
        x[i] = make_uint4(0, 0, 0, 0);
        if (p < n) x[i] = *reinterpret_cast<const uint4*>(src + (p < nq ? a.q_col + p * 8 : a.k_col + (p - nq) * 8));
    }
    uint16_t* v = reinterpret_cast<uint16_t*>(a.r.v) + (int64_t)slot * a.r.v_slot_stride + (int64_t)at * a.r.v_ld;
    for (int p = tid; p < nv; p += 256) {
        const int head = (int)__umulhi((uint32_t)p, v_magic);
        *reinterpret_cast<uint4*>(v + (int64_t)head * a.r.ring_len * a.r.v_ld + (p - head * per_v) * 8) = *reinterpret_cast<const uint4*>(src + a.v_col + p * 8);
    }
    if (a.gate != nullptr)
        for (int c = tid; c < a.heads; c += 256) a.gate[(int64_t)row * a.heads + c] = ns_sigmoid(ns_load(src + a.g_col + c));
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const uint32_t w[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const float lo = __uint_as_float(w[j] << 16), hi = __uint_as_float(w[j] & 0xFFFF0000u);
            s = fmaf(lo, lo, fmaf(hi, hi, s));
        }
        if (tid + 256 * i < nq) sq += s;
        else sk += s;
    }
    sq = ns_warp_sum(sq);
    sk = ns_warp_sum(sk);
    if ((tid & 31) == 0) red[tid >> 5] = make_float2(sq, sk);
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; w++) { sq += red[w].x; sk += red[w].y; }
    const float fq = 1.0f / sqrtf(sq / (float)(nq * 8) + a.eps), fk = 1.0f / sqrtf(sk / (float)((n - nq) * 8) + a.eps);
    uint16_t* q = reinterpret_cast<uint16_t*>(a.q) + (int64_t)row * a.heads * a.r.k_ld;
    uint16_t* k = reinterpret_cast<uint16_t*>(a.r.k) + (int64_t)slot * a.r.k_slot_stride + (int64_t)at * a.r.k_ld;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int p = tid + 256 * i;
        if (p >= n) continue;
        const bool query = p < nq;
        const int pp = query ? p : p - nq, head = (int)__umulhi((uint32_t)pp, k_magic);
        const float* w = query ? a.q_norm : a.k_norm;
        if (w != nullptr) {
            const float f = query ? fq : fk;
            const float4 w0 = __ldg(reinterpret_cast<const float4*>(w + pp * 8)), w1 = __ldg(reinterpret_cast<const float4*>(w + pp * 8 + 4));
            x[i].x = ns_pack_bf16x2(__uint_as_float(x[i].x << 16) * f * w0.x, __uint_as_float(x[i].x & 0xFFFF0000u) * f * w0.y);
            x[i].y = ns_pack_bf16x2(__uint_as_float(x[i].y << 16) * f * w0.z, __uint_as_float(x[i].y & 0xFFFF0000u) * f * w0.w);
            x[i].z = ns_pack_bf16x2(__uint_as_float(x[i].z << 16) * f * w1.x, __uint_as_float(x[i].z & 0xFFFF0000u) * f * w1.y);
            x[i].w = ns_pack_bf16x2(__uint_as_float(x[i].w << 16) * f * w1.z, __uint_as_float(x[i].w & 0xFFFF0000u) * f * w1.w);
        }
        uint16_t* dst = query ? q + head * a.r.k_ld : k + (int64_t)head * a.r.ring_len * a.r.k_ld;
        *reinterpret_cast<uint4*>(dst + (pp - head * per_k) * 8) = x[i];
    }
}

// ---------------------------------------------------------------------------------------------
// 32-bit attention: a warp per (row, head), a lane per key of a block of 32
// ---------------------------------------------------------------------------------------------
struct WindowArgs {
    const void* q;                 // [rows, heads, k_ld]
    Rings r;
    const float* sink;             // [heads] or null
    const float* gate;             // [rows, heads] or null
    const int32_t* slots;
    const int32_t* pos;
    int steps, heads, kv_heads, dim, vdim, window;
    float scale;
    void* o; int64_t o_ld;         // [rows, heads * vdim]
    // ns_window_decode
    float* part;                   // [batch, kv_heads, rows, splits, vdim + 2]: weighted sum, maximum (log2), sum
    int splits, rows;              // rows = steps * heads / kv_heads, token by token
};

template <typename T, int NR>
__global__ void __launch_bounds__(128) ns_window_attend_kernel(const WindowArgs a)
{
    extern __shared__ float wq_smem[];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y * 4 + warp;
    const int slot = a.slots[b], p = a.pos[slot] + row % a.steps, first = max(0, p - a.window + 1);
    if (head >= a.heads) return;
    const int kvh = head / (a.heads / a.kv_heads);
    float* q = wq_smem + warp * a.dim;
    for (int c = lane; c < a.dim; c += 32) q[c] = ns_load(reinterpret_cast<const T*>(a.q) + ((int64_t)row * a.heads + head) * a.r.k_ld + c);
    __syncwarp();
    const T* keys = reinterpret_cast<const T*>(a.r.k) + (int64_t)slot * a.r.k_slot_stride + (int64_t)kvh * a.r.ring_len * a.r.k_ld;
    const T* values = reinterpret_cast<const T*>(a.r.v) + (int64_t)slot * a.r.v_slot_stride + (int64_t)kvh * a.r.ring_len * a.r.v_ld;
    float m = -INFINITY, l = 0.0f, acc[NR];
    if (a.sink != nullptr) { m = a.sink[head]; l = 1.0f; }      // the sink is a key without a value
#pragma unroll
    for (int j = 0; j < NR; j++) acc[j] = 0.0f;
    for (int j0 = first; j0 <= p; j0 += 32) {
        const int count = min(32, p - j0 + 1);
        float s = -INFINITY;
        if (lane < count) {
            const T* k = keys + (int64_t)((j0 + lane) % a.r.ring_len) * a.r.k_ld;
            float d = 0.0f;
            for (int c = 0; c < a.dim; c++) d = fmaf(q[c], ns_load(k + c), d);
            s = d * a.scale;
        }
        float mt = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
        const float mn = fmaxf(m, mt), f = expf(m - mn), w = expf(s - mn);
        l = fmaf(l, f, ns_warp_sum(w));
        m = mn;
#pragma unroll
        for (int j = 0; j < NR; j++) acc[j] *= f;
        for (int r = 0; r < count; r++) {
            const float wr = __shfl_sync(0xffffffffu, w, r);
            const T* v = values + (int64_t)((j0 + r) % a.r.ring_len) * a.r.v_ld;
#pragma unroll
            for (int j = 0; j < NR; j++) {
                const int c = j * 32 + lane;
                if (c < a.vdim) acc[j] = fmaf(wr, ns_load(v + c), acc[j]);
            }
        }
    }
    const float f = (a.gate != nullptr ? a.gate[(int64_t)row * a.heads + head] : 1.0f) / l;
    T* o = reinterpret_cast<T*>(a.o) + (int64_t)row * a.o_ld + (int64_t)head * a.vdim;
#pragma unroll
    for (int j = 0; j < NR; j++) {
        const int c = j * 32 + lane;
        if (c < a.vdim) ns_store(o + c, acc[j] * f);
    }
}

// ---------------------------------------------------------------------------------------------
// few tokens, bf16: a CTA per (16 rows, key/value head, sequence, share of the window); each of its warps walks tiles of 16 keys on its
// own, with its own maximum, sum and weighted values, and its own copies in flight
// ---------------------------------------------------------------------------------------------
constexpr int WD_KEYS = 16, WD_STAGES = 3;

// KS: 16-wide steps over a key; NV: 8-wide column tiles of a value; WARPS: 2 where there are several CTAs per SM (short CTAs fill the SMs
// more evenly: 53 us against 62 for 64 sequences x 16 heads and 512 positions), else 4
template <int KS, int NV, int WARPS>
struct DecodeSmem {
    static constexpr int KLD = KS * 16 + 8, VLD = NV * 8 + 8, STAGE = WD_KEYS * (KLD + VLD);       // bf16 elements
    static constexpr int OLD = NV * 8 + 4;                                                         // floats of a row when the warps merge
    static constexpr int TILES = WARPS * WD_STAGES * STAGE * 2, MERGE = WARPS * 16 * OLD * 4;
    static constexpr int BYTES = (TILES > MERGE ? TILES : MERGE) + WARPS * 32 * 4;
};

NS_DEVINL void write_out(const WindowArgs& a, int b, int kvh, int r, int c, float weighted, float f)
{
    const int rep = a.heads / a.kv_heads, head = kvh * rep + r % rep;
    const int64_t row = (int64_t)b * a.steps + r / rep;
    reinterpret_cast<uint16_t*>(a.o)[row * a.o_ld + (int64_t)head * a.vdim + c] = ns_f32_to_bf16_bits(weighted * f);
}
// what a row's weighted values (relative to the maximum m) are multiplied with: gate / (sum + sink)
NS_DEVINL float out_factor(const WindowArgs& a, int b, int kvh, int r, float m, float l)
{
    const int rep = a.heads / a.kv_heads, head = kvh * rep + r % rep;
    const int64_t row = (int64_t)b * a.steps + r / rep;
    float f = 1.0f;
    if (a.sink != nullptr) {
        const float s = a.sink[head] * LOG2E, top = fmaxf(m, s);
        f = ns_exp2(m - top);
        l = fmaf(l, f, ns_exp2(s - top));
    }
    if (a.gate != nullptr) f *= a.gate[row * a.heads + head];
    return f / l;
}

template <int KS, int NV, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) ns_window_decode_kernel(const WindowArgs a)
{
    using L = DecodeSmem<KS, NV, WARPS>;
    extern __shared__ __align__(16) uint8_t wd_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const uint32_t mine = ns_smem_u32(wd_smem) + warp * WD_STAGES * L::STAGE * 2;
    float* sO = reinterpret_cast<float*>(wd_smem);
    float* sM = reinterpret_cast<float*>(wd_smem + (L::TILES > L::MERGE ? L::TILES : L::MERGE));    // [warp][16] maxima, then sums
    ns_pdl_wait();
    ns_pdl_trigger();
    const int rep = a.heads / a.kv_heads, tiles_r = (a.rows + 15) / 16;
    const int kvh = blockIdx.y, b = blockIdx.z, row0 = (int)(blockIdx.x % tiles_r) * 16, split = blockIdx.x / tiles_r;
    const int slot = a.slots[b], pos0 = a.pos[slot], k_ld = a.r.k_ld, v_ld = a.r.v_ld;
    // positions that this tile's rows see
    const int last = pos0 + min(row0 + 15, a.rows - 1) / rep, first = max(0, pos0 + row0 / rep - a.window + 1);
    const uint16_t* keys = reinterpret_cast<const uint16_t*>(a.r.k) + (int64_t)slot * a.r.k_slot_stride + (int64_t)kvh * a.r.ring_len * k_ld;
    const uint16_t* values = reinterpret_cast<const uint16_t*>(a.r.v) + (int64_t)slot * a.r.v_slot_stride + (int64_t)kvh * a.r.ring_len * v_ld;
    const int t_last = last / WD_KEYS, stride = WARPS * a.splits;
    int t_load = first / WD_KEYS + split * WARPS + warp;

    // columns between a row's length and the next multiple of 16 are read: zero in every stage
    if (k_ld < KS * 16)
        for (int e = lane; e < WD_STAGES * WD_KEYS; e += 32)
            ns_st_shared_v4(mine + ((e / WD_KEYS) * L::STAGE + (e % WD_KEYS) * L::KLD + k_ld) * 2, 0, 0, 0, 0);

    auto load_tile = [&](int stage) {
        if (t_load <= t_last) {
            const int ring_row = t_load * WD_KEYS % a.r.ring_len;
            const uint32_t sk = mine + stage * L::STAGE * 2, sv = sk + WD_KEYS * L::KLD * 2;
            const uint16_t* kp = keys + (int64_t)ring_row * k_ld;
            const uint16_t* vp = values + (int64_t)ring_row * v_ld;
#pragma unroll
            for (int e = lane; e < WD_KEYS * KS * 2; e += 32) {
                const int r = e / (KS * 2), c = (e % (KS * 2)) * 8;
                if (c < k_ld) ns_cp_async16(sk + (r * L::KLD + c) * 2, kp + r * k_ld + c);
            }
#pragma unroll
            for (int e = lane; e < WD_KEYS * NV; e += 32) {
                const int r = e / NV, c = (e % NV) * 8;
                if (c < v_ld) ns_cp_async16(sv + (r * L::VLD + c) * 2, vp + r * v_ld + c);
            }
        }
        t_load += stride;
        ns_cp_commit();
    };
    int t = t_load;
#pragma unroll
    for (int s = 0; s < WD_STAGES - 1; s++) load_tile(s);

    // query fragments straight from memory
    uint32_t qf[KS][4];
    const uint16_t* q = reinterpret_cast<const uint16_t*>(a.q);
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int r = row0 + g + h * 8;
        const bool in = r < a.rows;
        const int64_t row = in ? (((int64_t)b * a.steps + r / rep) * a.heads + kvh * rep + r % rep) : 0;
        const uint16_t* p = q + row * k_ld + t4 * 2;
#pragma unroll
        for (int k = 0; k < KS; k++) {
            qf[k][h] = in && k * 16 < k_ld ? *reinterpret_cast<const uint32_t*>(p + k * 16) : 0u;
            qf[k][2 + h] = in && k * 16 + 8 < k_ld ? *reinterpret_cast<const uint32_t*>(p + k * 16 + 8) : 0u;
        }
    }
    const int at0 = pos0 + (row0 + g) / rep, at1 = pos0 + (row0 + g + 8) / rep;       // the rows' positions
    const float scale2 = a.scale * LOG2E;
    float acc[NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[j][i] = 0.0f;

    int stage = 0;
    for (; t <= t_last; t += stride) {
        load_tile(stage == 0 ? WD_STAGES - 1 : stage - 1);
        ns_cp_wait<WD_STAGES - 1>();
        __syncwarp();
        const uint32_t sk = mine + stage * L::STAGE * 2, sv = sk + WD_KEYS * L::KLD * 2;
        float s[2][4], s2[2][4];
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[j][i] = s2[j][i] = 0.0f;
#pragma unroll
        for (int k = 0; k < KS; k++) {
            if (k * 16 >= k_ld) continue;
            uint32_t bf[4];
            ns_ldsm4(bf, ns_addr_b(sk, L::KLD, 0, k * 16, lane));
            ns_mma_bf16(k & 1 ? s2[0] : s[0], qf[k], bf[0], bf[1]);
            ns_mma_bf16(k & 1 ? s2[1] : s[1], qf[k], bf[2], bf[3]);
        }
        float f[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int at = h ? at1 : at0;
            float mt = -INFINITY;
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const int key = t * WD_KEYS + j * 8 + t4 * 2 + i;
                    const float x = (s[j][2 * h + i] + s2[j][2 * h + i]) * scale2;
                    s[j][2 * h + i] = key <= at && key > at - a.window ? x : -INFINITY;
                    mt = fmaxf(mt, s[j][2 * h + i]);
                }
            mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 1));
            mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, 2));
            const float mn = fmaxf(m[h], mt), base = mn == -INFINITY ? 0.0f : mn;
            f[h] = ns_exp2(m[h] - base);
            m[h] = mn;
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    s[j][2 * h + i] = ns_exp2(s[j][2 * h + i] - base);
                    sum += s[j][2 * h + i];
                }
            l[h] = fmaf(l[h], f[h], sum);
        }
        if (__any_sync(0xffffffffu, f[0] != 1.0f || f[1] != 1.0f)) {
#pragma unroll
            for (int j = 0; j < NV; j++) { acc[j][0] *= f[0]; acc[j][1] *= f[0]; acc[j][2] *= f[1]; acc[j][3] *= f[1]; }
        }
        const uint32_t pf[4] = {ns_pack_bf16x2(s[0][0], s[0][1]), ns_pack_bf16x2(s[0][2], s[0][3]), ns_pack_bf16x2(s[1][0], s[1][1]),
                                ns_pack_bf16x2(s[1][2], s[1][3])};
#pragma unroll
        for (int j = 0; j < NV / 2; j++) {
            if (j * 16 >= v_ld) continue;
            uint32_t vf[4];
            ns_ldsm4_t(vf, ns_addr_bt(sv, L::VLD, 0, j * 16, lane));
            ns_mma_bf16(acc[2 * j], pf, vf[0], vf[1]);
            ns_mma_bf16(acc[2 * j + 1], pf, vf[2], vf[3]);
        }
        __syncwarp();
        stage = stage + 1 == WD_STAGES ? 0 : stage + 1;
    }
    ns_cp_wait<0>();

    // the warps' results become one
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
    __syncthreads();
    if (t4 == 0)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            sM[warp * 32 + g + h * 8] = m[h];
            sM[warp * 32 + 16 + g + h * 8] = l[h];
        }
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
        for (int h = 0; h < 2; h++)
            *reinterpret_cast<float2*>(sO + (warp * 16 + g + h * 8) * L::OLD + j * 8 + t4 * 2) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
    __syncthreads();
    const int count = min(16, a.rows - row0);
    for (int r = warp; r < count; r += WARPS) {
        float top = -INFINITY, sum = 0.0f, w[WARPS];
#pragma unroll
        for (int i = 0; i < WARPS; i++) top = fmaxf(top, sM[i * 32 + r]);
#pragma unroll
        for (int i = 0; i < WARPS; i++) {
            w[i] = top == -INFINITY ? 0.0f : ns_exp2(sM[i * 32 + r] - top);
            sum = fmaf(sM[i * 32 + 16 + r], w[i], sum);
        }
        const bool whole = a.splits == 1;
        const float f = whole ? out_factor(a, b, kvh, row0 + r, top, sum) : 1.0f;
        float* part = whole ? nullptr : a.part + ((((int64_t)b * a.kv_heads + kvh) * a.rows + row0 + r) * a.splits + split) * (a.vdim + 2);
        for (int c = lane; c < a.vdim; c += 32) {
            float x = 0.0f;
#pragma unroll
            for (int i = 0; i < WARPS; i++) x = fmaf(sO[(i * 16 + r) * L::OLD + c], w[i], x);
            if (whole) write_out(a, b, kvh, row0 + r, c, x, f);
            else part[c] = x;
        }
        if (!whole && lane == 0) {
            part[a.vdim] = top;
            part[a.vdim + 1] = sum;
        }
    }
}

// the shares of a row, in order; a share without a visible key has the maximum -inf and adds nothing
__global__ void __launch_bounds__(128) ns_window_combine_kernel(const WindowArgs a)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int r = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z, n = a.vdim + 2;
    const float* p = a.part + (((int64_t)b * a.kv_heads + kvh) * a.rows + r) * a.splits * n;
    float m = -INFINITY, l = 0.0f;
    for (int s = 0; s < a.splits; s++) m = fmaxf(m, p[s * n + a.vdim]);
    for (int s = 0; s < a.splits; s++) l = fmaf(p[s * n + a.vdim + 1], ns_exp2(p[s * n + a.vdim] - m), l);
    const float f = out_factor(a, b, kvh, r, m, l);
    for (int c = threadIdx.x; c < a.vdim; c += 128) {
        float x = 0.0f;
        for (int s = 0; s < a.splits; s++) x = fmaf(p[s * n + c], ns_exp2(p[s * n + a.vdim] - m), x);
        write_out(a, b, kvh, r, c, x, f);
    }
}

template <typename T, int NR>
int launch_attend(NsDevice* d, const WindowArgs& a, int batch)
{
    const size_t smem = (size_t)4 * a.dim * 4;
    NS_REQUIRE(smem <= 48 * 1024, NS_ERR_ARGUMENT, "ns_window_attend: keys of %d values", a.dim);
    NS_CUDA(ns_launch_plain(ns_window_attend_kernel<T, NR>, dim3((unsigned)(batch * a.steps), (unsigned)((a.heads + 3) / 4)), dim3(128), smem, d->stream, a));
    return NS_OK;
}
template <typename T>
int dispatch_attend(NsDevice* d, const WindowArgs& a, int batch)
{
    if (a.vdim <= 64) return launch_attend<T, 2>(d, a, batch);
    if (a.vdim <= 128) return launch_attend<T, 4>(d, a, batch);
    if (a.vdim <= 256) return launch_attend<T, 8>(d, a, batch);
    return launch_attend<T, 32>(d, a, batch);
}

template <int KS, int NV, int WARPS>
int launch_decode_warps(NsDevice* d, const WindowArgs& a, int batch)
{
    constexpr int smem = DecodeSmem<KS, NV, WARPS>::BYTES;
    static_assert(smem <= 227 * 1024, "a CTA's shared memory");
    auto k = ns_window_decode_kernel<KS, NV, WARPS>;
    NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    NS_CUDA(ns_launch_plain(k, dim3((unsigned)((a.rows + 15) / 16 * a.splits), (unsigned)a.kv_heads, (unsigned)batch), dim3(WARPS * 32), (size_t)smem, d->stream, a));
    return NS_OK;
}
template <int KS, int NV>
int launch_decode(NsDevice* d, const WindowArgs& a, int batch)
{
    const int64_t ctas = (int64_t)batch * a.kv_heads * ((a.rows + 15) / 16) * a.splits;
    return ctas >= 4 * (int64_t)d->sm_count ? launch_decode_warps<KS, NV, 2>(d, a, batch) : launch_decode_warps<KS, NV, 4>(d, a, batch);
}
template <int KS>
int dispatch_decode(NsDevice* d, const WindowArgs& a, int batch)
{
    if (a.r.v_ld <= 64) return launch_decode<KS, 8>(d, a, batch);
    if (a.r.v_ld <= 128) return launch_decode<KS, 16>(d, a, batch);
    return launch_decode<KS, 32>(d, a, batch);
}

bool float_or_bf16(int dtype) { return dtype == NS_F32 || dtype == NS_BF16; }

int rings_of(Rings& r, const char* who, uint64_t k, uint64_t v, int64_t k_slot_stride, int64_t v_slot_stride, int ring_len, int k_ld, int v_ld, int dim, int vdim,
             int window, int steps)
{
    NS_REQUIRE(k && v && ((k | v) & 15) == 0 && k_ld >= dim && v_ld >= vdim && ((k_ld | v_ld) & 7) == 0 && ((k_slot_stride | v_slot_stride) & 7) == 0, NS_ERR_ARGUMENT,
               "%s: bad rings", who);
    NS_REQUIRE(window > 0 && ring_len % 128 == 0 && (int64_t)window - 1 + steps <= ring_len, NS_ERR_ARGUMENT,
               "%s: a window of %d and %d tokens do not fit rings of %d rows (a multiple of 128)", who, window, steps, ring_len);
    r.k = reinterpret_cast<void*>(k); r.v = reinterpret_cast<void*>(v);
    r.k_slot_stride = k_slot_stride; r.v_slot_stride = v_slot_stride;
    r.ring_len = ring_len; r.k_ld = k_ld; r.v_ld = v_ld;
    return NS_OK;
}

int window_args(WindowArgs& a, const char* who, uint64_t q, uint64_t k_ring, uint64_t v_ring, int64_t k_slot_stride, int64_t v_slot_stride, int ring_len, int k_ld,
                int v_ld, uint64_t sink, uint64_t gate, uint64_t slots, uint64_t pos, int batch, int steps, int heads, int kv_heads, int dim, int vdim, int window,
                float scale, uint64_t o, int64_t o_ld)
{
    NS_REQUIRE(q && slots && pos && o && batch > 0 && batch <= 65535 && steps > 0 && (q & 15) == 0, NS_ERR_ARGUMENT, "%s: bad argument", who);
    NS_REQUIRE(heads > 0 && kv_heads > 0 && kv_heads <= 65535 && heads % kv_heads == 0, NS_ERR_ARGUMENT, "%s: %d heads do not divide over %d key/value heads", who, heads,
               kv_heads);
    NS_REQUIRE(dim > 0 && vdim > 0 && o_ld >= (int64_t)heads * vdim, NS_ERR_ARGUMENT, "%s: bad sizes", who);
    int rc = rings_of(a.r, who, k_ring, v_ring, k_slot_stride, v_slot_stride, ring_len, k_ld, v_ld, dim, vdim, window, steps);
    if (rc != NS_OK) return rc;
    a.q = reinterpret_cast<const void*>(q);
    a.sink = reinterpret_cast<const float*>(sink);
    a.gate = reinterpret_cast<const float*>(gate);
    a.slots = reinterpret_cast<const int32_t*>(slots);
    a.pos = reinterpret_cast<const int32_t*>(pos);
    a.steps = steps; a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim; a.window = window; a.scale = scale;
    a.o = reinterpret_cast<void*>(o); a.o_ld = o_ld;
    a.part = nullptr; a.splits = 1; a.rows = steps * (heads / kv_heads);
    return NS_OK;
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }

extern "C" int ns_window_append(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int q_col, int k_col, int v_col, int g_col, int heads, int kv_heads,
                                int dim, int vdim, uint64_t q_norm, uint64_t k_norm, float eps, uint64_t slots, uint64_t pos, int batch, int steps, int dtype,
                                uint64_t q, uint64_t gate, uint64_t k_ring, uint64_t v_ring, int64_t k_slot_stride, int64_t v_slot_stride, int ring_len, int k_ld,
                                int v_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype), NS_ERR_ARGUMENT, "ns_window_append: bad source");
    NS_REQUIRE(q && slots && pos && batch > 0 && steps > 0 && float_or_bf16(dtype) && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0, NS_ERR_ARGUMENT,
               "ns_window_append: bad argument");
    NS_REQUIRE(q_col >= 0 && k_col >= 0 && v_col >= 0 && (gate == 0 || g_col >= 0) && q_col + heads * dim <= src_ld && k_col + kv_heads * dim <= src_ld &&
                   v_col + kv_heads * vdim <= src_ld && (gate == 0 || g_col + heads <= src_ld),
               NS_ERR_ARGUMENT, "ns_window_append: the source has too few columns");
    AppendArgs a;
    int rc = rings_of(a.r, "ns_window_append", k_ring, v_ring, k_slot_stride, v_slot_stride, ring_len, k_ld, v_ld, dim, vdim, 1, steps);
    if (rc != NS_OK) return rc;
    a.src = ns_source(src, splits, src_dtype, (int64_t)batch * steps, src_ld);
    a.q_col = q_col; a.k_col = k_col; a.v_col = v_col; a.g_col = g_col;
    a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim;
    a.q_norm = reinterpret_cast<const float*>(q_norm);
    a.k_norm = reinterpret_cast<const float*>(k_norm);
    a.eps = eps;
    a.slots = reinterpret_cast<const int32_t*>(slots);
    a.pos = reinterpret_cast<const int32_t*>(pos);
    a.steps = steps;
    a.q = reinterpret_cast<void*>(q);
    a.gate = reinterpret_cast<float*>(gate);
    const int groups = (heads + kv_heads) * (dim / 8);
    if (dtype == NS_BF16 && src_dtype == NS_BF16 && ((dim | vdim | q_col | k_col | v_col | src_ld) & 7) == 0 && ((src | q_norm | k_norm | q) & 15) == 0 && groups <= 2048 &&
        kv_heads * (vdim / 8) <= 65535) {
        // head of a group of eight: index * ceil(2^32 / groups per head) >> 32, exact for indexes and sizes below 2^16 (one group
        // per head does not fit 32 bits)
        if (dim > 8 && vdim > 8) {
            const uint32_t k_magic = (uint32_t)(((1ull << 32) + dim / 8 - 1) / (dim / 8)), v_magic = (uint32_t)(((1ull << 32) + vdim / 8 - 1) / (vdim / 8));
            auto rows = [&](auto k) -> int {
                NS_CUDA(ns_launch_plain(k, dim3((unsigned)(batch * steps)), dim3(256), 0, d->stream, a, k_magic, v_magic));
                return NS_OK;
            };
            if (groups <= 512) return rows(ns_window_append_rows_kernel<2>);
            return groups <= 1024 ? rows(ns_window_append_rows_kernel<4>) : rows(ns_window_append_rows_kernel<8>);
        }
    }
    const size_t smem = ((size_t)(heads + kv_heads) * dim + 3) / 4 * 16;
    NS_REQUIRE(smem <= 200 * 1024, NS_ERR_ARGUMENT, "ns_window_append: queries and keys of %zu bytes do not fit shared memory", smem);
    const bool vec = ((dim | vdim | q_col | k_col | v_col | src_ld) & 3) == 0 && ((src | q_norm | k_norm | q) & 15) == 0 && (a.src.slab & 3) == 0;
    auto k = dtype == NS_F32 ? (vec ? ns_window_append_kernel<float, true> : ns_window_append_kernel<float, false>)
                             : (vec ? ns_window_append_kernel<uint16_t, true> : ns_window_append_kernel<uint16_t, false>);
    if (smem > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    NS_CUDA(ns_launch_plain(k, dim3((unsigned)(batch * steps)), dim3(256), smem, d->stream, a));
    return NS_OK;
}

extern "C" int ns_window_attend(ns_device_t h, int dtype, uint64_t q, uint64_t k_ring, uint64_t v_ring, int64_t k_slot_stride, int64_t v_slot_stride, int ring_len,
                                int k_ld, int v_ld, uint64_t sink, uint64_t gate, uint64_t slots, uint64_t pos, int batch, int steps, int heads, int kv_heads, int dim,
                                int vdim, int window, float scale, uint64_t o, int64_t o_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(float_or_bf16(dtype), NS_ERR_ARGUMENT, "ns_window_attend: bad type");
    WindowArgs a;
    int rc = window_args(a, "ns_window_attend", q, k_ring, v_ring, k_slot_stride, v_slot_stride, ring_len, k_ld, v_ld, sink, gate, slots, pos, batch, steps, heads, kv_heads,
                         dim, vdim, window, scale, o, o_ld);
    if (rc != NS_OK) return rc;
    NS_REQUIRE(vdim <= 1024 && heads <= 4 * 65535, NS_ERR_ARGUMENT, "ns_window_attend: values of %d (at most 1024)", vdim);
    return dtype == NS_F32 ? dispatch_attend<float>(d, a, batch) : dispatch_attend<uint16_t>(d, a, batch);
}

extern "C" int ns_window_decode(ns_device_t h, uint64_t q, uint64_t k_ring, uint64_t v_ring, int64_t k_slot_stride, int64_t v_slot_stride, int ring_len, int k_ld,
                                int v_ld, uint64_t sink, uint64_t gate, uint64_t slots, uint64_t pos, int batch, int steps, int heads, int kv_heads, int dim, int vdim,
                                int window, float scale, uint64_t o, int64_t o_ld)
{
    NS_ENTER(h);
    WindowArgs a;
    int rc = window_args(a, "ns_window_decode", q, k_ring, v_ring, k_slot_stride, v_slot_stride, ring_len, k_ld, v_ld, sink, gate, slots, pos, batch, steps, heads, kv_heads,
                         dim, vdim, window, scale, o, o_ld);
    if (rc != NS_OK) return rc;
    NS_REQUIRE(k_ld <= 256 && v_ld <= 256, NS_ERR_ARGUMENT, "ns_window_decode: keys of %d and values of %d (at most 256)", dim, vdim);
    // about two CTAs per SM, two tiles of keys for each warp at least
    const int64_t ctas = (int64_t)batch * kv_heads * ((a.rows + 15) / 16);
    const int tiles = (window - 1 + (steps < 16 ? steps : 16)) / WD_KEYS + 2;
    int64_t splits = 2 * d->sm_count / ctas;
    if (splits > tiles / 8) splits = tiles / 8;
    a.splits = splits < 1 ? 1 : (splits > 32 ? 32 : (int)splits);
    if (a.splits > 1) {
        void* block = nullptr;
        rc = ns_scratch_reserve(d, (size_t)batch * kv_heads * a.rows * a.splits * (vdim + 2) * 4, &block);
        if (rc != NS_OK) return rc;
        a.part = reinterpret_cast<float*>(block);
    }
    if (k_ld <= 64) rc = dispatch_decode<4>(d, a, batch);
    else if (k_ld <= 128) rc = dispatch_decode<8>(d, a, batch);
    else rc = dispatch_decode<16>(d, a, batch);
    if (rc != NS_OK || a.splits == 1) return rc;
    NS_CUDA(ns_launch_plain(ns_window_combine_kernel, dim3((unsigned)a.rows, (unsigned)kv_heads, (unsigned)batch), dim3(128), 0, d->stream, a));
    return NS_OK;
}
