// Latent attention: keys and values of every head are linear in one cached vector per position, [latent | rotated key part],
// and a position sees a sliding window of them.
//
// The cache of a sequence is a ring of `ring_len` rows addressed by position modulo ring_len: with a window of `size` positions
// and steps of at most T tokens, size - 1 + T rows are all that is ever read, whatever the length of the sequence.
//
// Decoding works on the latents themselves: the unrotated query of a head is carried through the head's key matrix
// (ns_head_matmul), attention runs over the cached rows as one shared key / value head, and the weighted latent goes through
// the head's value matrix.  The reference's cache holds full keys and values (KeyValueCache, Layers/Decoding.cs:14-35) and has
// no counterpart.
#include "ns_seq.cuh"

int ns_head_matmul_tc(NsDevice* d, uint64_t x, int64_t x_ld, int x_head, uint64_t w, int64_t w_head, int64_t w_k, int64_t w_n, int y_dtype, uint64_t y, int64_t y_ld,
                      int y_head, int rows, int heads, int k, int n);   // ns_latent_tc.cu

namespace {

// ---------------------------------------------------------------------------------------------
// [query latent | key/value latent | rotated key part] of a row -> normalised query latent, cache row
// ---------------------------------------------------------------------------------------------
struct LatentAppendArgs {
    NsSource src;
    int q_rank, kv_rank, rot_dim, rot_dims;
    const float* q_norm;
    const float* kv_norm;
    float eps;
    const float* freq;        // [rot_dims / 2]
    const int32_t* slots;
    const int32_t* pos;
    int steps;
    void* cq;                 // [rows, cq_ld]
    int cq_ld;
    void* ring;               // slot 0's [ring_len, ring_ld]
    int64_t ring_slot_stride;
    int ring_len, ring_ld;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ns_latent_append_kernel(const LatentAppendArgs a)
{
    extern __shared__ float4 app_smem[];
    float* x = reinterpret_cast<float*>(app_smem);             // the row
    __shared__ float red[2][8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, i = row % a.steps, tid = threadIdx.x;
    const int slot = a.slots[b], p = a.pos[slot] + i;
    const int64_t base = (int64_t)row * a.src.ld;
    const int k1 = a.q_rank + a.kv_rank, n = k1 + a.rot_dim;
    float sq = 0.0f, sc = 0.0f;
    auto sum = [&](int c, float v) {
        if (c < a.q_rank) sq = fmaf(v, v, sq);
        else if (c < k1) sc = fmaf(v, v, sc);
    };
    if (VEC) {
        for (int c = tid * 4; c < n; c += 1024) {
            const float4 v = ns_source_at4(a.src, base + c);
            *reinterpret_cast<float4*>(x + c) = v;
            sum(c, v.x); sum(c + 1, v.y); sum(c + 2, v.z); sum(c + 3, v.w);
        }
    } else {
        for (int c = tid; c < n; c += 256) {
            x[c] = ns_source_at(a.src, base + c);
            sum(c, x[c]);
        }
    }
    const float iq = 1.0f / sqrtf(ns_cta_sum(sq, red[0]) / (float)a.q_rank + a.eps);
    const float ic = 1.0f / sqrtf(ns_cta_sum(sc, red[1]) / (float)a.kv_rank + a.eps);
    T* cq = reinterpret_cast<T*>(a.cq) + (int64_t)row * a.cq_ld;
    T* dst = reinterpret_cast<T*>(a.ring) + (int64_t)slot * a.ring_slot_stride + (int64_t)(p % a.ring_len) * a.ring_ld;
    const float* xc = x + a.q_rank;
    if (VEC) {
        for (int c = tid * 4; c < a.q_rank; c += 1024) {
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.q_norm + c));
            ns_store4(cq + c, make_float4(x[c] * iq * w.x, x[c + 1] * iq * w.y, x[c + 2] * iq * w.z, x[c + 3] * iq * w.w));
        }
        for (int c = tid * 4; c < a.kv_rank; c += 1024) {
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.kv_norm + c));
            ns_store4(dst + c, make_float4(xc[c] * ic * w.x, xc[c + 1] * ic * w.y, xc[c + 2] * ic * w.z, xc[c + 3] * ic * w.w));
        }
    } else {
        for (int c = tid; c < a.q_rank; c += 256) ns_store(cq + c, x[c] * iq * a.q_norm[c]);
        for (int c = tid; c < a.kv_rank; c += 256) ns_store(dst + c, xc[c] * ic * a.kv_norm[c]);
    }
    for (int c = a.q_rank + tid; c < a.cq_ld; c += 256) ns_store(cq + c, 0.0f);
    // a thread per pair, then what passes unturned
    const float* xr = x + k1;
    for (int c = 2 * (255 - tid); c < a.rot_dims; c += 512) {
        float sn, cs;
        sincosf((float)p * a.freq[c >> 1], &sn, &cs);
        ns_store(dst + a.kv_rank + c, fmaf(xr[c], cs, -xr[c + 1] * sn));
        ns_store(dst + a.kv_rank + c + 1, fmaf(xr[c + 1], cs, xr[c] * sn));
    }
    for (int c = a.rot_dims + tid; c < a.rot_dim; c += 256) ns_store(dst + a.kv_rank + c, xr[c]);
    for (int c = a.kv_rank + a.rot_dim + tid; c < a.ring_ld; c += 256) ns_store(dst + c, 0.0f);
}

// ---------------------------------------------------------------------------------------------
// per head [plain | rotated] -> the plain part to one matrix, the rotated part, turned to its position, to another
// ---------------------------------------------------------------------------------------------
struct RotateArgs {
    NsSource src;
    int heads, dim, rot_dim, rot_dims;
    const float* freq;
    const int32_t* slots;
    const int32_t* pos;
    int steps;
    void* plain; int64_t plain_ld; int plain_head;   // element (row, head, c) at row * ld + head * plain_head + c
    void* rot; int64_t rot_ld; int rot_head;
};

template <typename TP, typename TR, bool VEC>
__global__ void __launch_bounds__(256) ns_rotate_heads_kernel(const RotateArgs a)
{
    extern __shared__ float2 cs[];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, i = row % a.steps;
    const int p = a.pos[a.slots[b]] + i;
    for (int k = threadIdx.x; k < a.rot_dims / 2; k += blockDim.x) {
        float s, c;
        sincosf((float)p * a.freq[k], &s, &c);
        cs[k] = make_float2(c, s);
    }
    __syncthreads();
    const int w = a.dim + a.rot_dim, n = a.heads * w;
    if (VEC) {
        for (int e = threadIdx.x * 4; e < n; e += blockDim.x * 4) {
            const int head = e / w, c = e - head * w, r = c - a.dim;
            float4 v = ns_source_at4(a.src, (int64_t)row * a.src.ld + e);
            if (r < 0) {
                ns_store4(reinterpret_cast<TP*>(a.plain) + (int64_t)row * a.plain_ld + (int64_t)head * a.plain_head + c, v);
                continue;
            }
            if (r < a.rot_dims) {
                const float2 s = cs[r >> 1];
                v = make_float4(fmaf(v.x, s.x, -v.y * s.y), fmaf(v.y, s.x, v.x * s.y), v.z, v.w);
            }
            if (r + 2 < a.rot_dims) {
                const float2 t = cs[(r >> 1) + 1];
                v = make_float4(v.x, v.y, fmaf(v.z, t.x, -v.w * t.y), fmaf(v.w, t.x, v.z * t.y));
            }
            ns_store4(reinterpret_cast<TR*>(a.rot) + (int64_t)row * a.rot_ld + (int64_t)head * a.rot_head + r, v);
        }
        return;
    }
    for (int e = threadIdx.x; e < n; e += blockDim.x) {
        const int head = e / w, c = e - head * w;
        const int64_t at = (int64_t)row * a.src.ld + e;
        const float x = ns_source_at(a.src, at);
        if (c < a.dim) {
            ns_store(reinterpret_cast<TP*>(a.plain) + (int64_t)row * a.plain_ld + (int64_t)head * a.plain_head + c, x);
        } else {
            const int r = c - a.dim;
            float y = x;
            if (r < a.rot_dims) {
                const float2 t = cs[r >> 1];
                const float other = ns_source_at(a.src, (r & 1) ? at - 1 : at + 1);
                y = (r & 1) ? fmaf(x, t.x, other * t.y) : fmaf(x, t.x, -other * t.y);
            }
            ns_store(reinterpret_cast<TR*>(a.rot) + (int64_t)row * a.rot_ld + (int64_t)head * a.rot_head + r, y);
        }
    }
}

// ---------------------------------------------------------------------------------------------
// y[r, head, n] = sum_k x[r, head, k] w[head, k, n], 32-bit sums, 64 x 64 tiles
// ---------------------------------------------------------------------------------------------
struct HeadMatmulArgs {
    const void* x; int64_t x_ld; int x_head;
    const void* w; int64_t w_head, w_k, w_n;     // strides in elements
    void* y; int64_t y_ld; int y_head;
    int rows, k, n;
};

template <typename TX, typename TW, typename TY>
__global__ void __launch_bounds__(256) ns_head_matmul_kernel(const HeadMatmulArgs a)
{
    __shared__ float xs[16][68], ws[16][68];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int head = blockIdx.z, r0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tid = threadIdx.x;
    const TX* x = reinterpret_cast<const TX*>(a.x) + (int64_t)head * a.x_head;
    const TW* w = reinterpret_cast<const TW*>(a.w) + (int64_t)head * a.w_head;
    const int tr = (tid >> 4) * 4, tn = (tid & 15) * 4;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.0f;
    for (int k0 = 0; k0 < a.k; k0 += 16) {
        for (int e = tid; e < 1024; e += 256) {
            const int kk = e & 15, r = e >> 4;
            xs[kk][r] = (k0 + kk < a.k && r0 + r < a.rows) ? ns_load(x + (int64_t)(r0 + r) * a.x_ld + k0 + kk) : 0.0f;
        }
        for (int e = tid; e < 1024; e += 256) {
            // neighbouring threads walk the contiguous direction of w
            const int kk = a.w_n == 1 ? e >> 6 : e & 15, n = a.w_n == 1 ? e & 63 : e >> 4;
            ws[kk][n] = (k0 + kk < a.k && n0 + n < a.n) ? ns_load(w + (int64_t)(k0 + kk) * a.w_k + (int64_t)(n0 + n) * a.w_n) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 16; kk++) {
            float xv[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { xv[i] = xs[kk][tr + i]; wv[i] = ws[kk][tn + i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
    TY* y = reinterpret_cast<TY*>(a.y) + (int64_t)head * a.y_head;
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++)
            if (r0 + tr + i < a.rows && n0 + tn + j < a.n) ns_store(y + (int64_t)(r0 + tr + i) * a.y_ld + n0 + tn + j, acc[i][j]);
}

// ---------------------------------------------------------------------------------------------
// attention of carried-through queries over the ring, 32-bit throughout: a warp per head, tiles of 32 cached rows in shared
// memory, scores of a tile in the lanes
// ---------------------------------------------------------------------------------------------
struct LatentAttendArgs {
    const float* q;            // [rows, heads, width]: [carried-through | rotated]
    const void* ring;
    int64_t ring_slot_stride;
    int ring_len, ring_ld;
    int rank, width;           // width = rank + rotated size
    int window;                // 0: every earlier position
    float scale;
    const int32_t* slots;
    const int32_t* pos;
    int steps, heads;
    float* o;                  // [rows, heads, rank]
};

template <typename T, int NR>
__global__ void __launch_bounds__(256) ns_latent_attend_kernel(const LatentAttendArgs a)
{
    extern __shared__ float4 lat_smem[];
    float* tile = reinterpret_cast<float*>(lat_smem);          // [32][wld]
    const int wld = (a.width | 1);                             // odd: lanes that walk rows hit different banks
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / a.steps, i = row % a.steps;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y * 8 + warp;
    const int slot = a.slots[b], p = a.pos[slot] + i;
    const int first = a.window > 0 ? max(0, p - a.window + 1) : 0;
    const T* ring = reinterpret_cast<const T*>(a.ring) + (int64_t)slot * a.ring_slot_stride;
    float* qs = tile + 32 * wld + warp * a.width;
    if (head < a.heads)
        for (int c = lane; c < a.width; c += 32) qs[c] = a.q[((int64_t)row * a.heads + head) * a.width + c];
    float acc[NR], m = -INFINITY, l = 0.0f;
#pragma unroll
    for (int j = 0; j < NR; j++) acc[j] = 0.0f;
    for (int j0 = first; j0 <= p; j0 += 32) {
        const int count = min(32, p - j0 + 1);
        __syncthreads();
        for (int r = warp; r < count; r += 8) {
            const T* src = ring + (int64_t)((j0 + r) % a.ring_len) * a.ring_ld;
            for (int c = lane; c < a.width; c += 32) tile[r * wld + c] = ns_load(src + c);
        }
        __syncthreads();
        if (head < a.heads) {
            float s = -INFINITY;
            if (lane < count) {
                float d = 0.0f;
                for (int c = 0; c < a.width; c++) d = fmaf(qs[c], tile[lane * wld + c], d);
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
#pragma unroll
                for (int j = 0; j < NR; j++) {
                    const int c = j * 32 + lane;
                    if (c < a.rank) acc[j] = fmaf(wr, tile[r * wld + c], acc[j]);
                }
            }
        }
    }
    if (head < a.heads) {
        float* o = a.o + ((int64_t)row * a.heads + head) * a.rank;
        const float inv = 1.0f / l;
#pragma unroll
        for (int j = 0; j < NR; j++) {
            const int c = j * 32 + lane;
            if (c < a.rank) o[c] = acc[j] * inv;
        }
    }
}

template <typename T, int NR>
int launch_attend(NsDevice* d, const LatentAttendArgs& a, int rows)
{
    const size_t smem = (size_t)(32 * (a.width | 1) + 8 * a.width) * 4;
    NS_REQUIRE(smem <= 220 * 1024, NS_ERR_ARGUMENT, "ns_latent_attend: cached rows of %d values do not fit shared memory", a.width);
    auto k = ns_latent_attend_kernel<T, NR>;
    if (smem > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    NS_CUDA(ns_launch_plain(k, dim3((unsigned)rows, (unsigned)((a.heads + 7) / 8)), dim3(256), smem, d->stream, a));
    return NS_OK;
}

template <typename T>
int dispatch_attend(NsDevice* d, const LatentAttendArgs& a, int rows)
{
    if (a.rank <= 128) return launch_attend<T, 4>(d, a, rows);
    if (a.rank <= 256) return launch_attend<T, 8>(d, a, rows);
    if (a.rank <= 512) return launch_attend<T, 16>(d, a, rows);
    return launch_attend<T, 32>(d, a, rows);
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }
#define I32P(x) reinterpret_cast<const int32_t*>(x)
#define CF32P(x) reinterpret_cast<const float*>(x)

static bool float_or_bf16(int dtype) { return dtype == NS_F32 || dtype == NS_BF16; }

extern "C" int ns_latent_append(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int q_rank, int kv_rank, int rot_dim, int rot_dims,
                                uint64_t q_norm, uint64_t kv_norm, float eps, uint64_t freq, uint64_t slots, uint64_t pos, int batch, int steps, int dtype,
                                uint64_t cq, int cq_ld, uint64_t ring, int64_t ring_slot_stride, int ring_len, int ring_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype) && src_ld >= q_rank + kv_rank + rot_dim, NS_ERR_ARGUMENT, "ns_latent_append: bad source");
    NS_REQUIRE(q_rank > 0 && kv_rank > 0 && rot_dim >= 0 && rot_dims >= 0 && rot_dims <= rot_dim && (rot_dims & 1) == 0 && (rot_dims == 0 || freq),
               NS_ERR_ARGUMENT, "ns_latent_append: bad sizes");
    NS_REQUIRE(q_norm && kv_norm && slots && pos && cq && ring && batch > 0 && float_or_bf16(dtype), NS_ERR_ARGUMENT, "ns_latent_append: bad argument");
    NS_REQUIRE(steps > 0 && steps <= ring_len && cq_ld >= q_rank && ring_ld >= kv_rank + rot_dim, NS_ERR_ARGUMENT,
               "ns_latent_append: %d tokens do not fit a ring of %d rows", steps, ring_len);
    LatentAppendArgs a;
    a.src = ns_source(src, splits, src_dtype, (int64_t)batch * steps, src_ld);
    a.q_rank = q_rank; a.kv_rank = kv_rank; a.rot_dim = rot_dim; a.rot_dims = rot_dims;
    a.q_norm = CF32P(q_norm); a.kv_norm = CF32P(kv_norm); a.eps = eps; a.freq = CF32P(freq);
    a.slots = I32P(slots); a.pos = I32P(pos); a.steps = steps;
    a.cq = reinterpret_cast<void*>(cq); a.cq_ld = cq_ld;
    a.ring = reinterpret_cast<void*>(ring); a.ring_slot_stride = ring_slot_stride; a.ring_len = ring_len; a.ring_ld = ring_ld;
    const int n = q_rank + kv_rank + rot_dim;
    NS_REQUIRE(n <= 12000, NS_ERR_ARGUMENT, "ns_latent_append: rows of %d values do not fit shared memory", n);
    const bool vec = ((q_rank | kv_rank | rot_dim | src_ld | cq_ld | ring_ld) & 3) == 0 && (ring_slot_stride & 3) == 0 && ((src | q_norm | kv_norm | cq | ring) & 15) == 0;
    auto k = dtype == NS_F32 ? (vec ? ns_latent_append_kernel<float, true> : ns_latent_append_kernel<float, false>)
                             : (vec ? ns_latent_append_kernel<uint16_t, true> : ns_latent_append_kernel<uint16_t, false>);
    NS_CUDA(ns_launch_plain(k, dim3((unsigned)(batch * steps)), dim3(256), (size_t)((n + 3) & ~3) * 4, d->stream, a));
    return NS_OK;
}

extern "C" int ns_rotate_heads(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int heads, int dim, int rot_dim, int rot_dims, uint64_t freq,
                               uint64_t slots, uint64_t pos, int batch, int steps, int plain_dtype, uint64_t plain, int64_t plain_ld, int plain_head,
                               int rot_dtype, uint64_t rot, int64_t rot_ld, int rot_head)
{
    NS_ENTER(h);
    NS_REQUIRE(heads > 0 && dim >= 0 && rot_dim >= 0 && rot_dims >= 0 && rot_dims <= rot_dim && (rot_dims & 1) == 0 && (rot_dims == 0 || freq), NS_ERR_ARGUMENT,
               "ns_rotate_heads: bad sizes");
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype) && src_ld >= heads * (dim + rot_dim), NS_ERR_ARGUMENT, "ns_rotate_heads: bad source");
    NS_REQUIRE(slots && pos && plain && rot && batch > 0 && steps > 0 && float_or_bf16(plain_dtype) && float_or_bf16(rot_dtype), NS_ERR_ARGUMENT,
               "ns_rotate_heads: bad argument");
    RotateArgs a;
    a.src = ns_source(src, splits, src_dtype, (int64_t)batch * steps, src_ld);
    a.heads = heads; a.dim = dim; a.rot_dim = rot_dim; a.rot_dims = rot_dims; a.freq = CF32P(freq);
    a.slots = I32P(slots); a.pos = I32P(pos); a.steps = steps;
    a.plain = reinterpret_cast<void*>(plain); a.plain_ld = plain_ld; a.plain_head = plain_head;
    a.rot = reinterpret_cast<void*>(rot); a.rot_ld = rot_ld; a.rot_head = rot_head;
    const bool vec = ((dim | rot_dim | src_ld | plain_head | rot_head) & 3) == 0 && ((plain_ld | rot_ld) & 3) == 0 &&
                     (src & 15) == 0 && (plain & (plain_dtype == NS_F32 ? 15 : 7)) == 0 && (rot & (rot_dtype == NS_F32 ? 15 : 7)) == 0;
    auto go = [&](auto kern) -> int {
        NS_CUDA(ns_launch_plain(kern, dim3((unsigned)(batch * steps)), dim3(256), (size_t)(rot_dims / 2 + 1) * sizeof(float2), d->stream, a));
        return NS_OK;
    };
    if (plain_dtype == NS_F32 && rot_dtype == NS_F32) return vec ? go(ns_rotate_heads_kernel<float, float, true>) : go(ns_rotate_heads_kernel<float, float, false>);
    if (plain_dtype == NS_BF16 && rot_dtype == NS_BF16)
        return vec ? go(ns_rotate_heads_kernel<uint16_t, uint16_t, true>) : go(ns_rotate_heads_kernel<uint16_t, uint16_t, false>);
    return ns_fail(NS_ERR_ARGUMENT, "ns_rotate_heads: both outputs have one type");
}

extern "C" int ns_head_matmul(ns_device_t h, int x_dtype, uint64_t x, int64_t x_ld, int x_head, int w_dtype, uint64_t w, int64_t w_head, int64_t w_k, int64_t w_n,
                              int y_dtype, uint64_t y, int64_t y_ld, int y_head, int rows, int heads, int k, int n)
{
    NS_ENTER(h);
    NS_REQUIRE(x && w && y && rows > 0 && heads > 0 && k > 0 && n > 0, NS_ERR_ARGUMENT, "ns_head_matmul: bad argument");
    NS_REQUIRE(float_or_bf16(x_dtype) && float_or_bf16(w_dtype) && float_or_bf16(y_dtype), NS_ERR_ARGUMENT, "ns_head_matmul: bad types");
    NS_REQUIRE(heads <= 65535 && (rows + 63) / 64 <= 65535, NS_ERR_ARGUMENT, "ns_head_matmul: too many rows or heads");
    if (x_dtype == NS_BF16 && w_dtype == NS_BF16 && (w_k == 1 || w_n == 1))
        return ns_head_matmul_tc(d, x, x_ld, x_head, w, w_head, w_k, w_n, y_dtype, y, y_ld, y_head, rows, heads, k, n);
    HeadMatmulArgs a;
    a.x = reinterpret_cast<const void*>(x); a.x_ld = x_ld; a.x_head = x_head;
    a.w = reinterpret_cast<const void*>(w); a.w_head = w_head; a.w_k = w_k; a.w_n = w_n;
    a.y = reinterpret_cast<void*>(y); a.y_ld = y_ld; a.y_head = y_head;
    a.rows = rows; a.k = k; a.n = n;
    const dim3 grid((n + 63) / 64, (rows + 63) / 64, heads);
    auto go = [&](auto kern) -> int {
        NS_CUDA(ns_launch_plain(kern, grid, dim3(256), 0, d->stream, a));
        return NS_OK;
    };
    if (x_dtype == NS_F32 && w_dtype == NS_F32 && y_dtype == NS_F32) return go(ns_head_matmul_kernel<float, float, float>);
    if (x_dtype == NS_F32 && w_dtype == NS_BF16 && y_dtype == NS_BF16) return go(ns_head_matmul_kernel<float, uint16_t, uint16_t>);
    if (x_dtype == NS_F32 && w_dtype == NS_BF16 && y_dtype == NS_F32) return go(ns_head_matmul_kernel<float, uint16_t, float>);
    return ns_fail(NS_ERR_ARGUMENT, "ns_head_matmul: this combination of types is not built");
}

extern "C" int ns_latent_attend(ns_device_t h, uint64_t q, int dtype, uint64_t ring, int64_t ring_slot_stride, int ring_len, int ring_ld, int rank, int width,
                                int window, float scale, uint64_t slots, uint64_t pos, int batch, int steps, int heads, uint64_t o)
{
    NS_ENTER(h);
    NS_REQUIRE(q && ring && slots && pos && o && batch > 0 && steps > 0 && heads > 0 && float_or_bf16(dtype), NS_ERR_ARGUMENT, "ns_latent_attend: bad argument");
    NS_REQUIRE(rank > 0 && rank <= 1024 && width >= rank && ring_ld >= width && window >= 0, NS_ERR_ARGUMENT, "ns_latent_attend: bad sizes");
    NS_REQUIRE(window == 0 || window - 1 + steps <= ring_len, NS_ERR_ARGUMENT, "ns_latent_attend: a window of %d and %d tokens need more than %d ring rows",
               window, steps, ring_len);
    LatentAttendArgs a;
    a.q = CF32P(q);
    a.ring = reinterpret_cast<const void*>(ring); a.ring_slot_stride = ring_slot_stride; a.ring_len = ring_len; a.ring_ld = ring_ld;
    a.rank = rank; a.width = width; a.window = window; a.scale = scale;
    a.slots = I32P(slots); a.pos = I32P(pos); a.steps = steps; a.heads = heads;
    a.o = reinterpret_cast<float*>(o);
    return dtype == NS_F32 ? dispatch_attend<float>(d, a, batch * steps) : dispatch_attend<uint16_t>(d, a, batch * steps);
}
