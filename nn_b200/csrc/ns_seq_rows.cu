// Row operators of decoders that keep the residual stream in 32-bit floats: token + n-gram embedding, residual update with
// RMS normalisation, gated linear unit, and the bookkeeping of a sequence's position.
//
// Each of them takes a product as its float partial sums or as a finished matrix (NsSource), so that the few rows of a decoding
// step need one launch per product: its split-K sum happens in the row kernel that follows, as in ns_step_fused.cu for the
// int8 decoder.  The reference has LayerNorm only (layernorm_fused_f32, Backends/Cuda/PtxKernels.Decoding.cs:61-90) and no
// counterpart of the other operators.
#include "ns_seq.cuh"

namespace {

// ---------------------------------------------------------------------------------------------
// y[b, i, :] = scale * table[token] + bigram[row(previous token, token)]
// ---------------------------------------------------------------------------------------------
NS_DEVINL float4 embed_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
NS_DEVINL float4 embed_load4(const uint16_t* p)
{
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xFFFF0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xFFFF0000u));
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(128) ns_embed_ngram_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, int64_t table_ld, float scale,
                                                             const T* __restrict__ bigram, int64_t bigram_ld, int64_t buckets, int64_t mul_prev,
                                                             int64_t mul_cur, const int32_t* __restrict__ slots, const int32_t* __restrict__ last,
                                                             int steps, int dim, int vocab, float* __restrict__ y)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x, b = row / steps, i = row % steps;
    const int cur = min(max(ids[row], 0), vocab - 1);
    const T* t = table + (int64_t)cur * table_ld;
    const T* g = nullptr;
    if (bigram != nullptr) {
        const int prev = i > 0 ? min(max(ids[row - 1], 0), vocab - 1) : last[slots[b]];
        // the row after the last bucket belongs to a sequence's first token
        int64_t bucket = buckets;
        if (prev >= 0) {
            bucket = ((int64_t)prev * mul_prev + (int64_t)cur * mul_cur) % buckets;
            if (bucket < 0) bucket += buckets;
        }
        g = bigram + bucket * bigram_ld;
    }
    float* out = y + (int64_t)row * dim;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < dim; c += blockDim.x * 4) {
            float4 v = embed_load4(t + c);
            v = make_float4(__fmul_rn(v.x, scale), __fmul_rn(v.y, scale), __fmul_rn(v.z, scale), __fmul_rn(v.w, scale));
            if (g != nullptr) {
                const float4 r = embed_load4(g + c);
                v = make_float4(__fadd_rn(v.x, r.x), __fadd_rn(v.y, r.y), __fadd_rn(v.z, r.z), __fadd_rn(v.w, r.w));
            }
            *reinterpret_cast<float4*>(out + c) = v;
        }
        return;
    }
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
        float v = __fmul_rn(ns_load(t + c), scale);
        if (g != nullptr) v = __fadd_rn(v, ns_load(g + c));
        out[c] = v;
    }
}

// ---------------------------------------------------------------------------------------------
// x_out = x + alpha * source; y = x_out / sqrt(mean(x_out^2) + eps) * w
// ---------------------------------------------------------------------------------------------
struct RmsArgs {
    const float* x;          // [rows, cols], may be null (0)
    NsSource src;            // ptr null: nothing is added
    float alpha;
    float* x_out;            // may be null; may be x
    const float* w;          // null: no normalised output
    float eps;
    const int32_t* row_map;  // output row r reads input row row_map[r]; null: r
    int cols;
    void* y;
    int64_t y_ld;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ns_rms_rows_kernel(const RmsArgs a)
{
    extern __shared__ float4 rms_row4[];
    float* buf = reinterpret_cast<float*>(rms_row4);
    __shared__ float red[8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = a.row_map != nullptr ? a.row_map[blockIdx.x] : (int)blockIdx.x;
    const int64_t base = (int64_t)row * a.cols;
    float ss = 0.0f;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < a.cols; c += blockDim.x * 4) {
            float4 v = a.x != nullptr ? *reinterpret_cast<const float4*>(a.x + base + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (a.src.ptr != nullptr) {
                const float4 s = ns_source_at4(a.src, (int64_t)row * a.src.ld + c);
                v.x = fmaf(a.alpha, s.x, v.x); v.y = fmaf(a.alpha, s.y, v.y); v.z = fmaf(a.alpha, s.z, v.z); v.w = fmaf(a.alpha, s.w, v.w);
            }
            if (a.x_out != nullptr) *reinterpret_cast<float4*>(a.x_out + base + c) = v;
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
            *reinterpret_cast<float4*>(buf + c) = v;
        }
    } else {
        for (int c = threadIdx.x; c < a.cols; c += blockDim.x) {
            float v = a.x != nullptr ? a.x[base + c] : 0.0f;
            if (a.src.ptr != nullptr) v = fmaf(a.alpha, ns_source_at(a.src, (int64_t)row * a.src.ld + c), v);
            if (a.x_out != nullptr) a.x_out[base + c] = v;
            ss = fmaf(v, v, ss);
            buf[c] = v;
        }
    }
    if (a.w == nullptr) return;
    ss = ns_cta_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)a.cols + a.eps);
    T* y = reinterpret_cast<T*>(a.y) + (int64_t)blockIdx.x * a.y_ld;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < a.cols; c += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(buf + c);
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.w + c));
            ns_store4(y + c, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
        }
    } else {
        for (int c = threadIdx.x; c < a.cols; c += blockDim.x) ns_store(y + c, buf[c] * inv * a.w[c]);
    }
    for (int c = a.cols + threadIdx.x; c < a.y_ld; c += blockDim.x) ns_store(y + c, 0.0f);
}

// ---------------------------------------------------------------------------------------------
// x_out = x + source / sqrt(mean(source^2) + eps) * post_w (+ plus);  y = x_out / sqrt(mean(x_out^2) + eps) * w
// ---------------------------------------------------------------------------------------------
struct PostRmsArgs {
    RmsArgs r;               // alpha and row_map are not used
    const float* post_w;
    const float* plus;       // [rows, cols] or null
};

// Q: groups of four columns a thread keeps in registers
template <typename T, int Q>
__global__ void __launch_bounds__(256) ns_rms_post_rows_vec_kernel(const PostRmsArgs p)
{
    const RmsArgs& a = p.r;
    __shared__ float red[2][8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x;
    const int64_t base = (int64_t)row * a.cols;
    float4 s[Q], x[Q];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int c = (threadIdx.x + 256 * i) * 4;
        s[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= a.cols) continue;
        s[i] = ns_source_at4(a.src, (int64_t)row * a.src.ld + c);
        x[i] = *reinterpret_cast<const float4*>(a.x + base + c);
        if (p.plus != nullptr) {
            const float4 t = *reinterpret_cast<const float4*>(p.plus + base + c);
            x[i] = make_float4(x[i].x + t.x, x[i].y + t.y, x[i].z + t.z, x[i].w + t.w);
        }
    }
#pragma unroll
    for (int i = 0; i < Q; i++) { ss = fmaf(s[i].x, s[i].x, ss); ss = fmaf(s[i].y, s[i].y, ss); ss = fmaf(s[i].z, s[i].z, ss); ss = fmaf(s[i].w, s[i].w, ss); }
    const float post = 1.0f / sqrtf(ns_cta_sum(ss, red[0]) / (float)a.cols + a.eps);
    ss = 0.0f;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int c = (threadIdx.x + 256 * i) * 4;
        if (c >= a.cols) continue;
        const float4 w = __ldg(reinterpret_cast<const float4*>(p.post_w + c));
        x[i] = make_float4(fmaf(s[i].x * post, w.x, x[i].x), fmaf(s[i].y * post, w.y, x[i].y), fmaf(s[i].z * post, w.z, x[i].z), fmaf(s[i].w * post, w.w, x[i].w));
        *reinterpret_cast<float4*>(a.x_out + base + c) = x[i];
        ss = fmaf(x[i].x, x[i].x, ss); ss = fmaf(x[i].y, x[i].y, ss); ss = fmaf(x[i].z, x[i].z, ss); ss = fmaf(x[i].w, x[i].w, ss);
    }
    if (a.w == nullptr) return;
    const float inv = 1.0f / sqrtf(ns_cta_sum(ss, red[1]) / (float)a.cols + a.eps);
    T* y = reinterpret_cast<T*>(a.y) + (int64_t)row * a.y_ld;
#pragma unroll
    for (int i = 0; i < Q; i++) {
        const int c = (threadIdx.x + 256 * i) * 4;
        if (c >= a.cols) continue;
        const float4 w = __ldg(reinterpret_cast<const float4*>(a.w + c));
        ns_store4(y + c, make_float4(x[i].x * inv * w.x, x[i].y * inv * w.y, x[i].z * inv * w.z, x[i].w * inv * w.w));
    }
    for (int c = a.cols + threadIdx.x; c < a.y_ld; c += blockDim.x) ns_store(y + c, 0.0f);
}

template <typename T>
__global__ void __launch_bounds__(256) ns_rms_post_rows_kernel(const PostRmsArgs p)
{
    const RmsArgs& a = p.r;
    extern __shared__ float4 rms_row4[];
    float* buf = reinterpret_cast<float*>(rms_row4);
    __shared__ float red[2][8];
    ns_pdl_wait();
    ns_pdl_trigger();
    const int row = blockIdx.x;
    const int64_t base = (int64_t)row * a.cols;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < a.cols; c += blockDim.x) {
        buf[c] = ns_source_at(a.src, (int64_t)row * a.src.ld + c);
        ss = fmaf(buf[c], buf[c], ss);
    }
    const float post = 1.0f / sqrtf(ns_cta_sum(ss, red[0]) / (float)a.cols + a.eps);
    ss = 0.0f;
    for (int c = threadIdx.x; c < a.cols; c += blockDim.x) {
        const float v = fmaf(buf[c] * post, p.post_w[c], a.x[base + c] + (p.plus != nullptr ? p.plus[base + c] : 0.0f));
        a.x_out[base + c] = v;
        ss = fmaf(v, v, ss);
        buf[c] = v;
    }
    if (a.w == nullptr) return;
    const float inv = 1.0f / sqrtf(ns_cta_sum(ss, red[1]) / (float)a.cols + a.eps);
    T* y = reinterpret_cast<T*>(a.y) + (int64_t)row * a.y_ld;
    for (int c = threadIdx.x; c < a.cols; c += blockDim.x) ns_store(y + c, buf[c] * inv * a.w[c]);
    for (int c = a.cols + threadIdx.x; c < a.y_ld; c += blockDim.x) ns_store(y + c, 0.0f);
}

// ---------------------------------------------------------------------------------------------
// y = act(source[:, 0:ff]) * source[:, ff:2ff]
// ---------------------------------------------------------------------------------------------
template <typename T, int ACT>
NS_DEVINL float glu_act(float g)
{
    if (ACT == NS_ACT_RELU) return fmaxf(g, 0.0f);
    return sizeof(T) == 2 ? ns_gelu_fast(g) : ns_gelu_tanh(g);
}

template <typename T, bool VEC, int ACT>
__global__ void __launch_bounds__(256) ns_glu_rows_kernel(const NsSource s, int64_t rows, int ff, T* __restrict__ y, int64_t y_ld)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    if (VEC) {
        const int per_row = (int)(y_ld / 4);
        const int64_t n = rows * per_row;
        for (int64_t q = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; q < n; q += (int64_t)gridDim.x * blockDim.x) {
            const int64_t r = q / per_row;
            const int c = (int)(q - r * per_row) * 4;
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c < ff) {
                const float4 g = ns_source_at4(s, r * s.ld + c), u = ns_source_at4(s, r * s.ld + ff + c);
                o = make_float4(glu_act<T, ACT>(g.x) * u.x, glu_act<T, ACT>(g.y) * u.y, glu_act<T, ACT>(g.z) * u.z, glu_act<T, ACT>(g.w) * u.w);
            }
            ns_store4(y + r * y_ld + c, o);
        }
    } else {
        const int64_t n = rows * y_ld;
        for (int64_t q = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; q < n; q += (int64_t)gridDim.x * blockDim.x) {
            const int64_t r = q / y_ld;
            const int c = (int)(q - r * y_ld);
            float o = 0.0f;
            if (c < ff) o = glu_act<T, ACT>(ns_source_at(s, r * s.ld + c)) * ns_source_at(s, r * s.ld + ff + c);
            ns_store(y + q, o);
        }
    }
}

// y[r, 0:cols] = source[r, col:col+cols], y[r, cols:y_ld] = 0
template <typename T>
__global__ void __launch_bounds__(256) ns_copy_cols_kernel(const NsSource s, int col, int64_t rows, int cols, T* __restrict__ y, int64_t y_ld)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int64_t n = rows * y_ld;
    for (int64_t q = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; q < n; q += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = q / y_ld;
        const int c = (int)(q - r * y_ld);
        ns_store(y + q, c < cols ? ns_source_at(s, r * s.ld + col + c) : 0.0f);
    }
}

// last[slot] = the step's last token, pos[slot] += steps
__global__ void ns_seq_advance_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ slots, int batch, int steps, int32_t* pos, int32_t* last)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b >= batch) return;
    const int slot = slots[b];
    last[slot] = ids[b * steps + steps - 1];
    pos[slot] += steps;
}

__global__ void ns_ids_from_f32_kernel(const float* __restrict__ x, int32_t* __restrict__ ids, int n)
{
    ns_pdl_wait();
    ns_pdl_trigger();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) ids[i] = (int32_t)x[i];
}

unsigned flat_grid(const NsDevice* d, int64_t n)
{
    const int64_t blocks = (n + 255) / 256, most = (int64_t)d->sm_count * 16;
    return (unsigned)(blocks < most ? (blocks > 0 ? blocks : 1) : most);
}

}  // namespace

#define NS_ENTER(h)                          \
    NsDevice* d = ns_dev(h);                 \
    {                                        \
        int _rc = ns_device_make_current(d); \
        if (_rc != NS_OK) return _rc;        \
    }

static bool float_or_bf16(int dtype) { return dtype == NS_F32 || dtype == NS_BF16; }

extern "C" int ns_embed_ngram(ns_device_t h, uint64_t ids, uint64_t table, int table_dtype, int table_ld, float scale, uint64_t bigram, int bigram_ld,
                              int buckets, int64_t mul_prev, int64_t mul_cur, uint64_t slots, uint64_t last, int batch, int steps, int dim, int vocab, uint64_t y)
{
    NS_ENTER(h);
    NS_REQUIRE(ids && table && y && batch > 0 && steps > 0 && dim > 0 && vocab > 0, NS_ERR_ARGUMENT, "ns_embed_ngram: bad argument");
    NS_REQUIRE(float_or_bf16(table_dtype) && table_ld >= dim, NS_ERR_ARGUMENT, "ns_embed_ngram: bad table");
    NS_REQUIRE(bigram == 0 || (buckets > 0 && slots && last && bigram_ld >= dim), NS_ERR_ARGUMENT, "ns_embed_ngram: bad bigram table");
    const unsigned rows = (unsigned)batch * (unsigned)steps;
    const bool vec = ((dim | table_ld | (bigram ? bigram_ld : 0)) & 3) == 0 && ((table | bigram | y) & 15) == 0;
    auto launch = [&](auto kernel, auto zero) -> int {
        using T = decltype(zero);
        NS_CUDA(ns_launch_plain(kernel, dim3(rows), dim3(128), 0, d->stream, reinterpret_cast<const int32_t*>(ids), reinterpret_cast<const T*>(table),
                                (int64_t)table_ld, scale, reinterpret_cast<const T*>(bigram), (int64_t)bigram_ld, (int64_t)buckets, mul_prev, mul_cur,
                                reinterpret_cast<const int32_t*>(slots), reinterpret_cast<const int32_t*>(last), steps, dim, vocab, reinterpret_cast<float*>(y)));
        return NS_OK;
    };
    if (table_dtype == NS_F32) return vec ? launch(ns_embed_ngram_kernel<float, true>, float(0)) : launch(ns_embed_ngram_kernel<float, false>, float(0));
    return vec ? launch(ns_embed_ngram_kernel<uint16_t, true>, uint16_t(0)) : launch(ns_embed_ngram_kernel<uint16_t, false>, uint16_t(0));
}

extern "C" int ns_rms_rows(ns_device_t h, uint64_t x, uint64_t src, int splits, int src_dtype, int src_ld, float alpha, uint64_t x_out, uint64_t w, float eps,
                           uint64_t row_map, int64_t src_rows, int64_t rows, int cols, int out_dtype, uint64_t y, int y_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(rows > 0 && cols > 0 && (x || src), NS_ERR_ARGUMENT, "ns_rms_rows: bad argument");
    NS_REQUIRE(src == 0 || (ns_source_ok(src, splits, src_dtype) && src_ld >= cols), NS_ERR_ARGUMENT, "ns_rms_rows: bad source");
    NS_REQUIRE(w == 0 || (y && float_or_bf16(out_dtype) && y_ld >= cols), NS_ERR_ARGUMENT, "ns_rms_rows: bad output");
    NS_REQUIRE(w != 0 || x_out != 0, NS_ERR_ARGUMENT, "ns_rms_rows: nothing to write");
    NS_REQUIRE((size_t)cols * 4 <= 160 * 1024, NS_ERR_ARGUMENT, "ns_rms_rows: %d columns do not fit shared memory", cols);
    RmsArgs a;
    a.x = reinterpret_cast<const float*>(x);
    a.src = src ? ns_source(src, splits, src_dtype, src_rows, src_ld) : NsSource{nullptr, 1, NS_F32, 0, 0};
    a.alpha = alpha;
    a.x_out = reinterpret_cast<float*>(x_out);
    a.w = reinterpret_cast<const float*>(w);
    a.eps = eps;
    a.row_map = reinterpret_cast<const int32_t*>(row_map);
    a.cols = cols;
    a.y = reinterpret_cast<void*>(y);
    a.y_ld = y_ld;
    const bool vec = ((cols | (src ? src_ld : 0) | (w ? y_ld : 0)) & 3) == 0 && ((x | src | x_out | w | y) & 15) == 0 && (a.src.slab & 3) == 0;
    const size_t smem = (size_t)((cols + 3) & ~3) * 4;
    auto launch = [&](auto kernel) -> int {
        if (smem > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        NS_CUDA(ns_launch_plain(kernel, dim3((unsigned)rows), dim3(256), smem, d->stream, a));
        return NS_OK;
    };
    if (w == 0 || out_dtype == NS_F32) return vec ? launch(ns_rms_rows_kernel<float, true>) : launch(ns_rms_rows_kernel<float, false>);
    return vec ? launch(ns_rms_rows_kernel<uint16_t, true>) : launch(ns_rms_rows_kernel<uint16_t, false>);
}

extern "C" int ns_rms_post_rows(ns_device_t h, uint64_t x, uint64_t src, int splits, int src_dtype, int src_ld, uint64_t post_w, uint64_t plus, uint64_t x_out, uint64_t w,
                                float eps, int64_t rows, int cols, int out_dtype, uint64_t y, int y_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(rows > 0 && cols > 0 && x && x_out && post_w, NS_ERR_ARGUMENT, "ns_rms_post_rows: bad argument");
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype) && src_ld >= cols, NS_ERR_ARGUMENT, "ns_rms_post_rows: bad source");
    NS_REQUIRE(w == 0 || (y && float_or_bf16(out_dtype) && y_ld >= cols), NS_ERR_ARGUMENT, "ns_rms_post_rows: bad output");
    NS_REQUIRE((size_t)cols * 4 <= 160 * 1024, NS_ERR_ARGUMENT, "ns_rms_post_rows: %d columns do not fit shared memory", cols);
    PostRmsArgs p;
    RmsArgs& a = p.r;
    a.x = reinterpret_cast<const float*>(x);
    a.src = ns_source(src, splits, src_dtype, rows, src_ld);
    a.alpha = 1.0f;
    a.x_out = reinterpret_cast<float*>(x_out);
    a.w = reinterpret_cast<const float*>(w);
    a.eps = eps;
    a.row_map = nullptr;
    a.cols = cols;
    a.y = reinterpret_cast<void*>(y);
    a.y_ld = y_ld;
    p.post_w = reinterpret_cast<const float*>(post_w);
    p.plus = reinterpret_cast<const float*>(plus);
    const bool vec = ((cols | src_ld | (w ? y_ld : 0)) & 3) == 0 && ((x | src | x_out | w | y | post_w | plus) & 15) == 0 && (a.src.slab & 3) == 0 && cols <= 8192;
    const size_t smem = vec ? 0 : (size_t)((cols + 3) & ~3) * 4;
    auto launch = [&](auto kernel) -> int {
        if (smem > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        NS_CUDA(ns_launch_plain(kernel, dim3((unsigned)rows), dim3(256), smem, d->stream, p));
        return NS_OK;
    };
    auto pick = [&](auto zero) -> int {
        using T = decltype(zero);
        if (!vec) return launch(ns_rms_post_rows_kernel<T>);
        if (cols <= 1024) return launch(ns_rms_post_rows_vec_kernel<T, 1>);
        if (cols <= 2048) return launch(ns_rms_post_rows_vec_kernel<T, 2>);
        if (cols <= 4096) return launch(ns_rms_post_rows_vec_kernel<T, 4>);
        return launch(ns_rms_post_rows_vec_kernel<T, 8>);
    };
    return w == 0 || out_dtype == NS_F32 ? pick(float(0)) : pick(uint16_t(0));
}

extern "C" int ns_glu_rows(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int64_t rows, int ff, int act, int out_dtype, uint64_t y, int y_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(act == NS_ACT_GELU || act == NS_ACT_RELU, NS_ERR_ARGUMENT, "ns_glu_rows: unknown activation %d", act);
    NS_REQUIRE(rows > 0 && ff > 0 && y && y_ld >= ff && float_or_bf16(out_dtype), NS_ERR_ARGUMENT, "ns_glu_rows: bad argument");
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype) && src_ld >= 2 * ff, NS_ERR_ARGUMENT, "ns_glu_rows: bad source");
    const NsSource s = ns_source(src, splits, src_dtype, rows, src_ld);
    const bool vec = ((ff | src_ld | y_ld) & 3) == 0 && ((src | y) & 15) == 0;
    const unsigned grid = flat_grid(d, vec ? rows * (y_ld / 4) : rows * y_ld);
    auto launch = [&](auto zero, auto kernel) -> int {
        using T = decltype(zero);
        NS_CUDA(ns_launch_plain(kernel, dim3(grid), dim3(256), 0, d->stream, s, rows, ff, reinterpret_cast<T*>(y), (int64_t)y_ld));
        return NS_OK;
    };
    if (out_dtype == NS_F32) {
        if (act == NS_ACT_RELU) return vec ? launch(float(0), ns_glu_rows_kernel<float, true, NS_ACT_RELU>) : launch(float(0), ns_glu_rows_kernel<float, false, NS_ACT_RELU>);
        return vec ? launch(float(0), ns_glu_rows_kernel<float, true, NS_ACT_GELU>) : launch(float(0), ns_glu_rows_kernel<float, false, NS_ACT_GELU>);
    }
    if (act == NS_ACT_RELU) return vec ? launch(uint16_t(0), ns_glu_rows_kernel<uint16_t, true, NS_ACT_RELU>) : launch(uint16_t(0), ns_glu_rows_kernel<uint16_t, false, NS_ACT_RELU>);
    return vec ? launch(uint16_t(0), ns_glu_rows_kernel<uint16_t, true, NS_ACT_GELU>) : launch(uint16_t(0), ns_glu_rows_kernel<uint16_t, false, NS_ACT_GELU>);
}

extern "C" int ns_copy_cols(ns_device_t h, uint64_t src, int splits, int src_dtype, int src_ld, int col, int64_t rows, int cols, int out_dtype, uint64_t y,
                            int y_ld)
{
    NS_ENTER(h);
    NS_REQUIRE(rows > 0 && cols > 0 && col >= 0 && y && y_ld >= cols && float_or_bf16(out_dtype), NS_ERR_ARGUMENT, "ns_copy_cols: bad argument");
    NS_REQUIRE(ns_source_ok(src, splits, src_dtype) && src_ld >= col + cols, NS_ERR_ARGUMENT, "ns_copy_cols: bad source");
    const NsSource s = ns_source(src, splits, src_dtype, rows, src_ld);
    const unsigned grid = flat_grid(d, rows * y_ld);
    if (out_dtype == NS_F32)
        NS_CUDA(ns_launch_plain(ns_copy_cols_kernel<float>, dim3(grid), dim3(256), 0, d->stream, s, col, rows, cols, reinterpret_cast<float*>(y), (int64_t)y_ld));
    else
        NS_CUDA(ns_launch_plain(ns_copy_cols_kernel<uint16_t>, dim3(grid), dim3(256), 0, d->stream, s, col, rows, cols, reinterpret_cast<uint16_t*>(y),
                                (int64_t)y_ld));
    return NS_OK;
}

extern "C" int ns_seq_advance(ns_device_t h, uint64_t ids, uint64_t slots, int batch, int steps, uint64_t pos, uint64_t last)
{
    NS_ENTER(h);
    NS_REQUIRE(ids && slots && pos && last && batch > 0 && steps > 0, NS_ERR_ARGUMENT, "ns_seq_advance: bad argument");
    NS_CUDA(ns_launch_plain(ns_seq_advance_kernel, dim3((batch + 127) / 128), dim3(128), 0, d->stream, reinterpret_cast<const int32_t*>(ids),
                            reinterpret_cast<const int32_t*>(slots), batch, steps, reinterpret_cast<int32_t*>(pos), reinterpret_cast<int32_t*>(last)));
    return NS_OK;
}

extern "C" int ns_ids_from_f32(ns_device_t h, uint64_t x, uint64_t ids, int n)
{
    NS_ENTER(h);
    NS_REQUIRE(x && ids && n > 0, NS_ERR_ARGUMENT, "ns_ids_from_f32: bad argument");
    NS_CUDA(ns_launch_plain(ns_ids_from_f32_kernel, dim3((n + 127) / 128), dim3(128), 0, d->stream, reinterpret_cast<const float*>(x),
                            reinterpret_cast<int32_t*>(ids), n));
    return NS_OK;
}
