// Shared pieces of the kernels behind decoders with a 32-bit residual stream, recurrent layers and latent attention
// (ns_seq_rows.cu, ns_delta.cu, ns_latent.cu).
//
// A product of such a decoder is read by the row kernel that follows it, from one of two places: float partial sums
// [splits, rows, ld] that ns_linear_forward_partial left behind (the few rows of a decoding step), or one finished matrix
// [rows, ld] of float or bf16.  NsSource describes either.
#pragma once

#include "ns_common.cuh"

struct NsSource {
    const void* ptr;
    int splits;      // number of slabs that add up to the values
    int dtype;       // NS_F32, or NS_BF16 with splits == 1
    int64_t slab;    // elements between slabs
    int ld;          // elements between rows
};

static inline NsSource ns_source(uint64_t ptr, int splits, int dtype, int64_t rows, int ld)
{
    return NsSource{reinterpret_cast<const void*>(ptr), splits, dtype, rows * (int64_t)ld, ld};
}
static inline bool ns_source_ok(uint64_t ptr, int splits, int dtype)
{
    return ptr != 0 && splits >= 1 && (dtype == NS_F32 || (dtype == NS_BF16 && splits == 1));
}

#ifdef __CUDACC__

// the value at element `idx` (row * ld + column); slabs are added in order
NS_DEVINL float ns_source_at(const NsSource& s, int64_t idx)
{
    if (s.dtype == NS_BF16) return ns_bf16_bits_to_f32(reinterpret_cast<const uint16_t*>(s.ptr)[idx]);
    const float* p = reinterpret_cast<const float*>(s.ptr) + idx;
    float v = p[0];
    for (int i = 1; i < s.splits; i++) v = __fadd_rn(v, p[i * s.slab]);
    return v;
}
// four consecutive values; idx and ld are multiples of 4 and ptr is 16-byte aligned
NS_DEVINL float4 ns_source_at4(const NsSource& s, int64_t idx)
{
    if (s.dtype == NS_BF16) {
        const uint2 w = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(s.ptr) + idx);
        return make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xFFFF0000u), __uint_as_float(w.y << 16),
                           __uint_as_float(w.y & 0xFFFF0000u));
    }
    const float* p = reinterpret_cast<const float*>(s.ptr) + idx;
    float4 v = *reinterpret_cast<const float4*>(p);
    for (int i = 1; i < s.splits; i++) {
        const float4 t = *reinterpret_cast<const float4*>(p + i * s.slab);
        v.x = __fadd_rn(v.x, t.x); v.y = __fadd_rn(v.y, t.y); v.z = __fadd_rn(v.z, t.z); v.w = __fadd_rn(v.w, t.w);
    }
    return v;
}

NS_DEVINL void ns_store(float* p, float v) { *p = v; }
NS_DEVINL void ns_store(uint16_t* p, float v) { *p = ns_f32_to_bf16_bits(v); }
NS_DEVINL void ns_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
NS_DEVINL void ns_store4(uint16_t* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(ns_pack_bf16x2(v.x, v.y), ns_pack_bf16x2(v.z, v.w)); }
NS_DEVINL float ns_load(const float* p) { return *p; }
NS_DEVINL float ns_load(const uint16_t* p) { return ns_bf16_bits_to_f32(*p); }

NS_DEVINL float ns_warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// sum over the CTA, the same value in every thread; red holds one float per warp and is free again after the next barrier
NS_DEVINL float ns_cta_sum(float v, float* red)
{
    v = ns_warp_sum(v);
    const int warps = blockDim.x >> 5;
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float r = red[0];
    for (int w = 1; w < warps; w++) r += red[w];
    return r;
}

NS_DEVINL float ns_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
NS_DEVINL float ns_silu(float z) { return z / (1.0f + expf(-z)); }
NS_DEVINL float ns_softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

#endif  // __CUDACC__
