// Warp-level tensor-core pieces for kernels whose tiles are too small or too irregular for tcgen05: ldmatrix, mma.sync
// m16n8k16 (bf16 operands, float accumulators) and 16-byte cp.async.
//
// Fragment layout of m16n8k16, lane = 4 * g + t:  A regs {(g, 2t..), (g + 8, 2t..), (g, 2t + 8..), (g + 8, 2t + 8..)},
// B regs {(k 2t.., n g), (k 2t + 8.., n g)}, C regs {(g, 2t), (g, 2t + 1), (g + 8, 2t), (g + 8, 2t + 1)}.
#pragma once

#include "ns_common.cuh"

#ifdef __CUDACC__

NS_DEVINL void ns_ldsm4(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
NS_DEVINL void ns_ldsm4_t(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
NS_DEVINL void ns_mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
NS_DEVINL void ns_cp_async16(uint32_t dst, const void* src)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
NS_DEVINL void ns_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
NS_DEVINL void ns_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

NS_DEVINL float ns_exp2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Eight bf16 values src[0..8) of which the first `valid` exist (<= 0: none) to shared memory; the rest become zero.
// vec: src is 16-byte aligned whenever valid >= 8.
NS_DEVINL void ns_copy8(uint32_t dst, const uint16_t* src, int valid, bool vec)
{
    if (valid >= 8 && vec) {
        ns_cp_async16(dst, src);
        return;
    }
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t lo = 2 * i < valid ? src[2 * i] : 0, hi = 2 * i + 1 < valid ? src[2 * i + 1] : 0;
        w[i] = lo | (hi << 16);
    }
    ns_st_shared_v4(dst, w[0], w[1], w[2], w[3]);
}

// ldmatrix addresses inside a bf16 tile with `ld` elements per row.
// A operand (16 rows x 16 k) at (row, k): x4 -> the four registers of the fragment.
NS_DEVINL uint32_t ns_addr_a(uint32_t tile, int ld, int row, int k, int lane)
{
    return tile + ((row + (lane & 15)) * ld + k + (lane >> 4) * 8) * 2;
}
// B operand stored [n, k], 16 n x 16 k at (n, k): x4 -> {b0, b1} of n..n+7, {b0, b1} of n+8..n+15.
NS_DEVINL uint32_t ns_addr_b(uint32_t tile, int ld, int n, int k, int lane)
{
    return tile + ((n + (lane & 7) + (lane >> 4) * 8) * ld + k + ((lane >> 3) & 1) * 8) * 2;
}
// B operand stored [k, n] (transposed load), 16 k x 16 n at (k, n): x4.trans -> {b0, b1} of n..n+7, {b0, b1} of n+8..n+15.
NS_DEVINL uint32_t ns_addr_bt(uint32_t tile, int ld, int k, int n, int lane)
{
    return tile + ((k + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + n + (lane >> 4) * 8) * 2;
}
// A operand stored [k, m] (transposed load), 16 m x 16 k at (m, k): x4.trans -> the four registers of the fragment.
NS_DEVINL uint32_t ns_addr_at(uint32_t tile, int ld, int m, int k, int lane)
{
    return tile + ((k + (lane & 7) + (lane >> 4) * 8) * ld + m + ((lane >> 3) & 1) * 8) * 2;
}

#endif  // __CUDACC__
