// Warp-level pieces of the kernels that run a linear recurrence over tiles of tokens on the tensor cores: f32 operands as the
// sum of two bf16 numbers, swizzled operand rows, fast exponentials.
#pragma once

#include "gated_linear.cuh"
#include "mma_utils.cuh"

namespace llaisys::kernels {

__device__ __forceinline__ uint32_t swz(int row, int chunk, int row_bytes) { // 16-byte chunk `chunk` of row `row`
    return uint32_t(row * row_bytes + ((chunk ^ (row & 7)) << 4));
}
// x0, x1 as two packed pairs of bf16 (x0 in the low half): their upper halves as they are, and the rest rounded
__device__ __forceinline__ void split2(float x0, float x1, uint32_t &hi, uint32_t &lo) {
    const uint32_t u0 = __float_as_uint(x0), u1 = __float_as_uint(x1);
    hi = __byte_perm(u0, u1, 0x7632);
    lo = pack2<true>(x0 - __uint_as_float(u0 & 0xffff0000u), x1 - __uint_as_float(u1 & 0xffff0000u));
}
// 2^x without `volatile` (free to be interleaved); ex2(-inf) = 0
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float silu_fast(float g) { return __fdividef(g, 1.f + ex2(g * -1.4426950408889634f)); }
// log_sigmoid with the exponential as ex2 of a scaled argument
__device__ __forceinline__ float log_sigmoid_fast(float z) { return log_sigmoid_of(z, ex2(fabsf(z) * -1.4426950408889634f)); }
__device__ __forceinline__ float lo_half(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float hi_half(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

// mma.sync without `volatile`: products of different accumulators may be reordered and interleaved with loads
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

} // namespace llaisys::kernels
