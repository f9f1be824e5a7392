// Pieces shared by the kernels of gated linear attention.
#pragma once

#include "args.hpp"
#include "device_utils.cuh"

namespace llaisys::kernels {

template <typename T, int N>
struct alignas(sizeof(T) * N) Pieces {
    T v[N];
};

__device__ __forceinline__ float silu(float g) { return g / (1.f + expf(-g)); }
// log(1 / (1 + exp(-z))) = min(z, 0) - log(1 + x), x = exp(-|z|) in (0, 1]; log(1 + x) = 2 artanh(s) with s = x / (2 + x) <= 1/3
// by the odd power series of artanh up to s^13 (the first term left out is below 1e-8 of the sum).
__device__ __forceinline__ float log_sigmoid_of(float z, float x) {
    const float s = __fdividef(x, 2.f + x), s2 = s * s;
    float p = 1.f / 13.f;
    p = fmaf(p, s2, 1.f / 11.f);
    p = fmaf(p, s2, 1.f / 9.f);
    p = fmaf(p, s2, 1.f / 7.f);
    p = fmaf(p, s2, 1.f / 5.f);
    p = fmaf(p, s2, 1.f / 3.f);
    p = fmaf(p, s2, 1.f);
    return fminf(z, 0.f) - 2.f * s * p;
}
__device__ __forceinline__ float log_sigmoid(float z) { return log_sigmoid_of(z, expf(-fabsf(z))); }

// log a_t of key channel c of `head`: log_sigmoid(W_a2[h dk + c, :] . z + b[h dk + c]) / tau, z [rank] in shared memory
template <typename T>
__device__ __forceinline__ float decay_log(const GatedLinearArgs &a, const float *z, int head, int c) {
    const int64_t ch = int64_t(head) * a.dk + c;
    const T *w = static_cast<const T *>(a.decay_w) + ch * a.rank;
    float acc = to_f32(static_cast<const T *>(a.decay_b)[ch]);
    for (int r = 0; r < a.rank; ++r) {
        acc = fmaf(to_f32(w[r]), z[r], acc);
    }
    return log_sigmoid(acc) / a.tau;
}

// The tensor-core form (gated_linear_chunk.cu): bf16, key size at most 128, sizes and strides in whole 16-byte pieces.
// Sequences with a single row in the batch are left to the decode kernel. With more than 128 value columns a.raw receives
// the outputs before the norm.
bool gated_linear_tiles_apply(llaisysDataType_t dtype, const GatedLinearArgs &a);
void gated_linear_tiles(stream_t stream, const GatedLinearArgs &a);

} // namespace llaisys::kernels
