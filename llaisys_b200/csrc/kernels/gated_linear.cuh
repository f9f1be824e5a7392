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
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

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

} // namespace llaisys::kernels
