// Pieces shared by the kernels of the gated delta rule.
#pragma once

#include "gated_linear.cuh"

namespace llaisys::kernels {

// Where the parts of GatedDeltaArgs::scratch lie (float offsets, multiples of 4):
//   conv  [n_rows][conv_stride] model dtype: q | k | v of all heads after convolution and silu
//   unit  [n_rows][2 kv_heads]: factors that make q (q_scale included) and k unit vectors
//   beta, decay_log [n_rows][heads]: the write strength; the log of the decay where it is one per head
//   raw   [n_rows][heads * dv]: read-outs before the norm   } only where another kernel finishes them, or runs go
//   decay [n_rows][heads * dk]: decays per key channel      } token by token
struct DeltaScratch {
    int64_t conv_stride; // elements
    int64_t unit, beta, decay_log, raw, decay, total;
};

// The tensor-core form (gated_delta_chunk.cu) covers these sizes.
LLAISYS_ARGS_FN inline bool gated_delta_tiles_fit(llaisysDataType_t dtype, int64_t dk, int64_t dv) {
    return dtype == LLAISYS_DTYPE_BF16 && dk <= 128 && dk % 8 == 0 && dv % 8 == 0;
}

LLAISYS_ARGS_FN inline DeltaScratch delta_scratch(llaisysDataType_t dtype, int64_t n_rows, int64_t heads, int64_t kv_heads, int64_t dk,
                                                  int64_t dv) {
    DeltaScratch s;
    const bool tiles = gated_delta_tiles_fit(dtype, dk, dv);
    const int64_t elem = dtype == LLAISYS_DTYPE_F32 ? 4 : 2;
    auto up4 = [](int64_t n) { return (n + 3) / 4 * 4; };
    s.conv_stride = (2 * kv_heads * dk + heads * dv + 7) / 8 * 8;
    int64_t at = up4(n_rows * s.conv_stride * elem / 4);
    s.unit = at;
    at += up4(n_rows * 2 * kv_heads);
    s.beta = at;
    at += up4(n_rows * heads);
    s.decay_log = at;
    at += up4(n_rows * heads);
    s.raw = at;
    at += !tiles || dv > 128 ? up4(n_rows * heads * dv) : 0;
    s.decay = at;
    at += tiles ? 0 : up4(n_rows * heads * dk);
    s.total = at;
    return s;
}

__device__ __forceinline__ float sigmoid_of(float x) { return 1.f / (1.f + expf(-x)); }
// -exp(a_log) softplus(x) = exp(a_log) log(sigmoid(-x))
__device__ __forceinline__ float delta_decay_log(float a_log, float x) { return expf(a_log) * log_sigmoid(-x); }

// Channel `c` of head `head`: what softplus is taken of, decay_w z + dt_bias; z [rank] in shared memory
template <typename T>
__device__ __forceinline__ float delta_decay_input(const GatedDeltaArgs &a, const float *z, int head, int c) {
    const int64_t ch = int64_t(head) * a.dk + c;
    const T *w = static_cast<const T *>(a.decay_w) + ch * a.decay_ld;
    float acc = to_f32(static_cast<const T *>(a.dt_bias)[ch]);
    for (int r = 0; r < a.rank; ++r) {
        acc = fmaf(to_f32(w[r]), z[r], acc);
    }
    return acc;
}

// The convolution inputs of a sequence: element of the packed projection row that feeds channel `ch` of q | k | v, and the
// ring of earlier inputs in the state slot.
__device__ __forceinline__ int64_t delta_input_at(const GatedDeltaArgs &a, int ch) {
    const int nq = a.kv_heads * a.dk;
    return ch < nq ? a.q_at + ch : (ch < 2 * nq ? a.k_at + (ch - nq) : a.v_at + (ch - 2 * nq));
}
template <typename T>
__device__ __forceinline__ const T *delta_taps(const GatedDeltaArgs &a, int ch) {
    const int nq = a.kv_heads * a.dk;
    const void *w = ch < nq ? a.conv_q : (ch < 2 * nq ? a.conv_k : a.conv_v);
    return static_cast<const T *>(w) + int64_t(ch < nq ? ch : (ch < 2 * nq ? ch - nq : ch - 2 * nq)) * a.taps;
}
__device__ __forceinline__ float *delta_ring(const GatedDeltaArgs &a, int64_t slot) {
    return a.state + slot * a.slot_stride + int64_t(a.heads) * a.dk * a.dv;
}

// Runs of two or more tokens on the tensor cores, from the scratch that the preparing kernel filled. Read-outs of heads with
// more than 128 value columns go to scratch (raw).
void gated_delta_tiles(stream_t stream, const GatedDeltaArgs &a);

} // namespace llaisys::kernels
