// Pieces shared by the kernels of the Mamba-2 state space (see StateSpaceArgs).
#pragma once

#include "args.hpp"
#include "device_utils.cuh"

namespace llaisys::kernels {

// Where the parts of StateSpaceArgs::scratch lie (float offsets, multiples of 4):
//   y     [n_rows][y_stride] model dtype: read-outs with the skip, before gate and norm
//   conv  [n_rows][conv_stride] model dtype: x | B | C after convolution and silu   } runs only
//   dt    [n_rows][heads]: step sizes                                               }
struct StateScratch {
    int64_t y_stride, conv_stride; // elements
    int64_t y, conv, dt, total;
};

LLAISYS_ARGS_FN inline StateScratch state_scratch(llaisysDataType_t dtype, int64_t n_rows, int64_t heads, int64_t groups, int64_t dk, int64_t dv) {
    StateScratch s;
    const int64_t elem = dtype == LLAISYS_DTYPE_F32 ? 4 : 2;
    auto up = [](int64_t n, int64_t m) { return (n + m - 1) / m * m; };
    s.y_stride = up(heads * dv, 8);
    s.conv_stride = up(heads * dv + 2 * groups * dk, 8);
    s.y = 0;
    s.conv = up(n_rows * s.y_stride * elem / 4, 4);
    s.dt = s.conv + up(n_rows * s.conv_stride * elem / 4, 4);
    s.total = s.dt + up(n_rows * heads, 4);
    return s;
}

__device__ __forceinline__ float silu_of(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_of(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// The ring of convolution inputs in a state slot: position p at p mod taps, [channels] each.
__device__ __forceinline__ float *state_ring(const StateSpaceArgs &a, int64_t slot) {
    return a.state + slot * a.slot_stride + int64_t(a.heads) * a.dk * a.dv;
}

// A run's newest convolution inputs go to the ring: the caller's CTA stores the x channels of `head` and, for the first head of a group,
// the group's B and C. Row `last` has position pos_last; the run begins at row `first`.
template <typename T>
__device__ __forceinline__ void keep_run_inputs(const StateSpaceArgs &a, int head, int64_t slot, int first, int last, int pos_last) {
    float *ring = state_ring(a, slot);
    const int share = a.heads / a.groups, group = head / share, n_shared = head % share == 0 ? 2 * a.dk : 0, n = a.dv + n_shared;
    const int rows = min(last - first + 1, a.taps);
    const T *proj = static_cast<const T *>(a.proj);
    for (int u = int(threadIdx.x); u < n * rows; u += int(blockDim.x)) {
        const int back = u / n, j = u - back * n;
        const int ch = j < a.dv ? head * a.dv + j
                                : a.inner() + (j - a.dv < a.dk ? group * a.dk + (j - a.dv) : (a.groups + group) * a.dk + (j - a.dv - a.dk));
        ring[int64_t((pos_last - back) % a.taps) * a.channels() + ch] = to_f32(proj[int64_t(last - back) * a.row_stride + a.x_at + ch]);
    }
}

// Runs of two or more tokens on the tensor cores, from the scratch that the preparing kernel filled.
bool state_space_tiles_fit(llaisysDataType_t dtype, const StateSpaceArgs &a);
void state_space_tiles(stream_t stream, const StateSpaceArgs &a);

} // namespace llaisys::kernels
