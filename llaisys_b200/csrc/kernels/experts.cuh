// Pieces shared by the kernels of the mixture of experts (see ExpertArgs).
#pragma once

#include "args.hpp"
#include "device_utils.cuh"

namespace llaisys::kernels {

// Row tile `tile` of the line: the experts' rows are cut into tiles of `per_tile`, expert after expert. -> expert, first row, rows
// (0: there is no such tile). For whole warps.
__device__ __forceinline__ void find_tile(const int32_t *counts, int experts, int per_tile, int tile, int &expert, int &first, int &rows) {
    const int lane = int(threadIdx.x) & 31;
    int tiles = 0, before = 0;
    rows = 0;
    for (int base = 0; base < experts; base += 32) {
        const int c = base + lane < experts ? counts[base + lane] : 0;
        const int t = (c + per_tile - 1) / per_tile;
        int t_sum = t, c_sum = c; // inclusive scans
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
            const int tv = __shfl_up_sync(0xffffffffu, t_sum, o), cv = __shfl_up_sync(0xffffffffu, c_sum, o);
            t_sum += lane >= o ? tv : 0;
            c_sum += lane >= o ? cv : 0;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, tile < tiles + t_sum);
        if (hit != 0) {
            const int l = __ffs(int(hit)) - 1;
            const int t_before = tiles + __shfl_sync(0xffffffffu, t_sum - t, l), c_before = before + __shfl_sync(0xffffffffu, c_sum - c, l);
            const int here = __shfl_sync(0xffffffffu, c, l), off = (tile - t_before) * per_tile;
            expert = base + l;
            first = c_before + off;
            rows = min(per_tile, here - off);
            return;
        }
        tiles += __shfl_sync(0xffffffffu, t_sum, 31);
        before += __shfl_sync(0xffffffffu, c_sum, 31);
    }
}

// No more row tiles than this, whatever the routing.
inline int64_t expert_tiles_bound(const ExpertArgs &a, int per_tile) {
    const int64_t total = int64_t(a.n_rows) * a.top;
    return total / per_tile + (total < a.experts ? total : int64_t(a.experts));
}

} // namespace llaisys::kernels
