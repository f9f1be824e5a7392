// The experts' products on the 5th-generation tensor cores (tcgen05 + TMEM), operands staged by TMA: for the rows of the line that
// belong to one expert,
//     act = silu(gate_e x) * up_e x    and then    out = down_e act.
//
// The WEIGHTS are the A operand (128 TMEM lanes = output features), the rows the B operand (MMA N = rows of a tile, 32 to 256), so the
// same kernel streams weights past a few rows per expert (decode: HBM-bound) and runs full tiles (prompts: tensor-bound). A CTA owns
// TWO feature tiles of one row tile -- gate and up features of the same index, whose accumulators lie in the same TMEM lanes, or two
// neighbouring tiles of `down` -- so a stage of 64 K-elements moves 32 KiB of weights and the rows' 128 bytes each once:
//   warp 0       TMA into the ring; weights need only the routing, so the first stages' weights go out before the wait for
//                the previous kernel (which wrote the rows);
//   warp 1       issues eight MMAs per stage (the whole warp walks, an elected lane issues);
//   all 8 warps  epilogue from TMEM: thread = feature, columns = rows; warps 4 - 7 take the upper half of the columns.
// Row tiles are found from the experts' row counts on the device: the grid covers the most tiles the routing can make, CTAs past the
// last one leave at once, and nothing about the routing is known to the host (a decode step replays as a graph).
//
// Every mbarrier wait is bounded; a wait that runs out sets the error word and the CTA skips its stores.
#include "experts.cuh"
#include "launch_utils.cuh"
#include "matrix_map.cuh"
#include "tcgen05_utils.cuh"

#include <mutex>

namespace llaisys::kernels {

namespace {

constexpr int kFeatures = 128, kDepth = 64, kThreads = 256;
constexpr int kTileBytes = kFeatures * 128;      // one weight tile of a stage
constexpr int kRingBudget = 216 * 1024, kMaxStages = 6, kNumBars = 2 * kMaxStages + 1;

struct Params {
    const int32_t *counts;
    void *out;
    int32_t experts, n, k;    // n: features of an expert's output rows
    int32_t w_rows, second;   // rows per expert of the weights; from a CTA's first feature tile to its second
    int32_t step;             // features between neighbouring CTAs
    int32_t rows, stages;     // rows of a tile (MMA N)
    int32_t *error_flag;
};

template <bool kBf16>
__device__ __forceinline__ uint16_t pack1(float v) {
    if constexpr (kBf16) {
        return __bfloat16_as_ushort(__float2bfloat16_rn(v));
    } else {
        return __half_as_ushort(__float2half_rn(v));
    }
}

template <bool kBf16, bool kGlu>
__global__ void __launch_bounds__(kThreads, 1)
    experts_tc_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, Params p) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    int expert = 0, first = 0, rows = 0;
    find_tile(p.counts, p.experts, p.rows, int(blockIdx.y), expert, first, rows);
    if (rows == 0) { // uniform over the CTA
        grid_dependency_wait();
        grid_launch_dependents();
        return;
    }
    const uint32_t raw = smem_u32(smem_raw), base = (raw + 1023u) & ~1023u;
    const int stage_bytes = 2 * kTileBytes + p.rows * 128;
    uint64_t *bars = reinterpret_cast<uint64_t *>(smem_raw + (base - raw) + p.stages * stage_bytes);
    const uint32_t bars_u32 = smem_u32(bars);
    uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + kNumBars);
    volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
    auto full = [&](int st) { return bars_u32 + uint32_t(st) * 8; };
    auto empty = [&](int st) { return bars_u32 + uint32_t(kMaxStages + st) * 8; };
    const uint32_t accum = bars_u32 + uint32_t(2 * kMaxStages) * 8;
    uint32_t cols = 32;
    while (cols < uint32_t(2 * p.rows)) {
        cols *= 2;
    }
    if (tid == 0) {
        for (int i = 0; i < kNumBars; ++i) {
            mbar_init(bars_u32 + uint32_t(i) * 8, 1);
        }
        *s_abort = 0;
        mbar_init_fence();
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(s_tmem), cols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *s_tmem;
    const int chunks = (p.k + kDepth - 1) / kDepth;
    const int feature = int(blockIdx.x) * p.step, w_row = expert * p.w_rows + feature;
    auto give_up = [&]() {
        *s_abort = 1;
        atomicOr(p.error_flag, kErrGemmTimeout);
    };
    if (warp == 0) {
        auto weights = [&](int st, int c) {
            const uint32_t dst = base + uint32_t(st * stage_bytes);
            mbar_arrive_expect_tx(full(st), uint32_t(stage_bytes));
            tma_load_2d(dst, &tmap_w, c * kDepth, w_row, full(st));
            tma_load_2d(dst + kTileBytes, &tmap_w, c * kDepth, w_row + p.second, full(st));
        };
        auto inputs = [&](int st, int c) { tma_load_2d(base + uint32_t(st * stage_bytes + 2 * kTileBytes), &tmap_x, c * kDepth, first, full(st)); };
        const int head = chunks < p.stages ? chunks : p.stages;
        if (elect_one()) {
            for (int c = 0; c < head; ++c) {
                weights(c, c);
            }
        }
        __syncwarp();
        grid_dependency_wait();
        grid_launch_dependents();
        if (elect_one()) {
            for (int c = 0; c < head; ++c) {
                inputs(c, c);
            }
        }
        __syncwarp();
        int st = 0;
        uint32_t parity = 0;
        for (int c = head; c < chunks; ++c) {
            if (!__all_sync(0xffffffffu, wait_or_abort(empty(st), parity, s_abort))) {
                if (lane == 0) {
                    give_up();
                }
                break;
            }
            if (elect_one()) {
                weights(st, c);
                inputs(st, c);
            }
            __syncwarp();
            if (++st == p.stages) {
                st = 0;
                parity ^= 1;
            }
        }
    } else if (warp == 1) {
        grid_dependency_wait();
        grid_launch_dependents();
        const uint32_t idesc = make_idesc(kBf16, false, kFeatures, p.rows);
        int st = 0;
        uint32_t parity = 0;
        bool ok = true;
        for (int c = 0; c < chunks; ++c) {
            if (!__all_sync(0xffffffffu, wait_or_abort(full(st), parity, s_abort))) {
                ok = false;
                break;
            }
            tc_fence_after();
            const uint32_t at = base + uint32_t(st * stage_bytes);
            if (elect_one()) {
#pragma unroll
                for (int ks = 0; ks < kDepth / 16; ++ks) {
                    const uint64_t x = smem_desc_sw128(at + 2 * kTileBytes + ks * 32, 0, 1024);
                    umma_f16(tmem, smem_desc_sw128(at + ks * 32, 0, 1024), x, idesc, c > 0 || ks > 0 ? 1u : 0u);
                    umma_f16(tmem + uint32_t(p.rows), smem_desc_sw128(at + kTileBytes + ks * 32, 0, 1024), x, idesc, c > 0 || ks > 0 ? 1u : 0u);
                }
                umma_commit(empty(st));
                if (c == chunks - 1) {
                    umma_commit(accum);
                }
            }
            __syncwarp();
            if (++st == p.stages) {
                st = 0;
                parity ^= 1;
            }
        }
        if (!ok && lane == 0) {
            give_up();
        }
    } else {
        grid_dependency_wait();
        grid_launch_dependents();
    }
    __syncwarp();
    const bool done = __all_sync(0xffffffffu, wait_or_abort(accum, 0u, s_abort)); // (uniform: the loads below are warp-wide)
    if (!done && tid == 0) {
        give_up();
    }
    __syncwarp();
    tc_fence_after();
    // ---- epilogue ----
    const int f = feature + (warp & 3) * 32 + lane;
    const uint32_t taddr = tmem + (uint32_t((warp & 3) * 32) << 16);
    const int half = p.rows / 2, c0 = (warp >> 2) * half;
    uint16_t *out = static_cast<uint16_t *>(p.out) + int64_t(first) * p.n;
    for (int c = c0; c < c0 + half && c < rows && done; c += 16) {
        float g[16], u[16];
        tmem_ld16(taddr + uint32_t(c), g);
        tmem_ld16(taddr + uint32_t(p.rows + c), u);
        tmem_wait_ld();
        uint16_t *dst = out + int64_t(c) * p.n + f;
        if constexpr (kGlu) {
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                const float v = __fdividef(g[j], 1.f + __expf(-g[j])) * u[j];
                if (c + j < rows && f < p.n) {
                    dst[int64_t(j) * p.n] = pack1<kBf16>(v);
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                if (c + j < rows && f < p.n) {
                    dst[int64_t(j) * p.n] = pack1<kBf16>(g[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                if (c + j < rows && f + p.second < p.n) {
                    dst[int64_t(j) * p.n + p.second] = pack1<kBf16>(u[j]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tmem_dealloc(tmem, cols);
    }
}

template <bool kBf16, bool kGlu>
void launch(cudaStream_t s, const CUtensorMap &w, const CUtensorMap &x, const Params &p, dim3 grid) {
    static std::once_flag once[64];
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    std::call_once(once[dev & 63], [] {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(experts_tc_kernel<kBf16, kGlu>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                int(1024 + kRingBudget + kNumBars * 8 + 16)));
    });
    const size_t smem = 1024 + size_t(p.stages) * (2 * kTileBytes + p.rows * 128) + kNumBars * 8 + 16;
    launch_programmatic_smem(experts_tc_kernel<kBf16, kGlu>, grid, kThreads, smem, s, w, x, p);
}

} // namespace

bool experts_tc_covers(llaisysDataType_t dtype, const ExpertArgs &a) {
    return (dtype == LLAISYS_DTYPE_BF16 || dtype == LLAISYS_DTYPE_F16) && a.width % 8 == 0 && a.ff % 8 == 0 && a.rows != nullptr &&
           aligned16(a.rows) && aligned16(a.act) && aligned16(a.out) && aligned16(a.gate_up) && aligned16(a.down) &&
           expert_tiles_bound(a, 256) <= 65535 && int64_t(a.experts) * 2 * a.ff < (int64_t(1) << 31) &&
           int64_t(a.experts) * a.width < (int64_t(1) << 31);
}

void experts_tc(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &a) {
    const bool bf16 = dtype == LLAISYS_DTYPE_BF16;
    const int64_t total = int64_t(a.n_rows) * a.top;
    // tiles about as long as an expert's share of the rows
    const int64_t share = total / (a.experts + a.identity);
    int rows = 32;
    while (rows < 256 && (rows < share || expert_tiles_bound(a, rows) > 65535)) {
        rows *= 2;
    }
    Params p;
    p.counts = a.counts;
    p.experts = a.experts;
    p.rows = rows;
    p.stages = kRingBudget / (2 * kTileBytes + rows * 128);
    p.stages = p.stages > kMaxStages ? kMaxStages : p.stages;
    p.error_flag = gemm_error_word();
    CUtensorMap w1, w2, x1, x2;
    ASSERT(matrix_map(&w1, a.gate_up, uint64_t(a.experts) * 2 * a.ff, uint64_t(a.width), kFeatures, bf16) &&
               matrix_map(&w2, a.down, uint64_t(a.experts) * a.width, uint64_t(a.ff), kFeatures, bf16) &&
               matrix_map(&x1, a.rows, uint64_t(total), uint64_t(a.width), uint32_t(rows), bf16) &&
               matrix_map(&x2, a.act, uint64_t(total), uint64_t(a.ff), uint32_t(rows), bf16),
           "experts: no tensor map");
    auto s = static_cast<cudaStream_t>(stream);
    const unsigned tiles = unsigned(expert_tiles_bound(a, rows));
    p.out = a.act;
    p.n = a.ff;
    p.k = a.width;
    p.w_rows = 2 * a.ff;
    p.second = a.ff;
    p.step = kFeatures;
    dim3 grid(unsigned((a.ff + kFeatures - 1) / kFeatures), tiles);
    bf16 ? launch<true, true>(s, w1, x1, p, grid) : launch<false, true>(s, w1, x1, p, grid);
    p.out = a.out;
    p.n = a.width;
    p.k = a.ff;
    p.w_rows = a.width;
    p.second = kFeatures;
    p.step = 2 * kFeatures;
    grid.x = unsigned((a.width + 2 * kFeatures - 1) / (2 * kFeatures));
    bf16 ? launch<true, false>(s, w2, x2, p, grid) : launch<false, false>(s, w2, x2, p, grid);
    check_launch("experts_tc");
}

} // namespace llaisys::kernels
