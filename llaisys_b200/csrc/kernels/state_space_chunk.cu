// Mamba-2 over runs of tokens on the tensor cores, 64 tokens (a TILE) at a time.
//
// With b_t the sum of log decays -exp(a_log) dt up to token t of the tile (b_end behind its last one) and S the state in front of it,
//     y_t   = e^(b_t) S^T C_t + sum_{s <= t} e^(b_t - b_s) dt_s (C_t . B_s) x_s + D x_t
//     S_end = e^(b_end) S + sum_s e^(b_end - b_s) dt_s B_s x_s^T
// which is the recurrence exactly. There is one decay per head, so every exponent is formed as a difference and is never positive:
// nothing overflows, whatever the decay.
//
// Precision: the recurrence is f32. The tensor cores take 16-bit operands, so f32 operands (the state, the weighted scores, the
// weighted x) enter as the sum of two bf16 numbers; B, C and x are bf16 already. Accumulators and the state are f32.
//
// A CTA owns up to 128 value columns of one (run, head): warp w holds S^T for 16 of them (rows) and all state rows (columns) in its
// accumulator registers, where it doubles as the B operand of S^T C. Scores of a tile are computed once per CTA, its warps taking a
// block each, and pass through shared memory.
//
// Few (run, head) pairs leave SMs idle, so long runs are cut into SEGMENTS of whole tiles: a first launch computes what every
// segment adds to a zero state, a small scan turns these into the states in front of the segments, and the main launch starts all of
// them at once.
#include "kernels.hpp"
#include "launch_utils.cuh"
#include "linear_tiles.cuh"
#include "state_space.cuh"

#include <algorithm>

namespace llaisys::kernels {

namespace {

constexpr int kTile = 64;
constexpr int kMaxPairs = 2048;      // (segment, head) pairs of a call that is cut
constexpr int kWantedCtas = 148 * 6; // what a call is cut for

struct Cut {
    int segment; // tokens of a segment, whole tiles; larger than any run: not cut
    float *states; // [segment of the call][heads][dk][dv]
    float *decays; // [segment of the call][heads]: log of what is left of a state behind the segment
};

// Segment `index` of the batch, run after run; runs of one token have none. -> run, segment of the run, segments of the run (0: there
// is no such segment). The same for every thread.
__device__ __forceinline__ void find_segment(const StateSpaceArgs &a, int segment, int index, int &run, int &at, int &count) {
    const int lane = int(threadIdx.x) & 31;
    int before = 0;
    count = 0;
    for (int base = 0; base < a.n_seqs; base += 32) {
        const int i = base + lane;
        const int len = i < a.n_seqs ? a.q_starts[i + 1] - a.q_starts[i] : 0;
        const int n = len > 1 ? (len + segment - 1) / segment : 0;
        int sum = n;
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
            const int v = __shfl_up_sync(0xffffffffu, sum, o);
            sum += lane >= o ? v : 0;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, index < before + sum);
        if (hit != 0) {
            const int l = __ffs(int(hit)) - 1;
            run = base + l;
            count = __shfl_sync(0xffffffffu, n, l);
            at = index - before - (__shfl_sync(0xffffffffu, sum, l) - count);
            return;
        }
        before += __shfl_sync(0xffffffffu, sum, 31);
    }
}

__device__ __forceinline__ uint32_t pack_bf16(float x0, float x1) { return pack2<true>(x0, x1); }

// STATES: only what the segment adds to a zero state, into cut.states.
template <int NT, int WARPS, bool STATES>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 4 ? 3 : 1) state_tiles_kernel(StateSpaceArgs a, StateScratch sc, Cut cut) {
    constexpr int kNB = NT * 16 < 128 ? 128 : NT * 16; // bytes of a B or C row
    constexpr int kXB = WARPS * 32 < 128 ? 128 : WARPS * 32;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float s_b[kTile], s_dt[kTile], s_end;
    const uint32_t base = (smem_u32(smem) + 127u) & ~127u;
    const uint32_t s_x = base, s_B = s_x + kTile * kXB, s_C = s_B + kTile * kNB, s_hi = s_C + kTile * kNB, s_lo = s_hi + kTile * 128;
    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
    const int head = int(blockIdx.x) % a.heads, index = int(blockIdx.x) / a.heads, col0 = int(blockIdx.y) * WARPS * 16;
    grid_dependency_wait();
    grid_launch_dependents();
    int run = 0, seg = 0, segs = 0;
    find_segment(a, cut.segment, index, run, seg, segs);
    if (segs == 0 || (STATES && seg == segs - 1)) { // (what a run's last segment adds is not asked for)
        return;
    }
    const int first = a.q_starts[run], n_new = a.q_starts[run + 1] - first, pos_last = a.kv_lens[run] - 1;
    const int64_t slot = a.seq_ids[run];
    if (!STATES && seg == 0 && blockIdx.y == 0) {
        keep_run_inputs<__nv_bfloat16>(a, head, slot, first, first + n_new - 1, pos_last);
    }
    const int from = seg * cut.segment, upto = segs == 1 ? n_new : min(n_new, from + cut.segment);
    const int group = head / (a.heads / a.groups), dvb = min(a.dv - col0, WARPS * 16);
    const __nv_bfloat16 *conv = reinterpret_cast<const __nv_bfloat16 *>(a.scratch + sc.conv);
    const float *dts = a.scratch + sc.dt;
    const float rate = -expf(a.a_log[head]), skip = a.d_skip[head];

    // S^T: c[j][0..1] = (p0 + g; n = 8 j + 2 q, + 1), c[j][2..3] = (p0 + g + 8; ..), p0 = col0 + 16 warp
    float S[NT][4];
    const int p0 = col0 + warp * 16;
    auto each_state = [&](float *state, auto &&use) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = 8 * j + 2 * q + (e & 1), p = p0 + g + (e >> 1) * 8;
                use(S[j][e], state + int64_t(n) * a.dv + p, n < a.dk && p < a.dv);
            }
        }
    };
    float *slot_state = a.state + slot * a.slot_stride + int64_t(head) * a.dk * a.dv;
    float *cut_state = cut.states + (int64_t(index) * a.heads + head) * a.dk * a.dv;
    if (STATES || (segs == 1 && pos_last + 1 == n_new)) {
        each_state(nullptr, [](float &s, const float *, bool) { s = 0.f; });
    } else {
        each_state(segs == 1 ? slot_state : cut_state, [](float &s, const float *at, bool holds) { s = holds ? *at : 0.f; });
    }

    auto fetch = [&](int t0) {
        const int n_x = WARPS * 2, n_b = NT; // 16-byte pieces of a row
        auto rows = [&](uint32_t dst, int row_bytes, int pieces, int valid, const __nv_bfloat16 *src) {
            for (int u = tid; u < kTile * pieces; u += WARPS * 32) {
                const int t = u / pieces, c = u - t * pieces;
                const bool in = t0 + t < upto && c * 8 < valid;
                cp_async_16(dst + swz(t, c, row_bytes), in ? src + int64_t(first + t0 + t) * sc.conv_stride + c * 8 : conv, in ? 16 : 0);
            }
        };
        rows(s_x, kXB, n_x, dvb, conv + head * a.dv + col0);
        rows(s_B, kNB, n_b, a.dk, conv + a.inner() + group * a.dk);
        if (!STATES) {
            rows(s_C, kNB, n_b, a.dk, conv + a.inner() + (a.groups + group) * a.dk);
        }
        cp_async_commit();
        if (warp == 0) { // step sizes and the running log decay, two tokens per lane
            const int t = t0 + 2 * lane;
            const float d0 = t < upto ? dts[int64_t(first + t) * a.heads + head] : 0.f;
            const float d1 = t + 1 < upto ? dts[int64_t(first + t + 1) * a.heads + head] : 0.f;
            float sum = rate * d0 + rate * d1;
#pragma unroll
            for (int o = 1; o < 32; o *= 2) {
                const float v = __shfl_up_sync(0xffffffffu, sum, o);
                sum += lane >= o ? v : 0.f;
            }
            s_dt[2 * lane] = d0;
            s_dt[2 * lane + 1] = d1;
            s_b[2 * lane] = sum - rate * d1;
            s_b[2 * lane + 1] = sum;
            if (lane == 31) {
                s_end = sum;
            }
        }
        cp_async_wait<0>();
        __syncthreads();
    };

    float decay = 0.f;
    constexpr float kLog2e = 1.4426950408889634f;
    const int lm_row = (lane & 7) + ((lane >> 3) & 1) * 8, lm_chunk = lane >> 4;  // rows 0 - 15 of two 8-column chunks
    const int lt_row = (lane & 7) + (lane >> 4) * 8, lt_chunk = (lane >> 3) & 1;  // the other order of the four matrices
    for (int t0 = from; t0 < upto; t0 += kTile) {
        fetch(t0);
        float Y[4][2][4];
        if constexpr (!STATES) {
            // scores: 16 tokens x 32 tokens per unit, lower triangle only
            for (int unit = warp; unit < 8; unit += WARPS) {
                const int m = unit >> 1, half = unit & 1;
                if (half * 32 > m * 16 + 15) {
                    continue;
                }
                float G[4][4] = {};
#pragma unroll
                for (int ks = 0; ks < NT / 2; ++ks) {
                    uint32_t c[4];
                    ldmatrix_x4(c, s_C + swz(m * 16 + lm_row, 2 * ks + lm_chunk, kNB));
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        uint32_t b[4];
                        ldmatrix_x4(b, s_B + swz(half * 32 + j * 16 + lt_row, 2 * ks + lt_chunk, kNB));
                        mma_bf16(G[2 * j], c, b[0], b[1]);
                        mma_bf16(G[2 * j + 1], c, b[2], b[3]);
                    }
                }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int s = half * 32 + j * 8 + 2 * q;
                    const float b0 = s_b[s], b1 = s_b[s + 1], d0 = s_dt[s], d1 = s_dt[s + 1];
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const int t = m * 16 + g + r * 8;
                        const float bt = s_b[t];
                        const float v0 = s <= t ? G[j][2 * r] * d0 * ex2((bt - b0) * kLog2e) : 0.f;
                        const float v1 = s + 1 <= t ? G[j][2 * r + 1] * d1 * ex2((bt - b1) * kLog2e) : 0.f;
                        uint32_t hi, lo;
                        split2(v0, v1, hi, lo);
                        const uint32_t at = swz(t, s >> 3, 128) + uint32_t(s & 7) * 2;
                        asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(s_hi + at), "r"(hi) : "memory");
                        asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(s_lo + at), "r"(lo) : "memory");
                    }
                }
            }
            // y = e^(b_t) S^T C_t
#pragma unroll
            for (int m = 0; m < 4; ++m) {
#pragma unroll
                for (int j = 0; j < 2; ++j) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        Y[m][j][e] = 0.f;
                    }
                }
            }
#pragma unroll
            for (int ks = 0; ks < NT / 2; ++ks) {
                uint32_t hi[4], lo[4]; // value columns 0 - 7: (k 0 - 7, k 8 - 15), columns 8 - 15: the same
                split2(S[2 * ks][0], S[2 * ks][1], hi[0], lo[0]);
                split2(S[2 * ks + 1][0], S[2 * ks + 1][1], hi[1], lo[1]);
                split2(S[2 * ks][2], S[2 * ks][3], hi[2], lo[2]);
                split2(S[2 * ks + 1][2], S[2 * ks + 1][3], hi[3], lo[3]);
#pragma unroll
                for (int m = 0; m < 4; ++m) {
                    uint32_t c[4];
                    ldmatrix_x4(c, s_C + swz(m * 16 + lm_row, 2 * ks + lm_chunk, kNB));
                    mma_bf16(Y[m][0], c, hi[0], hi[1]);
                    mma_bf16(Y[m][1], c, hi[2], hi[3]);
                    mma_bf16(Y[m][0], c, lo[0], lo[1]);
                    mma_bf16(Y[m][1], c, lo[2], lo[3]);
                }
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                const float e0 = ex2(s_b[m * 16 + g] * kLog2e), e1 = ex2(s_b[m * 16 + g + 8] * kLog2e);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    Y[m][j][0] *= e0;
                    Y[m][j][1] *= e0;
                    Y[m][j][2] *= e1;
                    Y[m][j][3] *= e1;
                }
            }
            __syncthreads(); // the scores are complete
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                uint32_t x[4];
                ldmatrix_x4_trans(x, s_x + swz(ks * 16 + lm_row, warp * 2 + lm_chunk, kXB));
#pragma unroll
                for (int m = ks; m < 4; ++m) {
                    uint32_t w[4];
                    ldmatrix_x4(w, s_hi + swz(m * 16 + lm_row, 2 * ks + lm_chunk, 128));
                    mma_bf16(Y[m][0], w, x[0], x[1]);
                    mma_bf16(Y[m][1], w, x[2], x[3]);
                    ldmatrix_x4(w, s_lo + swz(m * 16 + lm_row, 2 * ks + lm_chunk, 128));
                    mma_bf16(Y[m][0], w, x[0], x[1]);
                    mma_bf16(Y[m][1], w, x[2], x[3]);
                }
            }
            __nv_bfloat16 *y = reinterpret_cast<__nv_bfloat16 *>(a.scratch + sc.y) + int64_t(first + t0) * sc.y_stride + int64_t(head) * a.dv;
#pragma unroll
            for (int m = 0; m < 4; ++m) {
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int t = m * 16 + g + r * 8;
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const int p = warp * 16 + j * 8 + 2 * q; // in the CTA's columns
                        if (t0 + t < upto && p < dvb) {
                            uint32_t x;
                            asm volatile("ld.shared.b32 %0, [%1];\n" : "=r"(x) : "r"(s_x + swz(t, p >> 3, kXB) + uint32_t(p & 7) * 2));
                            *reinterpret_cast<uint32_t *>(y + int64_t(t) * sc.y_stride + col0 + p) =
                                pack_bf16(fmaf(skip, lo_half(x), Y[m][j][2 * r]), fmaf(skip, hi_half(x), Y[m][j][2 * r + 1]));
                        }
                    }
                }
            }
        }
        // the state
        const float end = s_end, keep = ex2(end * kLog2e);
        decay += end;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                S[j][e] *= keep;
            }
        }
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            uint32_t x[4], hi[4], lo[4];
            ldmatrix_x4_trans(x, s_x + swz(ks * 16 + lt_row, warp * 2 + lt_chunk, kXB));
#pragma unroll
            for (int h = 0; h < 2; ++h) { // tokens 2 q, 2 q + 1 and the same eight further on
                const int s = ks * 16 + h * 8 + 2 * q;
                const float w0 = s_dt[s] * ex2((end - s_b[s]) * kLog2e), w1 = s_dt[s + 1] * ex2((end - s_b[s + 1]) * kLog2e);
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    split2(lo_half(x[2 * h + r]) * w0, hi_half(x[2 * h + r]) * w1, hi[2 * h + r], lo[2 * h + r]);
                }
            }
#pragma unroll
            for (int j = 0; j < NT / 2; ++j) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, s_B + swz(ks * 16 + lm_row, 2 * j + lm_chunk, kNB));
                mma_bf16(S[2 * j], hi, b[0], b[1]);
                mma_bf16(S[2 * j + 1], hi, b[2], b[3]);
                mma_bf16(S[2 * j], lo, b[0], b[1]);
                mma_bf16(S[2 * j + 1], lo, b[2], b[3]);
            }
        }
        __syncthreads(); // before the next tile's operands arrive
    }
    if (STATES) {
        each_state(cut_state, [](float &s, float *at, bool holds) {
            if (holds) {
                *at = s;
            }
        });
        if (tid == 0 && blockIdx.y == 0) {
            cut.decays[int64_t(index) * a.heads + head] = decay;
        }
    } else if (seg == segs - 1) {
        each_state(slot_state, [](float &s, float *at, bool holds) {
            if (holds) {
                *at = s;
            }
        });
    }
}

// What segments add -> the states in front of them, run by run: thread = one element of a (run, head); kAhead segments are fetched
// together.
__global__ void __launch_bounds__(256) state_scan_kernel(StateSpaceArgs a, Cut cut) {
    constexpr int kAhead = 4;
    grid_dependency_wait();
    grid_launch_dependents();
    const int head = int(blockIdx.x) % a.heads, run = int(blockIdx.x) / a.heads, size = a.dk * a.dv;
    const int n_new = a.q_starts[run + 1] - a.q_starts[run];
    const int segs = n_new > 1 ? (n_new + cut.segment - 1) / cut.segment : 0;
    if (segs <= 1) {
        return;
    }
    int index = 0; // of the run's first segment
    for (int i = int(threadIdx.x); i < run; i += 256) {
        const int len = a.q_starts[i + 1] - a.q_starts[i];
        index += len > 1 ? (len + cut.segment - 1) / cut.segment : 0;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        index += __shfl_xor_sync(0xffffffffu, index, o);
    }
    __shared__ int s_index[8];
    if ((threadIdx.x & 31) == 0) {
        s_index[threadIdx.x >> 5] = index;
    }
    __syncthreads();
    index = 0;
    for (int w = 0; w < 8; ++w) {
        index += s_index[w];
    }
    const int at = int(blockIdx.y) * 256 + int(threadIdx.x);
    if (at >= size) {
        return;
    }
    const bool fresh = a.kv_lens[run] == n_new;
    float s = fresh ? 0.f : a.state[int64_t(a.seq_ids[run]) * a.slot_stride + int64_t(head) * size + at];
    auto place = [&](int k) { return cut.states + (int64_t(index + k) * a.heads + head) * size + at; };
    for (int k0 = 0; k0 < segs; k0 += kAhead) {
        float added[kAhead], keep[kAhead];
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const bool more = k0 + i + 1 < segs; // (behind the last segment nothing starts)
            added[i] = more ? *place(k0 + i) : 0.f;
            keep[i] = more ? cut.decays[int64_t(index + k0 + i) * a.heads + head] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            if (k0 + i < segs) {
                *place(k0 + i) = s;
                s = fmaf(s, expf(keep[i]), added[i]);
            }
        }
    }
}

template <int NT, int WARPS>
void run_tiles(cudaStream_t s, const StateSpaceArgs &a, const StateScratch &sc) {
    constexpr int kNB = NT * 16 < 128 ? 128 : NT * 16, kXB = WARPS * 32 < 128 ? 128 : WARPS * 32;
    constexpr size_t smem = 128 + size_t(kTile) * (kXB + 2 * kNB + 2 * 128);
    const int blocks = (a.dv + WARPS * 16 - 1) / (WARPS * 16);
    // segments: as many as fill the GPU a few times over, if the scratch holds their states
    Cut cut{1 << 30, a.segments, nullptr};
    int segments = a.n_seqs;
    const int64_t tiles = (a.n_rows + kTile - 1) / kTile + a.n_seqs; // at most
    if (a.segments != nullptr && int64_t(a.n_seqs) * a.heads * blocks < kWantedCtas / 2) {
        const int64_t wanted = std::max<int64_t>(1, kWantedCtas / (int64_t(a.heads) * blocks));
        const int per = int(std::max<int64_t>(2, (tiles + wanted - 1) / wanted)) * kTile;
        const int64_t bound = a.n_rows / per + a.n_seqs;
        const size_t floats = size_t(bound) * a.heads * a.dk * a.dv;
        if (per < a.max_q_len && floats + size_t(bound) * a.heads <= a.segment_floats) {
            cut.segment = per;
            cut.decays = a.segments + floats;
            segments = int(bound);
        }
    }
    const dim3 grid(unsigned(segments) * unsigned(a.heads), unsigned(blocks));
    auto prepare = [&](auto kernel) {
        if (smem > 48 * 1024) {
            LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        }
        return kernel;
    };
    if (cut.segment < (1 << 30)) {
        launch_programmatic_smem(prepare(state_tiles_kernel<NT, WARPS, true>), grid, WARPS * 32, smem, s, a, sc, cut);
        launch_programmatic(state_scan_kernel, dim3(unsigned(a.n_seqs) * unsigned(a.heads), unsigned((a.dk * a.dv + 255) / 256)), 256u, s, a, cut);
    }
    launch_programmatic_smem(prepare(state_tiles_kernel<NT, WARPS, false>), grid, WARPS * 32, smem, s, a, sc, cut);
    check_launch("state_space tiles");
}

} // namespace

bool state_space_tiles_fit(llaisysDataType_t dtype, const StateSpaceArgs &a) {
    return dtype == LLAISYS_DTYPE_BF16 && a.dk <= 128 && a.dk % 8 == 0 && a.dv % 8 == 0 && a.max_q_len > 1;
}

size_t state_space_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv) {
    if (dtype != LLAISYS_DTYPE_BF16 || dk > 128 || heads == 0) {
        return 0;
    }
    return std::max<size_t>(kMaxPairs / heads, 1) * heads * (dk * dv + 1);
}

void state_space_tiles(stream_t stream, const StateSpaceArgs &a) {
    const StateScratch sc = state_scratch(LLAISYS_DTYPE_BF16, a.n_rows, a.heads, a.groups, a.dk, a.dv);
    auto s = static_cast<cudaStream_t>(stream);
    auto by_width = [&](auto warps) {
        constexpr int kWarps = decltype(warps)::value;
        if (a.dk <= 32) {
            run_tiles<4, kWarps>(s, a, sc);
        } else if (a.dk <= 64) {
            run_tiles<8, kWarps>(s, a, sc);
        } else {
            run_tiles<16, kWarps>(s, a, sc);
        }
    };
    if (a.dv <= 64) {
        by_width(std::integral_constant<int, 4>{});
    } else {
        by_width(std::integral_constant<int, 8>{});
    }
}

} // namespace llaisys::kernels
