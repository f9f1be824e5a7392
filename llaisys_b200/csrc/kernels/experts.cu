// Mixture of experts (see ExpertArgs): the choice of experts, the line of rows sorted by expert, the plain form of the experts'
// products (any dtype and sizes, f32 accumulation), and the sum into the stream with the norm that follows. The tensor-core form
// of the products is experts_tc.cu; it serves 16-bit models whose rows are whole 16-byte pieces.
#include "experts.cuh"
#include "launch_utils.cuh"
#include "mma_utils.cuh"

#include <cfloat>

namespace llaisys::kernels {

namespace {

constexpr int kRouteWarps = 4;

struct Best {
    float v;
    int i;
};
// The largest value of the warp's lanes, the lowest index among equals; the same for every lane.
__device__ __forceinline__ Best warp_best(Best b) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, b.v, o);
        const int i = __shfl_xor_sync(0xffffffffu, b.i, o);
        if (v > b.v || (v == b.v && i < b.i)) {
            b.v = v;
            b.i = i;
        }
    }
    return b;
}
__device__ __forceinline__ Best best_of(const float *v, int n, int lane) {
    Best b{-INFINITY, 0x7fffffff};
    for (int i = lane; i < n; i += 32) {
        const float x = v[i];
        if (x > b.v || (x == b.v && i < b.i)) {
            b.v = x;
            b.i = i;
        }
    }
    b = warp_best(b);
    b.i = b.i < n ? b.i : 0; // (NaN everywhere: any valid index)
    return b;
}

// One warp per row. Shared memory per warp: scores, choice scores and group scores.
__global__ void __launch_bounds__(kRouteWarps * 32) experts_route_kernel(ExpertArgs a) {
    extern __shared__ float smem[];
    grid_dependency_wait();
    grid_launch_dependents();
    const int warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31;
    const int row = int(blockIdx.x) * kRouteWarps + warp;
    const int n = a.experts + a.identity, size = n / a.groups;
    if (row >= a.n_rows) {
        return;
    }
    float *score = smem + warp * (2 * n + a.groups), *choice = score + n, *group = choice + n;
    const float *z = a.logits + int64_t(row) * n;
    float mx = -INFINITY;
    for (int i = lane; i < n; i += 32) {
        score[i] = z[i];
        mx = fmaxf(mx, z[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    }
    float sum = 0.f;
    for (int i = lane; i < n; i += 32) {
        score[i] = expf(score[i] - mx);
        sum += score[i];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sum += __shfl_xor_sync(0xffffffffu, sum, o);
    }
    const float inv = 1.f / sum;
    for (int i = lane; i < n; i += 32) {
        score[i] *= inv;
        choice[i] = score[i] + a.correction[i];
    }
    __syncwarp();
    if (a.keep < a.groups) {
        for (int g = lane; g < a.groups; g += 32) {
            float m = -INFINITY;
            for (int i = 0; i < size; ++i) {
                m = fmaxf(m, choice[g * size + i]);
            }
            group[g] = m;
        }
        __syncwarp();
        // the groups that stay are marked with +inf one after the other; the others' choice scores fall to -inf
        for (int k = 0; k < a.keep; ++k) {
            Best b{-INFINITY, 0x7fffffff};
            for (int g = lane; g < a.groups; g += 32) {
                const float v = group[g];
                if (v != INFINITY && (v > b.v || (v == b.v && g < b.i))) {
                    b.v = v;
                    b.i = g;
                }
            }
            b = warp_best(b);
            if (lane == 0 && b.i < a.groups) {
                group[b.i] = INFINITY;
            }
            __syncwarp();
        }
        for (int i = lane; i < n; i += 32) {
            if (group[i / size] != INFINITY) {
                choice[i] = -INFINITY;
            }
        }
        __syncwarp();
    }
    float total = 0.f, mine = 0.f;
    int my_expert = 0;
    for (int k = 0; k < a.top; ++k) {
        const Best b = best_of(choice, n, lane);
        const float s = score[b.i];
        total += s;
        if (k % 32 == lane) {
            mine = s;
            my_expert = b.i;
        }
        __syncwarp();
        if (lane == 0) {
            choice[b.i] = -INFINITY;
        }
        __syncwarp();
        if (k % 32 == 31 || k == a.top - 1) { // a full round of lanes (or the last) goes out
            const int slot = k / 32 * 32 + lane;
            if (slot <= k) {
                const int64_t at = int64_t(row) * a.top + slot;
                a.chosen[at] = my_expert;
                a.weights[at] = mine;
                a.place[at] = my_expert < a.experts ? atomicAdd(a.counts + my_expert, 1) : -1; // rank within the expert
            }
        }
    }
    const float factor = a.scale / (total + 1e-20f);
    for (int k = lane; k < a.top; k += 32) {
        a.weights[int64_t(row) * a.top + k] *= factor;
    }
}

// Ranks within experts become rows of the line (the experts' rows one after the other); every row of the line learns its source
// row, and (rows != null) receives a copy of it. One CTA per source row.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) experts_place_kernel(ExpertArgs a) {
    struct alignas(sizeof(T) * VEC) Piece {
        T v[VEC];
    };
    extern __shared__ int32_t s_place[]; // [top]
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = int(blockIdx.x), warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31;
    for (int k = warp; k < a.top; k += int(blockDim.x) >> 5) {
        const int64_t at = int64_t(row) * a.top + k;
        const int e = a.chosen[at];
        int place = -1;
        if (e < a.experts) {
            int before = 0;
            for (int i = lane; i < e; i += 32) {
                before += a.counts[i];
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                before += __shfl_xor_sync(0xffffffffu, before, o);
            }
            place = before + a.place[at];
            __syncwarp();
            if (lane == 0) {
                a.place[at] = place;
                a.line[place] = row;
            }
        }
        if (lane == 0) {
            s_place[k] = place;
        }
    }
    if (a.rows == nullptr) {
        return;
    }
    __syncthreads();
    const Piece *src = reinterpret_cast<const Piece *>(static_cast<const T *>(a.h) + int64_t(row) * a.width);
    for (int i = int(threadIdx.x); i < a.width / VEC; i += int(blockDim.x)) {
        const Piece p = src[i];
        for (int k = 0; k < a.top; ++k) {
            if (s_place[k] >= 0) {
                reinterpret_cast<Piece *>(static_cast<T *>(a.rows) + int64_t(s_place[k]) * a.width)[i] = p;
            }
        }
    }
}

// out[r, j] = in[src(r), :] . w_e[j, :] for the rows of a tile, or (GLU) silu of that times the same with w_e[n + j, :].
// CTA: 32 rows x 64 columns, thread: 2 rows x 4 columns.
template <typename T, bool GLU>
__global__ void __launch_bounds__(256) experts_plain_kernel(ExpertArgs a, const T *__restrict__ in, const int32_t *__restrict__ line,
                                                            const T *__restrict__ weight, T *__restrict__ out, int n, int k) {
    constexpr int kRows = 32, kCols = 64, kDepth = 32, kParts = GLU ? 2 : 1;
    __shared__ float s_in[kDepth][kRows + 1], s_w[kParts][kDepth][kCols + 4];
    grid_dependency_wait();
    grid_launch_dependents();
    int expert = 0, first = 0, rows = 0;
    find_tile(a.counts, a.experts, kRows, int(blockIdx.y), expert, first, rows);
    if (rows == 0) {
        return;
    }
    const int col0 = int(blockIdx.x) * kCols, tid = int(threadIdx.x), tx = tid % 16, ty = tid / 16;
    const T *w = weight + int64_t(expert) * kParts * n * k;
    float acc[kParts][2][4] = {};
    for (int k0 = 0; k0 < k; k0 += kDepth) {
        for (int i = tid; i < kRows * kDepth; i += 256) {
            const int r = i / kDepth, c = i % kDepth;
            float v = 0.f;
            if (r < rows && k0 + c < k) {
                const int64_t src = line != nullptr ? line[first + r] : first + r;
                v = to_f32(in[src * k + k0 + c]);
            }
            s_in[c][r] = v;
        }
        for (int i = tid; i < kParts * kCols * kDepth; i += 256) {
            const int part = i / (kCols * kDepth), j = i / kDepth % kCols, c = i % kDepth;
            s_w[part][c][j] = col0 + j < n && k0 + c < k ? to_f32(w[(int64_t(part) * n + col0 + j) * k + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int c = 0; c < kDepth; ++c) {
            const float x0 = s_in[c][2 * ty], x1 = s_in[c][2 * ty + 1];
#pragma unroll
            for (int part = 0; part < kParts; ++part) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float ww = s_w[part][c][tx * 4 + j];
                    acc[part][0][j] = fmaf(x0, ww, acc[part][0][j]);
                    acc[part][1][j] = fmaf(x1, ww, acc[part][1][j]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int col = col0 + tx * 4 + j;
            if (2 * ty + r < rows && col < n) {
                float v = acc[0][r][j];
                if constexpr (GLU) {
                    v = v / (1.f + expf(-v)) * acc[kParts - 1][r][j];
                }
                out[int64_t(first + 2 * ty + r) * n + col] = from_f32<T>(v);
            }
        }
    }
}

__device__ __forceinline__ float block_total(float v) {
    __shared__ float part[32];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        v += __shfl_xor_sync(0xffffffffu, v, o);
    }
    if ((threadIdx.x & 31) == 0) {
        part[threadIdx.x >> 5] = v;
    }
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < int(blockDim.x >> 5); ++i) {
        tot += part[i]; // every thread adds the few partials in the same order
    }
    return tot;
}

// One CTA per row: x += sum of the weighted outputs, in the order of the choices; then the norm that follows. The first PER_THREAD
// pieces of a thread stay in registers.
template <typename T, int VEC, int PER_THREAD>
__global__ void experts_combine_kernel(ExpertArgs a, float *__restrict__ x, T *next, const float *__restrict__ gain, float eps) {
    struct alignas(sizeof(T) * VEC) Piece {
        T v[VEC];
    };
    struct alignas(4 * VEC) F {
        float v[VEC];
    };
    extern __shared__ float s_w[]; // [top] weights, [top] places
    int32_t *s_place = reinterpret_cast<int32_t *>(s_w + a.top);
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    for (int k = int(threadIdx.x); k < a.top; k += int(blockDim.x)) {
        s_w[k] = a.weights[row * a.top + k];
        s_place[k] = a.place[row * a.top + k];
    }
    if (blockIdx.x == 0) { // the next layer's routing starts from zero
        for (int e = int(threadIdx.x); e < a.experts; e += int(blockDim.x)) {
            a.counts[e] = 0;
        }
    }
    __syncthreads();
    const int n_vec = a.width / VEC, step = int(blockDim.x);
    F *xr = reinterpret_cast<F *>(x + row * a.width);
    const T *h = static_cast<const T *>(a.h) + row * a.width, *out = static_cast<const T *>(a.out);
    float ss = 0.f;
    auto add = [&](int i) {
        F f = xr[i], sum{};
        for (int k = 0; k < a.top; ++k) {
            const T *src = s_place[k] < 0 ? h : out + int64_t(s_place[k]) * a.width;
            const Piece p = reinterpret_cast<const Piece *>(src)[i];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                sum.v[e] = fmaf(s_w[k], to_f32(p.v[e]), sum.v[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            f.v[e] += sum.v[e];
            ss = fmaf(f.v[e], f.v[e], ss);
        }
        xr[i] = f;
        return f;
    };
    F held[PER_THREAD];
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int i = int(threadIdx.x) + r * step;
        if (i < n_vec) {
            held[r] = add(i);
        }
    }
    for (int i = int(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        add(i);
    }
    if (next == nullptr) {
        return;
    }
    const float inv = rsqrtf(block_total(ss) / float(a.width) + eps) * *gain;
    auto store = [&](int i, const F &f) {
        Piece o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            o.v[e] = from_f32<T>(f.v[e] * inv);
        }
        reinterpret_cast<Piece *>(next + row * a.width)[i] = o;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int i = int(threadIdx.x) + r * step;
        if (i < n_vec) {
            store(i, held[r]);
        }
    }
    for (int i = int(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        store(i, xr[i]); // (written by this thread)
    }
}

void check_args(const ExpertArgs &a) {
    CHECK_ARGUMENT(a.experts > 0 && a.identity >= 0 && a.top > 0 && a.groups > 0 && (a.experts + a.identity) % a.groups == 0 && a.keep > 0 &&
                       a.keep <= a.groups && a.top <= a.keep * ((a.experts + a.identity) / a.groups) && a.width > 0 && a.ff > 0,
                   "experts: inconsistent sizes");
    CHECK_ARGUMENT(a.experts + a.identity <= 2048 && int64_t(a.n_rows) * a.top < (int64_t(1) << 31) && a.top <= 1024, "experts: too many");
}

} // namespace

void experts_route(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &a) {
    (void)dtype;
    if (a.n_rows == 0) {
        return;
    }
    check_args(a);
    const size_t smem = size_t(kRouteWarps) * (2 * size_t(a.experts + a.identity) + size_t(a.groups)) * sizeof(float);
    static_assert(kRouteWarps * 3 * 2048 * 4 <= 99 * 1024, "routing scores in shared memory");
    if (smem > 48 * 1024) {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(experts_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    }
    launch_programmatic_smem(experts_route_kernel, dim3(unsigned((a.n_rows + kRouteWarps - 1) / kRouteWarps)), kRouteWarps * 32, smem,
                             static_cast<cudaStream_t>(stream), a);
    check_launch("experts_route");
}

void experts_apply(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &args) {
    if (args.n_rows == 0) {
        return;
    }
    check_args(args);
    auto s = static_cast<cudaStream_t>(stream);
    ExpertArgs a = args;
    const bool tc = experts_tc_covers(dtype, a);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        if (!tc) {
            a.rows = nullptr; // read through the line
        }
        constexpr int kVec = 16 / int(sizeof(T));
        const bool wide = a.width % kVec == 0 && aligned16(a.h) && aligned16(a.rows);
        auto place = wide ? experts_place_kernel<T, kVec> : experts_place_kernel<T, 1>;
        const int vecs = wide ? a.width / kVec : a.width;
        const unsigned block = vecs <= 64 ? 64u : (vecs <= 128 ? 128u : 256u);
        launch_programmatic_smem(place, dim3(unsigned(a.n_rows)), block, size_t(a.top) * 4, s, a);
        if (tc) {
            experts_tc(stream, dtype, a);
            return;
        }
        const int64_t tiles = expert_tiles_bound(a, 32);
        CHECK_ARGUMENT(tiles <= 65535, "experts: too many rows for the plain form");
        launch_programmatic(experts_plain_kernel<T, true>, dim3(unsigned((a.ff + 63) / 64), unsigned(tiles)), 256u, s, a, static_cast<const T *>(a.h),
                            a.line, static_cast<const T *>(a.gate_up), static_cast<T *>(a.act), a.ff, a.width);
        launch_programmatic(experts_plain_kernel<T, false>, dim3(unsigned((a.width + 63) / 64), unsigned(tiles)), 256u, s, a,
                            static_cast<const T *>(a.act), nullptr, static_cast<const T *>(a.down), static_cast<T *>(a.out), a.width, a.ff);
    });
    check_launch("experts_apply");
}

void experts_combine(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &a, float *x, void *next, const float *gain, float eps) {
    if (a.n_rows == 0) {
        return;
    }
    check_args(a);
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = a.width % 4 == 0 && aligned16(x) && aligned16(a.h) && aligned16(a.out) && aligned16(next);
        auto kernel = wide ? experts_combine_kernel<T, 4, 4> : experts_combine_kernel<T, 1, 4>;
        const int vecs = wide ? a.width / 4 : a.width;
        const int want = (vecs + 1) / 2, block = want < 64 ? 64 : (want > 1024 ? 1024 : (want + 31) / 32 * 32);
        launch_programmatic_smem(kernel, dim3(unsigned(a.n_rows)), unsigned(block), size_t(a.top) * 8, s, a, x, static_cast<T *>(next), gain, eps);
    });
    check_launch("experts_combine");
}

} // namespace llaisys::kernels
