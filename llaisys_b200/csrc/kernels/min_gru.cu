// minGRU (MinGruArgs): a gated recurrence per channel whose gates read the current token only, so a run of tokens is a chain of
// affine maps S -> a S + b that compose in any grouping.
//
// Roofline: HBM (three projections read, one activation written, per token and channel). Decode: a thread per (sequence, VEC
// channels). Runs: one pass over the rows. A cluster of up to 8 CTAs owns a slice of 8 x VEC channels of one sequence and walks
// its tokens in tiles of 256 per CTA; a thread holds 8 tokens x VEC channels in registers, composes them, the CTA scans its 32
// groups of tokens with shuffles, and the CTAs of the cluster hand their totals to one another through distributed shared memory.
// State and gates are f32.
#include "gated_linear.cuh"
#include "kernels.hpp"
#include "mma_utils.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace llaisys::kernels {

namespace {

constexpr int kThreads = 256, kLanes = 8 /* threads side by side over channels */, kGroups = kThreads / kLanes, kTokens = 8;
constexpr int kTile = kGroups * kTokens, kMaxCluster = 8;

// 1 / (1 + e^-x); the 16-bit forms divide and exponentiate with the fast approximations (relative error near 2^-21)
template <typename T>
__device__ __forceinline__ float sigmoid(float x) {
    if constexpr (sizeof(T) == 4) {
        return 1.f / (1.f + expf(-x));
    } else {
        return __fdividef(1.f, 1.f + __expf(fminf(-x, 80.f)));
    }
}
template <typename T>
__device__ __forceinline__ void affine(float z, float u, float &a, float &b) {
    const float s = sigmoid<T>(z);
    a = 1.f - s;
    b = s * (u >= 0.f ? u + 0.5f : sigmoid<T>(u));
}

template <typename T, int VEC>
__global__ void min_gru_decode_kernel(MinGruArgs a) {
    grid_dependency_wait();
    grid_launch_dependents();
    using P = Pieces<T, VEC>;
    const int seq = blockIdx.y, c = (int(blockIdx.x) * int(blockDim.x) + int(threadIdx.x)) * VEC;
    if (c >= a.width) {
        return;
    }
    const T *row = static_cast<const T *>(a.proj) + int64_t(seq) * a.row_stride + c;
    const P z = *reinterpret_cast<const P *>(row + a.z_at), u = *reinterpret_cast<const P *>(row + a.x_at),
            g = *reinterpret_cast<const P *>(row + a.g_at);
    const P bz = *reinterpret_cast<const P *>(static_cast<const T *>(a.bias_z) + c), bx = *reinterpret_cast<const P *>(static_cast<const T *>(a.bias_x) + c);
    using S = Pieces<float, VEC>;
    S *state = reinterpret_cast<S *>(a.state + int64_t(a.seq_ids[seq]) * a.slot_stride + c);
    S s{};
    if (a.kv_lens[seq] > 1) {
        s = *state;
    }
    P o;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        float keep, add;
        affine<T>(to_f32(z.v[e]) + to_f32(bz.v[e]), to_f32(u.v[e]) + to_f32(bx.v[e]), keep, add);
        s.v[e] = fmaf(keep, s.v[e], add);
        const float gv = to_f32(g.v[e]);
        o.v[e] = from_f32<T>(s.v[e] * gv * sigmoid<T>(gv));
    }
    *state = s;
    *reinterpret_cast<P *>(static_cast<T *>(a.out) + int64_t(seq) * a.out_stride + c) = o;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads, 2) min_gru_chunk_kernel(MinGruArgs a) {
    grid_dependency_wait();
    grid_launch_dependents();
    constexpr int kChannels = kLanes * VEC;
    using P = Pieces<T, VEC>;
    __shared__ float s_a[kChannels][kGroups + 1], s_b[kChannels][kGroups + 1]; // a tile's groups, then what comes before each
    __shared__ float s_all[2][kMaxCluster][2][kChannels];                      // [parity][CTA][a | b]: tile totals
    const cg::cluster_group cluster = cg::this_cluster();
    const int n_ctas = int(cluster.num_blocks()), rank = int(cluster.block_rank());
    const int seq = blockIdx.y, slice = int(blockIdx.x) / n_ctas;
    const int group = int(threadIdx.x) / kLanes, lc = int(threadIdx.x) % kLanes * VEC, c = slice * kChannels + lc;
    const int warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31;
    const int64_t row0 = a.q_starts[seq];
    const int len = a.q_starts[seq + 1] - int(row0);
    const bool holds = c < a.width; // (VEC divides the width)
    float *state = a.state + int64_t(a.seq_ids[seq]) * a.slot_stride + c;
    float carry[VEC], bz[VEC], bx[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        carry[e] = holds && a.kv_lens[seq] > len ? state[e] : 0.f;
        bz[e] = holds ? to_f32(static_cast<const T *>(a.bias_z)[c + e]) : 0.f;
        bx[e] = holds ? to_f32(static_cast<const T *>(a.bias_x)[c + e]) : 0.f;
    }
    const T *proj = static_cast<const T *>(a.proj) + row0 * a.row_stride + c;
    T *out = static_cast<T *>(a.out) + row0 * a.out_stride + c;
    int parity = 0;
    for (int base = 0; base < len; base += kTile * n_ctas, parity ^= 1) {
        const int t0 = base + rank * kTile + group * kTokens;
        P z[kTokens], u[kTokens], g[kTokens];
#pragma unroll
        for (int i = 0; i < kTokens; ++i) {
            if (holds && t0 + i < len) {
                const T *row = proj + int64_t(t0 + i) * a.row_stride;
                z[i] = *reinterpret_cast<const P *>(row + a.z_at);
                u[i] = *reinterpret_cast<const P *>(row + a.x_at);
                g[i] = *reinterpret_cast<const P *>(row + a.g_at);
            }
        }
        float keep[kTokens][VEC], add[kTokens][VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float ta = 1.f, tb = 0.f;
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                keep[i][e] = 1.f;
                add[i][e] = 0.f;
                if (holds && t0 + i < len) {
                    affine<T>(to_f32(z[i].v[e]) + bz[e], to_f32(u[i].v[e]) + bx[e], keep[i][e], add[i][e]);
                }
                ta *= keep[i][e];
                tb = fmaf(keep[i][e], tb, add[i][e]);
            }
            s_a[lc + e][group] = ta;
            s_b[lc + e][group] = tb;
        }
        __syncthreads();
#pragma unroll
        for (int w = 0; w < kChannels / 8; ++w) { // a warp scans a channel's 32 groups
            const int ch = warp + 8 * w;
            float pa = s_a[ch][lane], pb = s_b[ch][lane];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
                if (lane >= o) {
                    pb = fmaf(pa, qb, pb);
                    pa *= qa;
                }
            }
            const float xa = __shfl_up_sync(0xffffffffu, pa, 1), xb = __shfl_up_sync(0xffffffffu, pb, 1);
            s_a[ch][lane] = lane == 0 ? 1.f : xa;
            s_b[ch][lane] = lane == 0 ? 0.f : xb;
            const float all_a = __shfl_sync(0xffffffffu, pa, 31), all_b = __shfl_sync(0xffffffffu, pb, 31);
            if (lane < n_ctas) {
                float *slot = cluster.map_shared_rank(&s_all[parity][rank][0][ch], unsigned(lane));
                slot[0] = all_a;
                slot[kChannels] = all_b;
            }
        }
        cluster.sync(); // (the other parity's slots have been read by every CTA before it arrives here)
        P o[kTokens];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float s = carry[e];
            for (int r = 0; r < n_ctas; ++r) {
                if (r == rank) {
                    s = carry[e];
                }
                carry[e] = fmaf(s_all[parity][r][0][lc + e], carry[e], s_all[parity][r][1][lc + e]);
            }
            s = fmaf(s_a[lc + e][group], s, s_b[lc + e][group]);
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                s = fmaf(keep[i][e], s, add[i][e]);
                const float gv = to_f32(g[i].v[e]);
                o[i].v[e] = from_f32<T>(s * gv * sigmoid<T>(gv));
            }
        }
        __syncthreads(); // s_a, s_b have been read
#pragma unroll
        for (int i = 0; i < kTokens; ++i) {
            if (holds && t0 + i < len) {
                *reinterpret_cast<P *>(out + int64_t(t0 + i) * a.out_stride) = o[i];
            }
        }
    }
    if (holds && rank == 0 && group == 0 && len > 0) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            state[e] = carry[e];
        }
    }
    cluster.sync(); // no CTA leaves while another may still write into its shared memory
}

bool vec4_fits(const MinGruArgs &a) {
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    return a.width % 4 == 0 && a.row_stride % 4 == 0 && a.z_at % 4 == 0 && a.x_at % 4 == 0 && a.g_at % 4 == 0 && a.out_stride % 4 == 0 &&
           a.slot_stride % 4 == 0 && aligned(a.proj) && aligned(a.bias_z) && aligned(a.bias_x) && aligned(a.state) &&
           reinterpret_cast<uintptr_t>(a.out) % 16 == 0;
}

template <typename F>
void dispatch(llaisysDataType_t dtype, F &&body) {
    switch (dtype) {
    case LLAISYS_DTYPE_F32:
        body(float{});
        break;
    case LLAISYS_DTYPE_F16:
        body(__half{});
        break;
    case LLAISYS_DTYPE_BF16:
        body(__nv_bfloat16{});
        break;
    default:
        EXCEPTION_UNSUPPORTED_DATATYPE(dtype);
    }
}

} // namespace

void min_gru_decode(stream_t stream, llaisysDataType_t dtype, const MinGruArgs &a) {
    if (a.n_seqs <= 0 || a.width <= 0) {
        return;
    }
    CHECK_ARGUMENT(a.n_seqs <= 65535, "minGRU: too many sequences for one launch");
    const bool wide = vec4_fits(a);
    const int pieces = wide ? a.width / 4 : a.width, block = pieces >= 1024 ? 128 : 64;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned((pieces + block - 1) / block), unsigned(a.n_seqs));
    cfg.blockDim = dim3(unsigned(block));
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, wide ? min_gru_decode_kernel<T, 4> : min_gru_decode_kernel<T, 1>, MinGruArgs(a)));
    });
    check_launch("min_gru_decode");
}

void min_gru_chunk(stream_t stream, llaisysDataType_t dtype, const MinGruArgs &a) {
    if (a.n_seqs <= 0 || a.width <= 0 || a.max_q_len <= 0) {
        return;
    }
    CHECK_ARGUMENT(a.n_seqs <= 65535, "minGRU: too many sequences for one launch");
    const bool wide = vec4_fits(a);
    const int channels = kLanes * (wide ? 4 : 1), slices = (a.width + channels - 1) / channels;
    // enough CTAs to fill the GPU twice, as far as the longest run has tiles for them
    int cluster = 1;
    while (cluster < kMaxCluster && int64_t(slices) * a.n_seqs * cluster < 2 * 148 && cluster * kTile < a.max_q_len) {
        cluster *= 2;
    }
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned(slices * cluster), unsigned(a.n_seqs));
    cfg.blockDim = dim3(kThreads);
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute attrs[2] = {};
    attrs[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attrs[0].val.programmaticStreamSerializationAllowed = 1;
    attrs[1].id = cudaLaunchAttributeClusterDimension;
    attrs[1].val.clusterDim.x = unsigned(cluster);
    attrs[1].val.clusterDim.y = 1;
    attrs[1].val.clusterDim.z = 1;
    cfg.attrs = attrs;
    cfg.numAttrs = 2;
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, wide ? min_gru_chunk_kernel<T, 4> : min_gru_chunk_kernel<T, 1>, MinGruArgs(a)));
    });
    check_launch("min_gru_chunk");
}

} // namespace llaisys::kernels
