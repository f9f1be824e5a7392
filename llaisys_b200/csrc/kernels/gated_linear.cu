// Gated linear attention with a decay per key channel (see GatedLinearArgs). Two forms of the same recurrence:
//   * decode: one token per sequence, everything from the projection row to the gated, normed output in one launch. A CTA
//     owns one (sequence, head): it reads that head's f32 state once, updates it and writes it back -- HBM-bound,
//     2 * dk * dv * 4 bytes per head.
//     In a batch of runs the same kernel serves the sequences that bring a single token.
//   * recurrent: runs of tokens, one after the other in f32 with the state in registers. A CTA owns 16 value columns of one
//     (sequence, head). Exact in the order of the definition.
//     (The third form, runs on the tensor cores, is gated_linear_chunk.cu; bf16 models run that one.)
// All arithmetic of the recurrence, the decay and the norm is f32.
#include "device_utils.cuh"
#include "gated_linear.cuh"
#include "kernels.hpp"
#include "mma_utils.cuh"

#include <utility>

namespace llaisys::kernels {

namespace {

constexpr int kDecodeThreads = 256;

template <typename T, int VEC>
__global__ void __launch_bounds__(kDecodeThreads) gated_linear_decode_kernel(GatedLinearArgs a, int col_groups) {
    extern __shared__ float smem[];
    float *s_z = smem;                // [rank]
    float *s_a = s_z + a.rank;        // [dk] decay
    float *s_k = s_a + a.dk;          // [dk]
    float *s_q = s_k + a.dk;          // [dk]
    float *s_o = s_q + a.dk;          // [row groups][dv]
    __shared__ float s_red[32];

    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int tid = int(threadIdx.x);
    const int64_t slot = a.seq_ids[i];
    const bool fresh = a.kv_lens[i] == 1;
    const int row_i = a.q_starts != nullptr ? a.q_starts[i] : i;
    grid_dependency_wait();
    grid_launch_dependents();
    if (a.q_starts != nullptr && a.q_starts[i + 1] - row_i != 1) {
        return; // a run of tokens (or none): another kernel's
    }

    float *state = a.state + slot * a.slot_stride + int64_t(head) * a.dk * a.dv;
    const T *row = static_cast<const T *>(a.proj) + int64_t(row_i) * a.row_stride;
    for (int r = tid; r < a.rank; r += kDecodeThreads) {
        s_z[r] = to_f32(row[a.z_at + r]);
    }
    for (int c = tid; c < a.dk; c += kDecodeThreads) {
        s_k[c] = to_f32(row[a.k_at + int64_t(head) * a.dk + c]);
        s_q[c] = to_f32(row[a.q_at + int64_t(head) * a.dk + c]) * a.q_scale;
    }
    __syncthreads();
    for (int c = tid; c < a.dk; c += kDecodeThreads) {
        s_a[c] = expf(decay_log<T>(a, s_z, head, c));
    }
    __syncthreads();

    // thread = (VEC columns, every row_groups-th row)
    using F = Pieces<float, VEC>;
    const int row_groups = kDecodeThreads / col_groups;
    const int cg = tid % col_groups, rg = tid / col_groups;
    for (int c0 = cg * VEC; c0 < a.dv; c0 += col_groups * VEC) {
        float v[VEC], o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            v[e] = to_f32(row[a.v_at + int64_t(head) * a.dv + c0 + e]);
            o[e] = 0.f;
        }
        constexpr int kBatch = 8; // state rows in flight per thread
        for (int r0 = rg; r0 < a.dk; r0 += row_groups * kBatch) {
            F s[kBatch];
#pragma unroll
            for (int u = 0; u < kBatch; ++u) {
                const int r = r0 + u * row_groups;
                if (r < a.dk && !fresh) {
                    s[u] = *reinterpret_cast<const F *>(state + int64_t(r) * a.dv + c0);
                } else {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[u].v[e] = 0.f;
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < kBatch; ++u) {
                const int r = r0 + u * row_groups;
                if (r < a.dk) {
                    const float ar = s_a[r], kr = s_k[r], qr = s_q[r];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[u].v[e] = fmaf(ar, s[u].v[e], kr * v[e]);
                        o[e] = fmaf(qr, s[u].v[e], o[e]);
                    }
                    *reinterpret_cast<F *>(state + int64_t(r) * a.dv + c0) = s[u];
                }
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            s_o[rg * a.dv + c0 + e] = o[e];
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < a.dv; c += kDecodeThreads) {
        float o = 0.f;
        for (int g = 0; g < row_groups; ++g) {
            o += s_o[g * a.dv + c];
        }
        s_o[c] = o; // (column c is read by this thread only)
        ss = fmaf(o, o, ss);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        ss += __shfl_xor_sync(0xffffffffu, ss, o);
    }
    if ((tid & 31) == 0) {
        s_red[tid >> 5] = ss;
    }
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < kDecodeThreads / 32; ++w) {
        tot += s_red[w];
    }
    const float inv = rsqrtf(tot / float(a.dv) + a.eps) * a.out_scale;
    T *out = static_cast<T *>(a.out) + int64_t(row_i) * a.out_stride + int64_t(head) * a.dv;
    const T *w = static_cast<const T *>(a.norm_w);
    for (int c = tid; c < a.dv; c += kDecodeThreads) {
        const float g = to_f32(row[a.g_at + int64_t(head) * a.dv + c]);
        out[c] = from_f32<T>(s_o[c] * inv * to_f32(w[c]) * silu(g));
    }
}

// decay[row, h * dk + c] = a_t of the row (not its logarithm)
template <typename T>
__global__ void gated_linear_decay_kernel(GatedLinearArgs a) {
    extern __shared__ float s_zrow[];
    const int64_t row = blockIdx.x;
    const T *proj = static_cast<const T *>(a.proj) + row * a.row_stride;
    for (int r = int(threadIdx.x); r < a.rank; r += int(blockDim.x)) {
        s_zrow[r] = to_f32(proj[a.z_at + r]);
    }
    __syncthreads();
    const int n = a.heads * a.dk;
    for (int c = int(threadIdx.x); c < n; c += int(blockDim.x)) {
        a.decay[row * n + c] = expf(decay_log<T>(a, s_zrow, 0, c));
    }
}

constexpr int kRecCols = 16, kRecRowGroups = 8, kRecThreads = kRecCols * kRecRowGroups;

// NR state rows per thread: row(j) = 4 * g + 32 * (j / 4) + j % 4 for row group g.
template <typename T, int NR>
__global__ void __launch_bounds__(kRecThreads) gated_linear_recurrent_kernel(GatedLinearArgs a) {
    constexpr int kRows = kRecRowGroups * NR;
    constexpr int kTok = NR > 32 ? 4 : 8; // tokens staged at a time
    __shared__ __align__(16) float s_q[kTok][kRows], s_k[kTok][kRows], s_a[kTok][kRows];
    __shared__ float s_v[kTok][kRecCols];
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int tid = int(threadIdx.x), g = tid % kRecRowGroups, cl = tid / kRecRowGroups;
    const int col = int(blockIdx.y) * kRecCols + cl;
    const int row0 = a.q_starts[i], row1 = a.q_starts[i + 1];
    const bool fresh = a.kv_lens[i] == row1 - row0;
    float *state = a.state + int64_t(a.seq_ids[i]) * a.slot_stride + int64_t(head) * a.dk * a.dv;
    auto row_of = [&](int j) { return 4 * g + 32 * (j / 4) + j % 4; };
    float s[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        s[j] = !fresh && row_of(j) < a.dk && col < a.dv ? state[int64_t(row_of(j)) * a.dv + col] : 0.f;
    }
    const T *proj = static_cast<const T *>(a.proj);
    for (int t0 = row0; t0 < row1; t0 += kTok) {
        __syncthreads();
        for (int u = tid; u < kTok * kRows; u += kRecThreads) {
            const int t = u / kRows, r = u - t * kRows;
            const bool in = t0 + t < row1 && r < a.dk;
            const int64_t at = int64_t(t0 + t) * a.row_stride + int64_t(head) * a.dk + r;
            s_q[t][r] = in ? to_f32(proj[at + a.q_at]) * a.q_scale : 0.f;
            s_k[t][r] = in ? to_f32(proj[at + a.k_at]) : 0.f;
            s_a[t][r] = in ? a.decay[int64_t(t0 + t) * a.heads * a.dk + int64_t(head) * a.dk + r] : 1.f;
        }
        for (int u = tid; u < kTok * kRecCols; u += kRecThreads) {
            const int t = u / kRecCols, c = u - t * kRecCols + int(blockIdx.y) * kRecCols;
            s_v[t][u % kRecCols] =
                t0 + t < row1 && c < a.dv ? to_f32(proj[int64_t(t0 + t) * a.row_stride + a.v_at + int64_t(head) * a.dv + c]) : 0.f;
        }
        __syncthreads();
        const int n = min(kTok, row1 - t0);
        for (int t = 0; t < n; ++t) {
            const float v = s_v[t][cl];
            float o = 0.f;
#pragma unroll
            for (int j = 0; j < NR; j += 4) {
                const float4 q4 = *reinterpret_cast<const float4 *>(&s_q[t][4 * g + 8 * j]);
                const float4 k4 = *reinterpret_cast<const float4 *>(&s_k[t][4 * g + 8 * j]);
                const float4 a4 = *reinterpret_cast<const float4 *>(&s_a[t][4 * g + 8 * j]);
                s[j] = fmaf(a4.x, s[j], k4.x * v);
                s[j + 1] = fmaf(a4.y, s[j + 1], k4.y * v);
                s[j + 2] = fmaf(a4.z, s[j + 2], k4.z * v);
                s[j + 3] = fmaf(a4.w, s[j + 3], k4.w * v);
                o = fmaf(q4.x, s[j], o);
                o = fmaf(q4.y, s[j + 1], o);
                o = fmaf(q4.z, s[j + 2], o);
                o = fmaf(q4.w, s[j + 3], o);
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            o += __shfl_xor_sync(0xffffffffu, o, 4);
            if (g == 0 && col < a.dv) {
                a.raw[int64_t(t0 + t) * a.heads * a.dv + int64_t(head) * a.dv + col] = o;
            }
        }
    }
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        if (row_of(j) < a.dk && col < a.dv) {
            state[int64_t(row_of(j)) * a.dv + col] = s[j];
        }
    }
}

// out = out_scale * rms_norm(raw) * silu(g): one warp per (row, head)
template <typename T>
__global__ void gated_linear_out_kernel(GatedLinearArgs a) {
    const int64_t item = int64_t(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = int(threadIdx.x) & 31;
    if (item >= int64_t(a.n_rows) * a.heads) {
        return;
    }
    const int64_t row = item / a.heads;
    const int head = int(item - row * a.heads);
    const float *o = a.raw + item * a.dv;
    float ss = 0.f;
    for (int c = lane; c < a.dv; c += 32) {
        ss = fmaf(o[c], o[c], ss);
    }
#pragma unroll
    for (int u = 16; u > 0; u >>= 1) {
        ss += __shfl_xor_sync(0xffffffffu, ss, u);
    }
    const float inv = rsqrtf(ss / float(a.dv) + a.eps) * a.out_scale;
    const T *g = static_cast<const T *>(a.proj) + row * a.row_stride + a.g_at + int64_t(head) * a.dv;
    const T *w = static_cast<const T *>(a.norm_w);
    T *out = static_cast<T *>(a.out) + row * a.out_stride + int64_t(head) * a.dv;
    for (int c = lane; c < a.dv; c += 32) {
        out[c] = from_f32<T>(o[c] * inv * to_f32(w[c]) * silu(to_f32(g[c])));
    }
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

template <typename T>
void recurrent(cudaStream_t s, const GatedLinearArgs &a) {
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads), unsigned((a.dv + kRecCols - 1) / kRecCols));
    const int nr = (a.dk + kRecRowGroups - 1) / kRecRowGroups;
    if (nr <= 4) {
        gated_linear_recurrent_kernel<T, 4><<<grid, kRecThreads, 0, s>>>(a);
    } else if (nr <= 8) {
        gated_linear_recurrent_kernel<T, 8><<<grid, kRecThreads, 0, s>>>(a);
    } else if (nr <= 16) {
        gated_linear_recurrent_kernel<T, 16><<<grid, kRecThreads, 0, s>>>(a);
    } else if (nr <= 32) {
        gated_linear_recurrent_kernel<T, 32><<<grid, kRecThreads, 0, s>>>(a);
    } else {
        gated_linear_recurrent_kernel<T, 64><<<grid, kRecThreads, 0, s>>>(a);
    }
}

void check_args(const GatedLinearArgs &a) {
    CHECK_ARGUMENT(a.heads > 0 && a.dk > 0 && a.dk <= 512 && a.dv > 0 && a.dv <= 2048 && a.rank > 0 && a.rank <= 2048,
                   "gated linear attention: key size at most 512, value size and rank at most 2048");
    CHECK_ARGUMENT(int64_t(a.n_seqs) * a.heads <= 0x7fffffff, "gated linear attention: too many (sequence, head) pairs");
}

void single_tokens(stream_t stream, llaisysDataType_t dtype, const GatedLinearArgs &a) {
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = a.dv % 4 == 0 && a.slot_stride % 4 == 0;
        const int groups = wide ? a.dv / 4 : a.dv;
        int col_groups = 1;
        while (col_groups < groups && col_groups < kDecodeThreads) {
            col_groups *= 2;
        }
        const size_t smem = (size_t(a.rank) + 3 * size_t(a.dk) + size_t(kDecodeThreads / col_groups) * size_t(a.dv)) * sizeof(float);
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3(unsigned(a.n_seqs) * unsigned(a.heads));
        cfg.blockDim = dim3(kDecodeThreads);
        cfg.dynamicSmemBytes = smem; // at most 2048 + 3 * 512 + 2048 floats
        cfg.stream = s;
        cudaLaunchAttribute attr{};
        attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr.val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = &attr;
        cfg.numAttrs = 1;
        auto kernel = wide ? gated_linear_decode_kernel<T, 4> : gated_linear_decode_kernel<T, 1>;
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, GatedLinearArgs(a), int(col_groups)));
    });
}

} // namespace

void gated_linear_decode(stream_t stream, llaisysDataType_t dtype, const GatedLinearArgs &args) {
    if (args.n_seqs == 0) {
        return;
    }
    check_args(args);
    GatedLinearArgs a = args;
    a.q_starts = nullptr; // row i is sequence i's
    single_tokens(stream, dtype, a);
    check_launch("gated_linear_decode");
}

void gated_linear_chunk(stream_t stream, llaisysDataType_t dtype, const GatedLinearArgs &a) {
    if (a.n_seqs == 0 || a.n_rows == 0) {
        return;
    }
    check_args(a);
    CHECK_ARGUMENT(a.raw != nullptr && a.decay != nullptr, "gated linear attention: scratch missing");
    auto s = static_cast<cudaStream_t>(stream);
    auto finish = [&](auto tag) {
        using T = decltype(tag);
        const int64_t items = int64_t(a.n_rows) * a.heads;
        gated_linear_out_kernel<T><<<unsigned((items + 7) / 8), 256, 0, s>>>(a);
    };
    if (gated_linear_tiles_apply(dtype, a)) {
        gated_linear_tiles(stream, a);
        if (a.dv > 128) {
            finish(__nv_bfloat16{}); // (rows of single tokens hold nothing yet: the next kernel writes them)
        }
        single_tokens(stream, dtype, a);
    } else {
        dispatch(dtype, [&](auto tag) {
            using T = decltype(tag);
            gated_linear_decay_kernel<T><<<unsigned(a.n_rows), 128, size_t(a.rank) * sizeof(float), s>>>(a);
            recurrent<T>(s, a);
            finish(tag);
        });
    }
    check_launch("gated_linear_chunk");
}

} // namespace llaisys::kernels
