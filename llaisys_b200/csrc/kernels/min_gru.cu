// minGRU (MinGruArgs): a gated recurrence per channel whose gates read the current token only, so a run of tokens is a chain of
// affine maps S -> a S + b that compose in any grouping.
//
// Roofline: HBM (three projections read, one activation written, per token and channel); six multi-function operations per element
// come close to it. Decode: a thread per (sequence, VEC channels). Runs are cut into segments of 128 tokens, a thread per segment and
// VEC channels: one launch composes the maps of every segment but a sequence's last into (a, b), a second starts each segment from
// the state that those before it leave and writes the outputs. Runs of one segment take the second launch only. State and gates are
// f32.
#include "gated_linear.cuh"
#include "kernels.hpp"
#include "mma_utils.cuh"

namespace llaisys::kernels {

namespace {

constexpr int kThreads = 128, kSegment = 128, kAhead = 8;

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

// Where the composed maps of a sequence lie in the scratch, [entry][width][2]. Only segments with one behind them have an entry, so
// these are whole, and sequences' entries do not overlap. A sequence's first entry holds (state before the run, state after it).
__device__ __forceinline__ float *first_entry(const MinGruArgs &a, int row0) { return a.scratch + int64_t(row0 / kSegment) * a.width * 2; }

// OUT false: composes; true: outputs.
template <typename T, int VEC, bool OUT>
__global__ void __launch_bounds__(kThreads) min_gru_segment_kernel(MinGruArgs a) {
    grid_dependency_wait();
    grid_launch_dependents();
    using P = Pieces<T, VEC>;
    using S = Pieces<float, VEC>;
    using M = Pieces<float, 2 * VEC>; // (a, b) of each channel
    const int seq = blockIdx.z, segment = blockIdx.y, c = (int(blockIdx.x) * kThreads + int(threadIdx.x)) * VEC;
    const int row0 = a.q_starts[seq], len = a.q_starts[seq + 1] - row0, t0 = segment * kSegment, n = min(kSegment, len - t0);
    const bool last = t0 + kSegment >= len;
    if (c >= a.width || n <= 0 || (!OUT && last)) {
        return;
    }
    S *state = reinterpret_cast<S *>(a.state + int64_t(a.seq_ids[seq]) * a.slot_stride + c);
    float *entry = first_entry(a, row0) + int64_t(c) * 2;
    const int64_t entry_stride = int64_t(a.width) * 2;
    const P bz = *reinterpret_cast<const P *>(static_cast<const T *>(a.bias_z) + c), bx = *reinterpret_cast<const P *>(static_cast<const T *>(a.bias_x) + c);
    S s{}, whole; // the state (OUT, and a first segment), or b of the segment so far; a of the segment so far
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        whole.v[e] = 1.f;
    }
    S before{};
    if (segment == 0 && (!OUT || last)) {
        if (a.kv_lens[seq] > len) {
            s = *state;
        }
        before = s;
    } else if (OUT) {
        const M first = *reinterpret_cast<const M *>(entry);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            s.v[e] = segment == 0 ? first.v[2 * e] : first.v[2 * e + 1];
        }
#pragma unroll 8
        for (int k = 1; k < segment; ++k) {
            const M m = *reinterpret_cast<const M *>(entry + k * entry_stride);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                s.v[e] = fmaf(m.v[2 * e], s.v[e], m.v[2 * e + 1]);
            }
        }
    }
    const T *row = static_cast<const T *>(a.proj) + int64_t(row0 + t0) * a.row_stride + c;
    T *out = static_cast<T *>(a.out) + int64_t(row0 + t0) * a.out_stride + c;
    struct Group {
        P z[kAhead], u[kAhead], g[OUT ? kAhead : 1];
    };
    auto load = [&](Group &x, int t) {
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            if (t + i < n) {
                const T *at = row + int64_t(t + i) * a.row_stride;
                x.z[i] = *reinterpret_cast<const P *>(at + a.z_at);
                x.u[i] = *reinterpret_cast<const P *>(at + a.x_at);
                if constexpr (OUT) {
                    x.g[i] = *reinterpret_cast<const P *>(at + a.g_at);
                }
            }
        }
    };
    Group now, next;
    load(now, 0);
    for (int t = 0; t < n; t += kAhead) {
        load(next, t + kAhead);
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            if (t + i < n) {
                P o;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    float keep, add;
                    affine<T>(to_f32(now.z[i].v[e]) + to_f32(bz.v[e]), to_f32(now.u[i].v[e]) + to_f32(bx.v[e]), keep, add);
                    s.v[e] = fmaf(keep, s.v[e], add);
                    if constexpr (OUT) {
                        const float gv = to_f32(now.g[i].v[e]);
                        o.v[e] = from_f32<T>(s.v[e] * gv * sigmoid<T>(gv));
                    } else {
                        whole.v[e] *= keep;
                    }
                }
                if constexpr (OUT) {
                    *reinterpret_cast<P *>(out + int64_t(t + i) * a.out_stride) = o;
                }
            }
        }
        now = next;
    }
    if constexpr (OUT) {
        if (last) {
            *state = s;
        }
    } else {
        M m;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            m.v[2 * e] = segment == 0 ? before.v[e] : whole.v[e];
            m.v[2 * e + 1] = s.v[e];
        }
        *reinterpret_cast<M *>(entry + segment * entry_stride) = m;
    }
}

bool vec_fits(const MinGruArgs &a, int vec) {
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    return a.width % vec == 0 && a.row_stride % vec == 0 && a.z_at % vec == 0 && a.x_at % vec == 0 && a.g_at % vec == 0 &&
           a.out_stride % vec == 0 && a.slot_stride % vec == 0 && aligned(a.proj) && aligned(a.bias_z) && aligned(a.bias_x) &&
           aligned(a.state) && aligned(a.out) && aligned(a.scratch);
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
    const bool wide = vec_fits(a, 4);
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
    const int segments = (a.max_q_len + kSegment - 1) / kSegment;
    CHECK_ARGUMENT(a.n_seqs <= 65535 && segments <= 65535, "minGRU: too many sequences or too long a run for one launch");
    CHECK_ARGUMENT(segments == 1 || (a.scratch != nullptr && a.scratch_floats >= min_gru_scratch_floats(size_t(a.n_rows), size_t(a.width))),
                   "minGRU: the scratch is too small");
    const bool wide = vec_fits(a, 2);
    const int block = kThreads * (wide ? 2 : 1);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned((a.width + block - 1) / block), unsigned(segments), unsigned(a.n_seqs));
    cfg.blockDim = dim3(kThreads);
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        if (segments > 1) {
            --cfg.gridDim.y; // (no sequence's last segment is composed)
            LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, wide ? min_gru_segment_kernel<T, 2, false> : min_gru_segment_kernel<T, 1, false>, MinGruArgs(a)));
            ++cfg.gridDim.y;
        }
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, wide ? min_gru_segment_kernel<T, 2, true> : min_gru_segment_kernel<T, 1, true>, MinGruArgs(a)));
    });
    check_launch("min_gru_chunk");
}

size_t min_gru_scratch_floats(size_t n_rows, size_t width) { return (n_rows / kSegment + 1) * width * 2; }

} // namespace llaisys::kernels
