// Operators of a decoder whose residual stream stays in f32 between layers: the embedding with its scale, the norm that
// turns stream rows into activations, the cast that feeds the stream to a projection, the squared-relu activation and the
// soft cap of the logits with the greedy choice behind it. All HBM-bound, one pass over their data.
#include "launch_utils.cuh"
#include "mma_utils.cuh"

namespace llaisys::kernels {

namespace {

template <typename T, int N>
struct alignas(sizeof(T) * N) Vec {
    T v[N];
};

template <typename T, int VEC>
__global__ void embed_scaled_kernel(float *__restrict__ x, T *__restrict__ copy, int64_t copy_stride,
                                    const int64_t *__restrict__ tokens, const T *__restrict__ w, float scale, int32_t d,
                                    int64_t vocab) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    int64_t tok = tokens[row];
    tok = tok < 0 || tok >= vocab ? 0 : tok; // validated on the host; never read out of range here
    const T *src = w + tok * d;
    for (int32_t i = int32_t(threadIdx.x) * VEC; i < d; i += int32_t(blockDim.x) * VEC) {
        const Vec<T, VEC> in = *reinterpret_cast<const Vec<T, VEC> *>(src + i);
        Vec<float, VEC> f;
        Vec<T, VEC> c;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            f.v[e] = to_f32(in.v[e]) * scale;
            c.v[e] = from_f32<T>(f.v[e]);
        }
        *reinterpret_cast<Vec<float, VEC> *>(x + row * d + i) = f;
        if (copy != nullptr) {
            *reinterpret_cast<Vec<T, VEC> *>(copy + row * copy_stride + i) = c;
        }
    }
}

template <typename T, int VEC>
__global__ void embed_pairs_kernel(float *__restrict__ x, const int64_t *__restrict__ tokens, const int64_t *__restrict__ prev,
                                   const T *__restrict__ w, const T *__restrict__ pairs, int64_t mul_prev, int64_t mul_cur,
                                   int64_t buckets, int32_t d, int64_t vocab) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    int64_t tok = tokens[row];
    tok = tok < 0 || tok >= vocab ? 0 : tok; // validated on the host; never read out of range here
    const int64_t before = prev[row];
    const int64_t bucket =
        before < 0 ? buckets : ((before % buckets) * mul_prev + (tok % buckets) * mul_cur) % buckets; // factors below buckets
    const T *src = w + tok * d, *pair = pairs + bucket * d;
    for (int32_t i = int32_t(threadIdx.x) * VEC; i < d; i += int32_t(blockDim.x) * VEC) {
        const Vec<T, VEC> a = *reinterpret_cast<const Vec<T, VEC> *>(src + i), b = *reinterpret_cast<const Vec<T, VEC> *>(pair + i);
        Vec<float, VEC> f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            f.v[e] = to_f32(a.v[e]) + to_f32(b.v[e]);
        }
        *reinterpret_cast<Vec<float, VEC> *>(x + row * d + i) = f;
    }
}

// One thread per column pair (sine, cosine); the angle is reduced in f64, so that far positions lose nothing.
template <typename T>
__global__ void embed_positions_kernel(float *__restrict__ x, const int64_t *__restrict__ tokens, const int32_t *__restrict__ positions,
                                       const double *__restrict__ freq, const T *__restrict__ w, int32_t d, int64_t vocab) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    int64_t tok = tokens[row];
    tok = tok < 0 || tok >= vocab ? 0 : tok; // validated on the host; never read out of range here
    const double pos = double(positions[row]);
    constexpr double kTurn = 6.283185307179586;
    for (int32_t i = int32_t(threadIdx.x); 2 * i < d; i += int32_t(blockDim.x)) {
        const double angle = pos * freq[i];
        float s, c;
        sincosf(float(fma(-kTurn, rint(angle * (1.0 / kTurn)), angle)), &s, &c);
        x[row * d + 2 * i] = to_f32(w[tok * d + 2 * i]) + s;
        if (2 * i + 1 < d) {
            x[row * d + 2 * i + 1] = to_f32(w[tok * d + 2 * i + 1]) + c;
        }
    }
}

template <typename T, int VEC>
__global__ void stream_cast_kernel(T *__restrict__ out, int64_t out_stride, const float *__restrict__ x, int32_t d) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    for (int32_t i = int32_t(threadIdx.x) * VEC; i < d; i += int32_t(blockDim.x) * VEC) {
        const Vec<float, VEC> in = *reinterpret_cast<const Vec<float, VEC> *>(x + row * d + i);
        Vec<T, VEC> c;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            c.v[e] = from_f32<T>(in.v[e]);
        }
        *reinterpret_cast<Vec<T, VEC> *>(out + row * out_stride + i) = c;
    }
}

// One CTA per row; the first PER_THREAD pieces of a thread stay in registers between the two passes, what a very long row
// has beyond them is read again.
template <typename T, int VEC, int PER_THREAD>
__global__ void stream_rms_norm_kernel(T *__restrict__ out, const float *__restrict__ x, const int64_t *__restrict__ row_index,
                                       const T *__restrict__ w, const float *__restrict__ gain, float eps, int32_t d, float offset) {
    grid_dependency_wait();
    grid_launch_dependents();
    using F = Vec<float, VEC>;
    const int64_t row = row_index != nullptr ? row_index[blockIdx.x] : int64_t(blockIdx.x);
    const float *src = x + row * d;
    const int32_t n_vec = d / VEC;
    F held[PER_THREAD];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * int32_t(blockDim.x);
        if (i < n_vec) {
            held[r] = *reinterpret_cast<const F *>(src + int64_t(i) * VEC);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                ss = fmaf(held[r].v[e], held[r].v[e], ss);
            }
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * int32_t(blockDim.x); i < n_vec; i += int32_t(blockDim.x)) {
        const F f = *reinterpret_cast<const F *>(src + int64_t(i) * VEC);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            ss = fmaf(f.v[e], f.v[e], ss);
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        ss += __shfl_xor_sync(0xffffffffu, ss, o);
    }
    __shared__ float s_part[32];
    if ((threadIdx.x & 31) == 0) {
        s_part[threadIdx.x >> 5] = ss;
    }
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < int(blockDim.x >> 5); ++i) {
        tot += s_part[i]; // every thread sums the few partials in the same order
    }
    const float inv = rsqrtf(tot / float(d) + eps) * (w == nullptr ? *gain : 1.f);
    T *dst = out + int64_t(blockIdx.x) * d;
    auto store = [&](int32_t i, const F &f) {
        Vec<T, VEC> o;
        if (w == nullptr) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                o.v[e] = from_f32<T>(f.v[e] * inv);
            }
        } else {
            const Vec<T, VEC> ww = *reinterpret_cast<const Vec<T, VEC> *>(w + int64_t(i) * VEC);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                o.v[e] = from_f32<T>(f.v[e] * inv * (offset + to_f32(ww.v[e])));
            }
        }
        *reinterpret_cast<Vec<T, VEC> *>(dst + int64_t(i) * VEC) = o;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * int32_t(blockDim.x);
        if (i < n_vec) {
            store(i, held[r]);
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * int32_t(blockDim.x); i < n_vec; i += int32_t(blockDim.x)) {
        store(i, *reinterpret_cast<const F *>(src + int64_t(i) * VEC));
    }
}

// Sum over the CTA, the same value for every thread (partials in the same order); `part` holds 32 floats.
__device__ __forceinline__ float block_sum(float v, float *part) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        v += __shfl_xor_sync(0xffffffffu, v, o);
    }
    __syncthreads(); // `part` may still be read by an earlier call
    if ((threadIdx.x & 31) == 0) {
        part[threadIdx.x >> 5] = v;
    }
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < int(blockDim.x >> 5); ++i) {
        tot += part[i];
    }
    return tot;
}

// One CTA per row, like stream_rms_norm_kernel: norms over the rows of a and (TWO) b, their sum into the stream, and the norm
// that follows. The first PER_THREAD pieces of a thread stay in registers.
template <typename T, int VEC, int PER_THREAD, bool TWO>
__global__ void stream_add_normed_kernel(float *__restrict__ x, const float *__restrict__ a, const T *__restrict__ wa,
                                         const float *__restrict__ b, const T *__restrict__ wb, float scale, float eps,
                                         T *__restrict__ h, const T *__restrict__ w, float offset, int32_t d, float branch_offset) {
    grid_dependency_wait();
    grid_launch_dependents();
    using F = Vec<float, VEC>;
    using W = Vec<T, VEC>;
    __shared__ float s_a[32], s_b[32];
    const int64_t row = int64_t(blockIdx.x) * d;
    const int32_t n_vec = d / VEC, step = int32_t(blockDim.x);
    F ha[PER_THREAD], hb[PER_THREAD];
    float sa = 0.f, sb = 0.f;
    auto square = [](const F &f, float &s) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            s = fmaf(f.v[e], f.v[e], s);
        }
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * step;
        if (i < n_vec) {
            ha[r] = reinterpret_cast<const F *>(a + row)[i];
            square(ha[r], sa);
            if constexpr (TWO) {
                hb[r] = reinterpret_cast<const F *>(b + row)[i];
                square(hb[r], sb);
            }
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        square(reinterpret_cast<const F *>(a + row)[i], sa);
        if constexpr (TWO) {
            square(reinterpret_cast<const F *>(b + row)[i], sb);
        }
    }
    const float ia = rsqrtf(block_sum(sa, s_a) / float(d) + eps) * scale;
    const float ib = TWO ? rsqrtf(block_sum(sb, s_b) / float(d) + eps) * scale : 0.f;
    float sx = 0.f;
    auto add = [&](int32_t i, const F &fa, const F &fb) {
        F f = reinterpret_cast<const F *>(x + row)[i];
        const W va = reinterpret_cast<const W *>(wa)[i];
        W vb;
        if constexpr (TWO) {
            vb = reinterpret_cast<const W *>(wb)[i];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float more = fa.v[e] * ia * (branch_offset + to_f32(va.v[e]));
            if constexpr (TWO) {
                more += fb.v[e] * ib * (branch_offset + to_f32(vb.v[e]));
            }
            f.v[e] += more;
        }
        square(f, sx);
        reinterpret_cast<F *>(x + row)[i] = f;
        return f;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * step;
        if (i < n_vec) {
            ha[r] = add(i, ha[r], hb[r]); // from here on the new stream
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        add(i, reinterpret_cast<const F *>(a + row)[i], TWO ? reinterpret_cast<const F *>(b + row)[i] : F{});
    }
    if (h == nullptr) {
        return;
    }
    const float inv = rsqrtf(block_sum(sx, s_a) / float(d) + eps);
    auto store = [&](int32_t i, const F &f) {
        const W ww = reinterpret_cast<const W *>(w)[i];
        W o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            o.v[e] = from_f32<T>(f.v[e] * inv * (offset + to_f32(ww.v[e])));
        }
        reinterpret_cast<W *>(h + row)[i] = o;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * step;
        if (i < n_vec) {
            store(i, ha[r]);
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        store(i, reinterpret_cast<const F *>(x + row)[i]); // (written by this thread)
    }
}

// z / 2 (1 + tanh(y)) = z / (1 + exp(-2 y)), y = sqrt(2 / pi) (z + 0.044715 z^3)
template <typename T>
__device__ __forceinline__ float gelu(float z) {
    const float y2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
    if constexpr (sizeof(T) == 4) {
        return z / (1.f + expf(-y2));
    } else {
        return __fdividef(z, 1.f + __expf(fminf(-y2, 80.f)));
    }
}

template <typename T, int VEC>
__global__ void gelu_tanh_kernel(T *__restrict__ out, int64_t out_stride, const T *__restrict__ in, int64_t in_stride, int32_t n_vec) {
    grid_dependency_wait();
    grid_launch_dependents();
    using P = Vec<T, VEC>;
    const P *src = reinterpret_cast<const P *>(in + int64_t(blockIdx.y) * in_stride);
    P *dst = reinterpret_cast<P *>(out + int64_t(blockIdx.y) * out_stride);
    for (int32_t i = int32_t(blockIdx.x) * int32_t(blockDim.x) + int32_t(threadIdx.x); i < n_vec; i += int32_t(gridDim.x) * int32_t(blockDim.x)) {
        P p = src[i];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            p.v[e] = from_f32<T>(gelu<T>(to_f32(p.v[e])));
        }
        dst[i] = p;
    }
}

__global__ void rotary_table_kernel(float2 *__restrict__ table, const int32_t *__restrict__ positions, const float *__restrict__ freq,
                                    int32_t half, int64_t total) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t at = int64_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (at < total) {
        const int64_t row = at / half;
        float s, c;
        sincosf(float(positions[row]) * freq[at - row * half], &s, &c);
        table[at] = make_float2(c, s);
    }
}

// The angle in f64, reduced there, so that far positions lose nothing.
__global__ void rotary_table_wide_kernel(float2 *__restrict__ table, const int32_t *__restrict__ positions, const double *__restrict__ freq,
                                         int32_t half, int64_t total) {
    grid_dependency_wait();
    grid_launch_dependents();
    constexpr double kTurn = 6.283185307179586;
    const int64_t at = int64_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (at < total) {
        const int64_t row = at / half;
        const double angle = double(positions[row]) * freq[at - row * half];
        float s, c;
        sincosf(float(fma(-kTurn, rint(angle * (1.0 / kTurn)), angle)), &s, &c);
        table[at] = make_float2(c, s);
    }
}

// One thread per pair of a head
template <typename T>
__global__ void rotate_pairs_kernel(T *out, int64_t out_dim, int64_t out_at, const T *q, int32_t dim, int32_t half,
                                    const float2 *__restrict__ table, int32_t nh, int64_t total) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t at = int64_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (at >= total) {
        return;
    }
    const int64_t head = at / half, row = head / nh; // head: of all rows
    const int32_t i = int32_t(at - head * half);
    const T *src = q + head * (dim + 2 * half) + dim + 2 * i;
    const float u = to_f32(src[0]), v = to_f32(src[1]);
    const float2 t = table[row * half + i];
    T *dst = out + head * out_dim + out_at + 2 * i;
    dst[0] = from_f32<T>(u * t.x - v * t.y);
    dst[1] = from_f32<T>(v * t.x + u * t.y);
}

template <typename T, int VEC>
__global__ void relu_squared_kernel(T *__restrict__ v, size_t n_vec) {
    grid_dependency_wait();
    grid_launch_dependents();
    using P = Vec<T, VEC>;
    const size_t stride = size_t(gridDim.x) * blockDim.x;
    for (size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x; i < n_vec; i += stride) {
        P p = reinterpret_cast<const P *>(v)[i];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float f = fmaxf(to_f32(p.v[e]), 0.f);
            p.v[e] = from_f32<T>(f * f);
        }
        reinterpret_cast<P *>(v)[i] = p;
    }
}

// The split argmax of ops_misc.cu with the soft cap applied on the way: a row's CTAs fold (value, index) into one 64-bit
// key, the last of them to arrive writes the index and leaves key and counter zero.
__global__ void softcap_argmax_kernel(float *__restrict__ logits, float cap, int64_t *__restrict__ idx_out, size_t n,
                                      unsigned long long *__restrict__ keys, unsigned *__restrict__ counters) {
    const size_t row_i = blockIdx.y;
    float *row = logits + row_i * n;
    const size_t chunk = (n + gridDim.x - 1) / gridDim.x;
    const size_t lo = size_t(blockIdx.x) * chunk, hi = lo + chunk < n ? lo + chunk : n;
    unsigned long long best = 0;
    for (size_t i = lo + threadIdx.x; i < hi; i += blockDim.x) {
        float v = row[i];
        if (cap > 0.f) {
            v = cap * tanhf(v / cap);
            row[i] = v;
        }
        if (v == v) { // NaN never wins
            const unsigned b = __float_as_uint(v);
            const unsigned ord = (b & 0x80000000u) ? ~b : (b | 0x80000000u);
            const unsigned long long key =
                (static_cast<unsigned long long>(ord) << 32) | static_cast<unsigned long long>(0xffffffffu - unsigned(i));
            best = key > best ? key : best;
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
        best = other > best ? other : best;
    }
    __shared__ unsigned long long s_best[32];
    if ((threadIdx.x & 31) == 0) {
        s_best[threadIdx.x >> 5] = best;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int i = 1; i < int(blockDim.x >> 5); ++i) {
            best = s_best[i] > best ? s_best[i] : best;
        }
        atomicMax(keys + row_i, best);
        __threadfence();
        if (atomicAdd(counters + row_i, 1u) == gridDim.x - 1) {
            __threadfence();
            const unsigned long long win = atomicExch(keys + row_i, 0ull);
            counters[row_i] = 0u;
            idx_out[row_i] = win == 0ull ? 0 : int64_t(0xffffffffu - unsigned(win & 0xffffffffull));
        }
    }
}

unsigned block_for(size_t n_vec, size_t per_thread) {
    const size_t want = (n_vec + per_thread - 1) / per_thread;
    const size_t block = (want + 31) / 32 * 32;
    return unsigned(block < 64 ? 64 : (block > 1024 ? 1024 : block));
}
} // namespace

void embed_scaled(stream_t stream, llaisysDataType_t dtype, float *x, void *copy, int64_t copy_stride, const int64_t *tokens,
                  const void *w, float scale, size_t rows, size_t d, size_t vocab) {
    if (rows == 0 || d == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && copy_stride % 4 == 0 && aligned16(x) && aligned16(w) && (copy == nullptr || aligned16(copy));
        auto kernel = wide ? embed_scaled_kernel<T, 4> : embed_scaled_kernel<T, 1>;
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, x, static_cast<T *>(copy), copy_stride,
                            tokens, static_cast<const T *>(w), scale, int32_t(d), int64_t(vocab));
    });
    check_launch("embed_scaled");
}

void embed_pairs(stream_t stream, llaisysDataType_t dtype, float *x, const int64_t *tokens, const int64_t *prev, const void *w,
                 const void *pairs, int64_t mul_prev, int64_t mul_cur, int64_t buckets, size_t rows, size_t d, size_t vocab) {
    if (rows == 0 || d == 0) {
        return;
    }
    CHECK_ARGUMENT(buckets > 0 && buckets < (int64_t(1) << 31), "embed_pairs: 1 to 2^31 - 1 buckets");
    auto s = static_cast<cudaStream_t>(stream);
    auto mod = [&](int64_t v) { return (v % buckets + buckets) % buckets; };
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(pairs);
        auto kernel = wide ? embed_pairs_kernel<T, 4> : embed_pairs_kernel<T, 1>;
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, x, tokens, prev, static_cast<const T *>(w),
                            static_cast<const T *>(pairs), mod(mul_prev), mod(mul_cur), buckets, int32_t(d), int64_t(vocab));
    });
    check_launch("embed_pairs");
}

void embed_positions(stream_t stream, llaisysDataType_t dtype, float *x, const int64_t *tokens, const int32_t *positions,
                     const double *freq, const void *w, size_t rows, size_t d, size_t vocab) {
    if (rows == 0 || d == 0) {
        return;
    }
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        launch_programmatic(embed_positions_kernel<T>, dim3(unsigned(rows)), block_for((d + 1) / 2, 2), static_cast<cudaStream_t>(stream), x,
                            tokens, positions, freq, static_cast<const T *>(w), int32_t(d), int64_t(vocab));
    });
    check_launch("embed_positions");
}

void stream_cast(stream_t stream, llaisysDataType_t dtype, void *out, int64_t out_stride, const float *x, size_t rows, size_t d) {
    if (rows == 0 || d == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && out_stride % 4 == 0 && aligned16(x) && aligned16(out);
        auto kernel = wide ? stream_cast_kernel<T, 4> : stream_cast_kernel<T, 1>;
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, static_cast<T *>(out), out_stride, x,
                            int32_t(d));
    });
    check_launch("stream_cast");
}

void stream_rms_norm(stream_t stream, llaisysDataType_t dtype, void *out, const float *x, const int64_t *row_index,
                     const void *w, float eps, size_t rows, size_t d, float offset) {
    if (rows == 0 || d == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && aligned16(x) && aligned16(out) && aligned16(w);
        auto kernel = wide ? stream_rms_norm_kernel<T, 4, 4> : stream_rms_norm_kernel<T, 1, 4>;
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, static_cast<T *>(out), x, row_index,
                            static_cast<const T *>(w), nullptr, eps, int32_t(d), offset);
    });
    check_launch("stream_rms_norm");
}

void stream_rms_norm_gain(stream_t stream, llaisysDataType_t dtype, void *out, const float *x, const int64_t *row_index,
                          const float *gain, float eps, size_t rows, size_t d) {
    if (rows == 0 || d == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && aligned16(x) && aligned16(out);
        auto kernel = wide ? stream_rms_norm_kernel<T, 4, 4> : stream_rms_norm_kernel<T, 1, 4>;
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, static_cast<T *>(out), x, row_index,
                            nullptr, gain, eps, int32_t(d), 0.f);
    });
    check_launch("stream_rms_norm_gain");
}

void stream_add_normed(stream_t stream, llaisysDataType_t dtype, float *x, const float *a, const void *wa, const float *b,
                       const void *wb, float scale, float eps, void *h, const void *w, float offset, size_t rows, size_t d,
                       float branch_offset) {
    if (rows == 0 || d == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = d % 4 == 0 && aligned16(x) && aligned16(a) && aligned16(b) && aligned16(wa) && aligned16(wb) && aligned16(h) &&
                          aligned16(w);
        auto kernel = b != nullptr ? (wide ? stream_add_normed_kernel<T, 4, 3, true> : stream_add_normed_kernel<T, 1, 3, true>)
                                   : (wide ? stream_add_normed_kernel<T, 4, 4, false> : stream_add_normed_kernel<T, 1, 4, false>);
        launch_programmatic(kernel, dim3(unsigned(rows)), block_for(wide ? d / 4 : d, 2), s, x, a, static_cast<const T *>(wa), b,
                            static_cast<const T *>(wb), scale, eps, static_cast<T *>(h), static_cast<const T *>(w), offset, int32_t(d),
                            branch_offset);
    });
    check_launch("stream_add_normed");
}

void gelu_tanh(stream_t stream, llaisysDataType_t dtype, void *out, int64_t out_stride, const void *in, int64_t in_stride,
               size_t rows, size_t n) {
    if (rows == 0 || n == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        constexpr int kVec = 16 / int(sizeof(T));
        const bool wide = n % kVec == 0 && out_stride % kVec == 0 && in_stride % kVec == 0 && aligned16(out) && aligned16(in);
        const size_t n_vec = wide ? n / kVec : n;
        auto kernel = wide ? gelu_tanh_kernel<T, kVec> : gelu_tanh_kernel<T, 1>;
        constexpr size_t kRows = 65535;
        for (size_t r = 0; r < rows; r += kRows) {
            const size_t m = rows - r < kRows ? rows - r : kRows;
            launch_programmatic(kernel, dim3(unsigned((n_vec + 511) / 512), unsigned(m)), 256u, s,
                                static_cast<T *>(out) + int64_t(r) * out_stride, out_stride,
                                static_cast<const T *>(in) + int64_t(r) * in_stride, in_stride, int32_t(n_vec));
        }
    });
    check_launch("gelu_tanh");
}

void rotary_table(stream_t stream, float *table, const int32_t *positions, const float *freq, size_t rows, size_t half) {
    if (rows == 0 || half == 0) {
        return;
    }
    const int64_t total = int64_t(rows) * int64_t(half);
    launch_programmatic(rotary_table_kernel, dim3(unsigned((total + 255) / 256)), 256u, static_cast<cudaStream_t>(stream),
                        reinterpret_cast<float2 *>(table), positions, freq, int32_t(half), total);
    check_launch("rotary_table");
}

void rotary_table(stream_t stream, float *table, const int32_t *positions, const double *freq, size_t rows, size_t half) {
    if (rows == 0 || half == 0) {
        return;
    }
    const int64_t total = int64_t(rows) * int64_t(half);
    launch_programmatic(rotary_table_wide_kernel, dim3(unsigned((total + 255) / 256)), 256u, static_cast<cudaStream_t>(stream),
                        reinterpret_cast<float2 *>(table), positions, freq, int32_t(half), total);
    check_launch("rotary_table");
}

void rotate_pairs(stream_t stream, llaisysDataType_t dtype, void *out, size_t out_dim, size_t out_at, const void *q, size_t dim, size_t rot_dims,
                  const float *rot_table, size_t n_rows, size_t nh) {
    const int64_t half = int64_t(rot_dims / 2), total = int64_t(n_rows) * int64_t(nh) * half;
    if (total == 0) {
        return;
    }
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        launch_programmatic(rotate_pairs_kernel<T>, dim3(unsigned((total + 255) / 256)), 256u, static_cast<cudaStream_t>(stream),
                            static_cast<T *>(out), int64_t(out_dim), int64_t(out_at), static_cast<const T *>(q), int32_t(dim), int32_t(half),
                            reinterpret_cast<const float2 *>(rot_table), int32_t(nh), total);
    });
    check_launch("rotate_pairs");
}

void relu_squared(stream_t stream, llaisysDataType_t dtype, void *v, size_t n) {
    if (n == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        constexpr int kVec = 16 / int(sizeof(T));
        const bool wide = n % kVec == 0 && aligned16(v);
        const size_t n_vec = wide ? n / kVec : n;
        const size_t want = (n_vec + 255) / 256, cap = 148 * 16;
        auto kernel = wide ? relu_squared_kernel<T, kVec> : relu_squared_kernel<T, 1>;
        launch_programmatic(kernel, dim3(unsigned(want < cap ? want : cap)), 256u, s, static_cast<T *>(v), n_vec);
    });
    check_launch("relu_squared");
}

void softcap_argmax(stream_t stream, float *logits, float cap, int64_t *idx_out, size_t rows, size_t n, void *scratch) {
    if (rows == 0 || n == 0) {
        return;
    }
    CHECK_ARGUMENT(n < 0xffffffffull && rows <= 65535, "softcap_argmax: rows too many or too long");
    auto s = static_cast<cudaStream_t>(stream);
    auto *keys = static_cast<unsigned long long *>(scratch);
    auto *counters = reinterpret_cast<unsigned *>(keys + rows);
    size_t splits = (n + 4095) / 4096;
    const size_t cap_splits = (148 * 8 + rows - 1) / rows;
    splits = splits > cap_splits ? cap_splits : splits;
    const dim3 grid{static_cast<unsigned>(splits), static_cast<unsigned>(rows), 1u};
    softcap_argmax_kernel<<<grid, 256, 0, s>>>(logits, cap, idx_out, n, keys, counters);
    check_launch("softcap_argmax");
}

} // namespace llaisys::kernels
