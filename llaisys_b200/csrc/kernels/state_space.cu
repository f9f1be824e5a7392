// Mamba-2 state space (see StateSpaceArgs): what precedes and follows the recurrence, its two plain forms, and the choice of form.
//   * decode: one token per sequence. A CTA owns one (sequence, head): short convolutions, step size, state and read-out. The state
//     is read and written once -- HBM-bound, 2 * dk * dv * 4 bytes per head. In a batch with runs on the tensor cores the same kernel
//     serves the sequences that bring a single token.
//   * prepare: for runs, convolutions + silu (rounded to the model dtype) and step sizes of all rows.
//   * recurrent: runs of tokens one after the other in f32. A CTA owns up to 32 value columns of one (sequence, head). Exact in the
//     order of the definition.
//   * finish: gate and norm of the concatenated heads, in parts.
//     (Runs on the tensor cores are state_space_chunk.cu; bf16 models run those.)
#include "launch_utils.cuh"
#include "mma_utils.cuh"
#include "state_space.cuh"

#include <algorithm>

namespace llaisys::kernels {

namespace {

constexpr int kDecodeThreads = 128;
constexpr int kConvRows = 8, kConvRowsAny = 4; // rows of a thread of the preparing kernel: with a known number of taps, without

template <int VEC>
struct alignas(4 * VEC) Floats {
    float v[VEC];
};

// thread = (VEC columns, every row_groups-th of the dk rows)
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(kDecodeThreads, 10) state_decode_kernel(StateSpaceArgs a, int64_t y_stride, int col_groups) {
    using F = Floats<VEC>;
    extern __shared__ __align__(16) float smem[];
    auto up4 = [](int n) { return (n + 3) / 4 * 4; };
    float *s_x = smem, *s_b = s_x + up4(a.dv), *s_c = s_b + up4(a.dk), *s_part = s_c + up4(a.dk); // s_part [row groups][columns of a pass]
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads, tid = int(threadIdx.x);
    const int64_t slot = a.seq_ids[i];
    const int row = a.q_starts != nullptr ? a.q_starts[i] : i, n_new = a.q_starts != nullptr ? a.q_starts[i + 1] - row : 1;
    if (n_new != 1) {
        grid_dependency_wait();
        grid_launch_dependents();
        return;
    }
    const int pos = a.kv_lens[i] - 1, share = a.heads / a.groups, group = head / share, channels = a.channels();
    const bool fresh = pos == 0;
    // Everything that no kernel of this step writes is fetched before the wait for the previous kernel.
    float *state = a.state + slot * a.slot_stride + int64_t(head) * a.dk * a.dv;
    const int row_groups = kDecodeThreads / col_groups, cg = tid % col_groups, rg = tid / col_groups;
    const bool works = rg < row_groups;
    F s[NR];
    auto load = [&](int c0, int r0) {
#pragma unroll
        for (int u = 0; u < NR; ++u) {
            const int r = r0 + rg + u * row_groups;
            if (works && !fresh && r < a.dk && c0 < a.dv) {
                s[u] = *reinterpret_cast<const F *>(state + int64_t(r) * a.dv + c0);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[u].v[e] = 0.f;
                }
            }
        }
    };
    load(cg * VEC, 0);
    float *ring = state_ring(a, slot);
    const T *w = static_cast<const T *>(a.conv_w), *bias = static_cast<const T *>(a.conv_b);
    const T *proj = static_cast<const T *>(a.proj) + int64_t(row) * a.row_stride;
    const int n = a.dv + 2 * a.dk;
    auto channel = [&](int j) {
        return j < a.dv ? head * a.dv + j
                        : a.inner() + (j - a.dv < a.dk ? group * a.dk + (j - a.dv) : (a.groups + group) * a.dk + (j - a.dv - a.dk));
    };
    // the earlier inputs' share of the first two channels of a thread, before the wait as well
    auto earlier = [&](int ch) {
        float acc = to_f32(bias[ch]);
        for (int back = min(a.taps - 1, pos); back >= 1; --back) {
            acc = fmaf(to_f32(w[int64_t(ch) * a.taps + a.taps - 1 - back]), ring[int64_t((pos - back) % a.taps) * channels + ch], acc);
        }
        return acc;
    };
    float early[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int j = tid + u * kDecodeThreads;
        early[u] = j < n ? earlier(channel(j)) : 0.f;
    }
    const float rate = -expf(a.a_log[head]), dt_bias = a.dt_bias[head], skip = a.d_skip[head];
    grid_dependency_wait();
    grid_launch_dependents();
    auto convolve = [&](int j, float acc) {
        const int ch = channel(j);
        const float in = to_f32(proj[a.x_at + ch]);
        acc = fmaf(to_f32(w[int64_t(ch) * a.taps + a.taps - 1]), in, acc);
        if (j < a.dv || head % share == 0) { // (the place written is none that this step reads)
            ring[int64_t(pos % a.taps) * channels + ch] = in;
        }
        const float v = to_f32(from_f32<T>(silu_of(acc)));
        (j < a.dv ? s_x[j] : (j - a.dv < a.dk ? s_b[j - a.dv] : s_c[j - a.dv - a.dk])) = v;
    };
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        if (tid + u * kDecodeThreads < n) {
            convolve(tid + u * kDecodeThreads, early[u]);
        }
    }
    for (int j = tid + 2 * kDecodeThreads; j < n; j += kDecodeThreads) {
        convolve(j, earlier(channel(j)));
    }
    const float dt = softplus_of(to_f32(proj[a.dt_at + head]) + dt_bias), keep = expf(rate * dt);
    __syncthreads();
    T *y = reinterpret_cast<T *>(a.scratch) + int64_t(row) * y_stride + int64_t(head) * a.dv;
    for (int pass = 0; pass < a.dv; pass += col_groups * VEC) {
        const int c0 = pass + cg * VEC;
        float acc[VEC] = {};
        for (int r0 = 0; r0 < a.dk; r0 += NR * row_groups) {
            if (pass != 0 || r0 != 0) {
                load(c0, r0);
            }
#pragma unroll
            for (int u = 0; u < NR; ++u) {
                const int r = r0 + rg + u * row_groups;
                if (works && r < a.dk && c0 < a.dv) {
                    const float b = dt * s_b[r], c = s_c[r];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[u].v[e] = fmaf(keep, s[u].v[e], b * s_x[c0 + e]);
                        acc[e] = fmaf(c, s[u].v[e], acc[e]);
                    }
                    *reinterpret_cast<F *>(state + int64_t(r) * a.dv + c0) = s[u];
                }
            }
        }
        if (works) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                s_part[rg * col_groups * VEC + cg * VEC + e] = acc[e];
            }
        }
        __syncthreads();
        for (int c = tid; c < col_groups * VEC && pass + c < a.dv; c += kDecodeThreads) {
            float sum = 0.f;
            for (int g = 0; g < row_groups; ++g) {
                sum += s_part[g * col_groups * VEC + c];
            }
            y[pass + c] = from_f32<T>(fmaf(skip, s_x[pass + c], sum));
        }
        __syncthreads();
    }
}

// The activation behind the convolutions of runs, rounded to the model dtype
template <typename T>
__device__ __forceinline__ T conv_out(float v) {
    if constexpr (sizeof(T) == 4) {
        return silu_of(v);
    } else {
        return from_f32<T>(__fdividef(v, 1.f + __expf(-v)));
    }
}

// CTA: ROWS rows, thread: VEC channels of them; the last CTAs of a row in x compute step sizes. TAPS > 0: weights and the rows' inputs are
// fetched once, all together; TAPS == 0: any number, tap by tap.
template <typename T, int VEC, int TAPS, int ROWS>
__global__ void __launch_bounds__(128) state_prepare_kernel(StateSpaceArgs a, StateScratch sc) {
    struct alignas(sizeof(T) * VEC) Piece {
        T v[VEC];
    };
    grid_dependency_wait();
    grid_launch_dependents();
    __shared__ int s_first[ROWS], s_pos[ROWS], s_slot[ROWS];
    const int row0 = int(blockIdx.y) * ROWS, channels = a.channels(), ch = (int(blockIdx.x) * int(blockDim.x) + int(threadIdx.x)) * VEC;
    const T *proj = static_cast<const T *>(a.proj);
    const bool convolves = ch < channels;
    constexpr int kIn = ROWS + TAPS - 1;
    Piece in[TAPS > 0 ? kIn : 1], weight[TAPS > 0 ? TAPS : 1]; // weight: VEC channels x TAPS, as they lie in memory
    if constexpr (TAPS > 0) {
        if (convolves) {
#pragma unroll
            for (int i = 0; i < kIn; ++i) {
                const int row = row0 - (TAPS - 1) + i;
                if (row >= 0 && row < a.n_rows) { // (of whatever sequence: the first rows of a run do not use it)
                    in[i] = *reinterpret_cast<const Piece *>(proj + int64_t(row) * a.row_stride + a.x_at + ch);
                }
            }
#pragma unroll
            for (int i = 0; i < TAPS; ++i) {
                weight[i] = reinterpret_cast<const Piece *>(static_cast<const T *>(a.conv_w) + int64_t(ch) * TAPS)[i];
            }
        }
    }
    if (threadIdx.x < ROWS && row0 + int(threadIdx.x) < a.n_rows) {
        const int row = row0 + int(threadIdx.x);
        int lo = 0, hi = a.n_seqs - 1;
        while (lo < hi) { // last sequence whose first row is not behind this one
            const int mid = (lo + hi + 1) >> 1;
            if (a.q_starts[mid] <= row) {
                lo = mid;
            } else {
                hi = mid - 1;
            }
        }
        s_first[threadIdx.x] = a.q_starts[lo];
        s_pos[threadIdx.x] = a.kv_lens[lo] - a.q_starts[lo + 1] + row;
        s_slot[threadIdx.x] = a.seq_ids[lo];
    }
    __syncthreads();
    if (!convolves) {
        float *dt = a.scratch + sc.dt;
        const int head = ch / VEC - (channels + VEC - 1) / VEC;
        if (head < a.heads) {
            for (int u = 0; u < ROWS && row0 + u < a.n_rows; ++u) {
                dt[int64_t(row0 + u) * a.heads + head] =
                    softplus_of(to_f32(proj[int64_t(row0 + u) * a.row_stride + a.dt_at + head]) + a.dt_bias[head]);
            }
        }
        return;
    }
    const T *w = static_cast<const T *>(a.conv_w) + int64_t(ch) * a.taps, *bias = static_cast<const T *>(a.conv_b) + ch;
    T *conv = reinterpret_cast<T *>(a.scratch + sc.conv);
    const int taps = TAPS > 0 ? TAPS : a.taps;
    auto earlier = [&](int u, int back) { return state_ring(a, s_slot[u]) + int64_t((s_pos[u] - back) % taps) * channels + ch; };
    auto store = [&](int u, const float (&acc)[VEC]) {
        Piece p;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            p.v[e] = conv_out<T>(acc[e]);
        }
        *reinterpret_cast<Piece *>(conv + int64_t(row0 + u) * sc.conv_stride + ch) = p;
    };
    if constexpr (TAPS > 0) {
        float ww[TAPS][VEC], bb[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            bb[e] = to_f32(bias[e]);
#pragma unroll
            for (int tap = 0; tap < TAPS; ++tap) {
                ww[tap][e] = to_f32(weight[(e * TAPS + tap) / VEC].v[(e * TAPS + tap) % VEC]);
            }
        }
#pragma unroll
        for (int u = 0; u < ROWS; ++u) {
            if (row0 + u >= a.n_rows) {
                break;
            }
            float acc[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                acc[e] = bb[e];
            }
#pragma unroll
            for (int tap = 0; tap < TAPS; ++tap) {
                const int back = TAPS - 1 - tap;
                if (row0 + u - back >= s_first[u]) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        acc[e] = fmaf(ww[tap][e], to_f32(in[u + tap].v[e]), acc[e]);
                    }
                } else if (s_pos[u] >= back) {
                    const float *ring = earlier(u, back);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        acc[e] = fmaf(ww[tap][e], ring[e], acc[e]);
                    }
                }
            }
            store(u, acc);
        }
    } else {
        for (int u = 0; u < ROWS && row0 + u < a.n_rows; ++u) {
            float acc[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                acc[e] = to_f32(bias[e]);
            }
            for (int back = min(taps - 1, s_pos[u]); back >= 0; --back) {
                const int tap = taps - 1 - back;
                const bool here = row0 + u - back >= s_first[u];
                const T *now = proj + int64_t(row0 + u - back) * a.row_stride + a.x_at + ch;
                const float *ring = earlier(u, back);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    acc[e] = fmaf(to_f32(w[e * taps + tap]), here ? to_f32(now[e]) : ring[e], acc[e]);
                }
            }
            store(u, acc);
        }
    }
}

constexpr int kRecThreads = 256, kRecCols = 32, kRecGroups = kRecThreads / kRecCols;

// thread = one column, every kRecGroups-th state row; `batch` tokens are staged at a time.
template <typename T>
__global__ void __launch_bounds__(kRecThreads) state_recurrent_kernel(StateSpaceArgs a, StateScratch sc, int batch) {
    extern __shared__ __align__(16) float smem[];
    float *s_state = smem;                                  // [dk][kRecCols]
    float *s_b = s_state + a.dk * kRecCols;                 // [batch][dk]
    float *s_c = s_b + batch * a.dk;                        // [batch][dk]
    float *s_x = s_c + batch * a.dk;                        // [batch][kRecCols]
    float *s_dt = s_x + batch * kRecCols;                   // [batch]
    float *s_part = s_dt + (batch + 3) / 4 * 4;             // [batch][kRecGroups][kRecCols]
    grid_dependency_wait();
    grid_launch_dependents();
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads, tid = int(threadIdx.x);
    const int first = a.q_starts[i], n_new = a.q_starts[i + 1] - first;
    if (n_new <= 0) {
        return;
    }
    const int64_t slot = a.seq_ids[i];
    const int group = head / (a.heads / a.groups), col0 = int(blockIdx.y) * kRecCols, col = tid % kRecCols, rg = tid / kRecCols;
    if (blockIdx.y == 0) {
        keep_run_inputs<T>(a, head, slot, first, first + n_new - 1, a.kv_lens[i] - 1);
    }
    const bool fresh = a.kv_lens[i] == n_new, holds = col0 + col < a.dv;
    float *state = a.state + slot * a.slot_stride + int64_t(head) * a.dk * a.dv + col0 + col;
    for (int r = rg; r < a.dk; r += kRecGroups) {
        s_state[r * kRecCols + col] = fresh || !holds ? 0.f : state[int64_t(r) * a.dv];
    }
    const float rate = -expf(a.a_log[head]), skip = a.d_skip[head];
    const T *conv = reinterpret_cast<const T *>(a.scratch + sc.conv);
    const float *dt = a.scratch + sc.dt;
    T *y = reinterpret_cast<T *>(a.scratch + sc.y);
    for (int t0 = 0; t0 < n_new; t0 += batch) {
        const int n = min(batch, n_new - t0);
        __syncthreads();
        for (int u = tid; u < n * a.dk; u += kRecThreads) {
            const int t = u / a.dk, c = u - t * a.dk;
            const T *row = conv + int64_t(first + t0 + t) * sc.conv_stride + a.inner() + group * a.dk + c;
            s_b[t * a.dk + c] = to_f32(row[0]);
            s_c[t * a.dk + c] = to_f32(row[a.groups * a.dk]);
        }
        for (int u = tid; u < n * kRecCols; u += kRecThreads) {
            const int t = u / kRecCols, c = u % kRecCols;
            s_x[u] = col0 + c < a.dv ? to_f32(conv[int64_t(first + t0 + t) * sc.conv_stride + head * a.dv + col0 + c]) : 0.f;
        }
        for (int t = tid; t < n; t += kRecThreads) {
            s_dt[t] = dt[int64_t(first + t0 + t) * a.heads + head];
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float step = s_dt[t], keep = expf(rate * step), in = step * s_x[t * kRecCols + col];
            float acc = 0.f;
            for (int r = rg; r < a.dk; r += kRecGroups) {
                const float s = fmaf(keep, s_state[r * kRecCols + col], s_b[t * a.dk + r] * in);
                s_state[r * kRecCols + col] = s;
                acc = fmaf(s_c[t * a.dk + r], s, acc);
            }
            s_part[(t * kRecGroups + rg) * kRecCols + col] = acc;
        }
        __syncthreads();
        for (int u = tid; u < n * kRecCols; u += kRecThreads) {
            const int t = u / kRecCols, c = u % kRecCols;
            if (col0 + c < a.dv) {
                float sum = skip * s_x[u];
                for (int g = 0; g < kRecGroups; ++g) {
                    sum += s_part[(t * kRecGroups + g) * kRecCols + c];
                }
                y[int64_t(first + t0 + t) * sc.y_stride + head * a.dv + col0 + c] = from_f32<T>(sum);
            }
        }
    }
    for (int r = rg; r < a.dk && holds; r += kRecGroups) {
        state[int64_t(r) * a.dv] = s_state[r * kRecCols + col];
    }
}

// CTA: one part of one row. The first PER_THREAD pieces of a thread stay in registers between the sum and the stores.
template <typename T, int VEC, int PER_THREAD>
__global__ void state_finish_kernel(StateSpaceArgs a, StateScratch sc) {
    struct alignas(sizeof(T) * VEC) Piece {
        T v[VEC];
    };
    grid_dependency_wait();
    grid_launch_dependents();
    const int64_t row = blockIdx.x;
    const int size = a.inner() / a.norm_groups, at = int(blockIdx.y) * size, n_vec = size / VEC, step = int(blockDim.x);
    const Piece *y = reinterpret_cast<const Piece *>(reinterpret_cast<const T *>(a.scratch + sc.y) + row * sc.y_stride + at);
    const Piece *z = reinterpret_cast<const Piece *>(static_cast<const T *>(a.proj) + row * a.row_stride + a.z_at + at);
    const Piece *w = reinterpret_cast<const Piece *>(static_cast<const T *>(a.norm_w) + at);
    Piece *out = reinterpret_cast<Piece *>(static_cast<T *>(a.out) + row * a.out_stride + at);
    float ss = 0.f;
    auto gated = [&](int i) {
        const Piece py = y[i], pz = z[i];
        Floats<VEC> f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            f.v[e] = to_f32(py.v[e]) * silu_of(to_f32(pz.v[e]));
        }
        return f;
    };
    Floats<VEC> held[PER_THREAD];
    auto square = [&](const Floats<VEC> &f) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            ss = fmaf(f.v[e], f.v[e], ss);
        }
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int i = int(threadIdx.x) + r * step;
        if (i < n_vec) {
            held[r] = gated(i);
            square(held[r]);
        }
    }
    for (int i = int(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        square(gated(i));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        ss += __shfl_xor_sync(0xffffffffu, ss, o);
    }
    __shared__ float part[32];
    if ((threadIdx.x & 31) == 0) {
        part[threadIdx.x >> 5] = ss;
    }
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < step >> 5; ++i) {
        tot += part[i]; // every thread adds the few partials in the same order
    }
    const float inv = rsqrtf(tot / float(size) + a.eps);
    auto store = [&](int i, const Floats<VEC> &f) {
        const Piece pw = w[i];
        Piece o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            o.v[e] = from_f32<T>(f.v[e] * inv * to_f32(pw.v[e]));
        }
        out[i] = o;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int i = int(threadIdx.x) + r * step;
        if (i < n_vec) {
            store(i, held[r]);
        }
    }
    for (int i = int(threadIdx.x) + PER_THREAD * step; i < n_vec; i += step) {
        store(i, gated(i));
    }
}

void check_sizes(llaisysDataType_t dtype, const StateSpaceArgs &a) {
    CHECK_ARGUMENT(a.heads > 0 && a.groups > 0 && a.heads % a.groups == 0 && a.dk > 0 && a.dv > 0 && a.taps > 0 && a.norm_groups > 0 &&
                       a.inner() % a.norm_groups == 0 && a.dk <= 1024 && a.dv <= 1024 && a.norm_groups <= 65535,
                   "state space: inconsistent sizes");
    CHECK_ARGUMENT(a.scratch != nullptr && a.scratch_floats >= size_t(state_scratch(dtype, a.n_rows, a.heads, a.groups, a.dk, a.dv).total),
                   "state space: scratch missing or too small");
}

template <typename T>
void run_decode(cudaStream_t s, const StateSpaceArgs &a, const StateScratch &sc) {
    const bool wide = a.dv % 4 == 0;
    const int vec = wide ? 4 : 1, col_groups = std::min((a.dv + vec - 1) / vec, kDecodeThreads), row_groups = kDecodeThreads / col_groups;
    auto up4 = [](int n) { return (n + 3) / 4 * 4; };
    const size_t smem = size_t(up4(a.dv) + 2 * up4(a.dk) + row_groups * col_groups * vec) * sizeof(float);
    auto kernel = wide ? state_decode_kernel<T, 4, 4> : state_decode_kernel<T, 1, 4>;
    launch_programmatic_smem(kernel, dim3(unsigned(a.n_seqs) * unsigned(a.heads)), kDecodeThreads, smem, s, a, sc.y_stride, col_groups);
    check_launch("state_space decode");
}

template <typename T>
void run_finish(cudaStream_t s, const StateSpaceArgs &a, const StateScratch &sc) {
    constexpr int kVec = 16 / int(sizeof(T));
    const int size = a.inner() / a.norm_groups;
    const bool wide = size % kVec == 0 && a.row_stride % kVec == 0 && a.z_at % kVec == 0 && a.out_stride % kVec == 0 && aligned16(a.proj) &&
                      aligned16(a.out) && aligned16(a.norm_w);
    const int vecs = wide ? size / kVec : size, want = (vecs + 1) / 2;
    auto kernel = wide ? state_finish_kernel<T, kVec, 2> : state_finish_kernel<T, 1, 4>;
    launch_programmatic(kernel, dim3(unsigned(a.n_rows), unsigned(a.norm_groups)), unsigned(want < 64 ? 64 : (want > 512 ? 512 : (want + 31) / 32 * 32)),
                        s, a, sc);
    check_launch("state_space finish");
}

template <typename T>
void run_prepare(cudaStream_t s, const StateSpaceArgs &a, const StateScratch &sc) {
    constexpr int kVec = sizeof(T) == 2 ? 8 : 4;
    const bool wide = a.channels() % kVec == 0 && a.row_stride % kVec == 0 && a.x_at % kVec == 0 && aligned16(a.proj);
    const bool known = wide && a.taps >= 2 && a.taps <= 4 && aligned16(a.conv_w);
    const int vec = wide ? kVec : 1, items = (a.channels() + vec - 1) / vec + a.heads, rows = known ? kConvRows : kConvRowsAny;
    auto kernel = !wide           ? state_prepare_kernel<T, 1, 0, kConvRowsAny>
                  : !known        ? state_prepare_kernel<T, kVec, 0, kConvRowsAny>
                  : a.taps == 4   ? state_prepare_kernel<T, kVec, 4, kConvRows>
                  : a.taps == 3   ? state_prepare_kernel<T, kVec, 3, kConvRows>
                                  : state_prepare_kernel<T, kVec, 2, kConvRows>;
    const int64_t tiles = (a.n_rows + rows - 1) / rows;
    CHECK_ARGUMENT(tiles <= 65535, "state space: too many rows in one call");
    launch_programmatic(kernel, dim3(unsigned((items + 127) / 128), unsigned(tiles)), 128u, s, a, sc);
    check_launch("state_space prepare");
}

template <typename T>
void run_recurrent(cudaStream_t s, const StateSpaceArgs &a, const StateScratch &sc) {
    auto smem_for = [&](int batch) {
        return (size_t(a.dk) * kRecCols + size_t(batch) * (2 * a.dk + kRecCols + kRecGroups * kRecCols) + size_t(batch + 3) / 4 * 4) * sizeof(float);
    };
    int batch = 16;
    while (batch > 1 && smem_for(batch) > 200 * 1024) {
        batch /= 2;
    }
    const size_t smem = smem_for(batch);
    if (smem > 48 * 1024) {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(state_recurrent_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    }
    launch_programmatic_smem(state_recurrent_kernel<T>, dim3(unsigned(a.n_seqs) * unsigned(a.heads), unsigned((a.dv + kRecCols - 1) / kRecCols)),
                             kRecThreads, smem, s, a, sc, batch);
    check_launch("state_space recurrent");
}

} // namespace

size_t state_space_state_floats(size_t heads, size_t groups, size_t dk, size_t dv, size_t taps) {
    return heads * dk * dv + taps * (heads * dv + 2 * groups * dk);
}

size_t state_space_scratch_floats(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t groups, size_t dk, size_t dv) {
    return size_t(state_scratch(dtype, int64_t(n_rows), int64_t(heads), int64_t(groups), int64_t(dk), int64_t(dv)).total);
}

void state_space_decode(stream_t stream, llaisysDataType_t dtype, const StateSpaceArgs &args) {
    if (args.n_rows == 0) {
        return;
    }
    check_sizes(dtype, args);
    StateSpaceArgs a = args;
    a.q_starts = nullptr;
    const StateScratch sc = state_scratch(dtype, a.n_rows, a.heads, a.groups, a.dk, a.dv);
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        run_decode<decltype(tag)>(s, a, sc);
        run_finish<decltype(tag)>(s, a, sc);
    });
}

void state_space_chunk(stream_t stream, llaisysDataType_t dtype, const StateSpaceArgs &a) {
    if (a.n_rows == 0) {
        return;
    }
    check_sizes(dtype, a);
    const StateScratch sc = state_scratch(dtype, a.n_rows, a.heads, a.groups, a.dk, a.dv);
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        run_prepare<T>(s, a, sc);
        if (state_space_tiles_fit(dtype, a)) {
            state_space_tiles(stream, a);
            run_decode<T>(s, a, sc);
        } else {
            run_recurrent<T>(s, a, sc);
        }
        run_finish<T>(s, a, sc);
    });
}

} // namespace llaisys::kernels
