// Gated delta rule (see GatedDeltaArgs): what precedes the recurrence, its two plain forms, and the choice between forms.
//   * decode: one token per sequence, everything from the projection row to the gated, normed output in one launch: short
//     convolutions, unit vectors, decay, state and read-out. A CTA owns one (sequence, head) and holds that head's f32 state in
//     registers between the read-out for the correction and the update: it is read and written once -- HBM-bound,
//     2 * dk * dv * 4 bytes per head. In a batch with runs the same launch serves the sequences that bring a single token, and
//     stores the newest convolution inputs of the others.
//   * prepare: for the rows of runs, convolutions + silu (rounded to the model dtype), the factors that make q and k unit
//     vectors, write strengths and (one per head) log decays.
//   * recurrent: runs of tokens, one after the other in f32 with the state in registers. A CTA owns 16 value columns of one
//     (sequence, head). Exact in the order of the definition.
//     (The third form, runs on the tensor cores, is gated_delta_chunk.cu; bf16 models run that one.)
#include "device_utils.cuh"
#include "gated_delta.cuh"
#include "kernels.hpp"
#include "mma_utils.cuh"

#include <type_traits>
#include <utility>

namespace llaisys::kernels {

namespace {

constexpr int kDecodeThreads = 512;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        v += __shfl_xor_sync(0xffffffffu, v, o);
    }
    return v;
}

// The newest inputs of a run's convolutions go to the ring: the CTA of (sequence, head) stores its value channels, the first
// head of a group its q and k channels too. `first` .. `last`: rows whose inputs are kept, pos_last the last one's position.
template <typename T>
__device__ void keep_inputs(const GatedDeltaArgs &a, int head, int64_t slot, int first, int last, int pos_last) {
    float *ring = delta_ring(a, slot);
    const int group = a.heads / a.kv_heads, nq = a.kv_heads * a.dk, channels = a.channels();
    const int n_qk = head % group == 0 ? 2 * a.dk : 0, n = n_qk + a.dv;
    const T *proj = static_cast<const T *>(a.proj);
    for (int u = int(threadIdx.x); u < n * (last - first + 1); u += int(blockDim.x)) {
        const int back = u / n, j = u - back * n;
        const int kvh = head / group;
        const int ch = j < n_qk ? (j < a.dk ? kvh * a.dk + j : nq + kvh * a.dk + (j - a.dk)) : 2 * nq + head * a.dv + (j - n_qk);
        ring[int64_t((pos_last - back) % a.taps) * channels + ch] = to_f32(proj[int64_t(last - back) * a.row_stride + delta_input_at(a, ch)]);
    }
}

// Sum over ranks of w[r] z[r], by the four neighbouring lanes `lane4` = 0 .. 3 of one channel; every one gets the sum.
template <typename T>
__device__ __forceinline__ float decay_product(const T *w, const float *z, int rank, bool wide, int lane4) {
    float acc = 0.f;
    constexpr int kVec = 16 / int(sizeof(T));
    if (wide) { // rows of w in whole 16-byte pieces (padding included, which meets zeros in z)
        using P = Pieces<T, kVec>;
#pragma unroll 4
        for (int r = lane4 * kVec; r < rank; r += 4 * kVec) {
            const P p = *reinterpret_cast<const P *>(w + r);
#pragma unroll
            for (int e = 0; e < kVec; ++e) {
                acc = fmaf(to_f32(p.v[e]), z[r + e], acc);
            }
        }
    } else {
#pragma unroll 4
        for (int r = lane4; r < rank; r += 4) {
            acc = fmaf(to_f32(w[r]), z[r], acc);
        }
    }
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    return acc + __shfl_xor_sync(0xffffffffu, acc, 2);
}

// thread = (VEC columns, every row_groups-th of the dk rows, NR of them at most). Everything that no kernel of this step writes
// is fetched before the wait for the previous kernel: the state, the convolutions' earlier inputs and weights.
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(kDecodeThreads, 2) gated_delta_decode_kernel(GatedDeltaArgs a, int col_groups, int wide_decay) {
    extern __shared__ __align__(16) float smem[];
    auto up4 = [](int n) { return (n + 3) / 4 * 4; };
    const int rank_pad = (a.rank + 31) / 32 * 32;
    float *s_q = smem;                   // [dk] unit vectors
    float *s_k = s_q + up4(a.dk);        // [dk]
    float *s_a = s_k + up4(a.dk);        // [dk] decay
    float *s_v = s_a + up4(a.dk);        // [dv]
    float *s_o = s_v + up4(a.dv);        // [dv]
    float *s_z = s_o + up4(a.dv);        // [rank, padded]
    float *s_u = s_z + rank_pad;         // [columns of a pass]
    float *s_part = s_u + up4(col_groups * VEC); // [row groups][columns of a pass]
    __shared__ float s_red[3][kDecodeThreads / 32];

    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    const int64_t slot = a.seq_ids[i];
    const int row_i = a.q_starts != nullptr ? a.q_starts[i] : i, n_new = a.q_starts != nullptr ? a.q_starts[i + 1] - row_i : 1;
    const int pos = a.kv_lens[i] - 1; // of the newest token
    if (n_new != 1) {
        grid_dependency_wait();
        grid_launch_dependents();
        if (n_new > 1) {
            keep_inputs<T>(a, head, slot, row_i + max(n_new - a.taps, 0), row_i + n_new - 1, pos);
        }
        return;
    }
    const bool fresh = pos == 0;

    float *state = a.state + slot * a.slot_stride + int64_t(head) * a.dk * a.dv;
    using F = Pieces<float, VEC>;
    const int row_groups = kDecodeThreads / col_groups, cg = tid % col_groups, rg = tid / col_groups;
    F s[NR];
    auto load = [&](int c0) {
#pragma unroll
        for (int u = 0; u < NR; ++u) {
            const int r = rg + u * row_groups;
            if (!fresh && r < a.dk && c0 < a.dv) {
                s[u] = *reinterpret_cast<const F *>(state + int64_t(r) * a.dv + c0);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[u].v[e] = 0.f;
                }
            }
        }
    };
    load(cg * VEC);

    // ---- convolutions: channel j of this head's q | k | v ---------------------------------------------------------------
    const int group = a.heads / a.kv_heads, kvh = head / group, nq = a.kv_heads * a.dk, channels = a.channels();
    float *ring = delta_ring(a, slot);
    auto channel = [&](int j) {
        return j < a.dk ? kvh * a.dk + j : (j < 2 * a.dk ? nq + kvh * a.dk + (j - a.dk) : 2 * nq + head * a.dv + (j - 2 * a.dk));
    };
    auto history = [&](int ch, float &w_now) { // what the earlier inputs add to the channel's sum
        const T *w = delta_taps<T>(a, ch);
        w_now = to_f32(w[a.taps - 1]);
        float x[3], y[3], acc = 0.f;
#pragma unroll
        for (int b = 1; b <= 3; ++b) {
            const bool in = b < a.taps && b <= pos;
            x[b - 1] = in ? ring[int64_t((pos - b) % a.taps) * channels + ch] : 0.f;
            y[b - 1] = in ? to_f32(w[a.taps - 1 - b]) : 0.f;
        }
#pragma unroll
        for (int b = 0; b < 3; ++b) {
            acc = fmaf(x[b], y[b], acc);
        }
        for (int b = 4; b < a.taps && b <= pos; ++b) {
            acc = fmaf(ring[int64_t((pos - b) % a.taps) * channels + ch], to_f32(w[a.taps - 1 - b]), acc);
        }
        return acc;
    };
    const int n_channels = 2 * a.dk + a.dv;
    float w_now = 0.f, acc_first = tid < n_channels ? history(channel(tid), w_now) : 0.f;
    const float a_log = to_f32(static_cast<const T *>(a.a_log)[head]);
    const float norm = tid < a.dv ? to_f32(static_cast<const T *>(a.norm_w)[tid]) : 0.f;
    grid_dependency_wait();
    grid_launch_dependents();

    const T *row = static_cast<const T *>(a.proj) + int64_t(row_i) * a.row_stride;
    const T *gate = static_cast<const T *>(a.gate) + int64_t(row_i) * a.gate_stride + int64_t(head) * a.dv;
    const float gate_in = tid < a.dv ? to_f32(gate[tid]) : 0.f;
    const float beta = sigmoid_of(to_f32(row[a.b_at + head]));
    if (a.decay_w != nullptr) {
        for (int r = tid; r < rank_pad; r += kDecodeThreads) {
            s_z[r] = r < a.rank ? to_f32(row[a.a_at + r]) : 0.f;
        }
    }
    float ss[2] = {0.f, 0.f};
    for (int j = tid; j < n_channels; j += kDecodeThreads) {
        const int ch = channel(j), part = j < a.dk ? 0 : (j < 2 * a.dk ? 1 : 2);
        const float now = to_f32(row[delta_input_at(a, ch)]);
        float acc = j == tid ? acc_first : history(ch, w_now);
        acc = fmaf(now, w_now, acc);
        if (part == 2 || head % group == 0) {
            ring[int64_t(pos % a.taps) * channels + ch] = now; // (no other CTA reads this place in this launch)
        }
        const float y = to_f32(from_f32<T>(silu(acc)));
        (part == 0 ? s_q[j] : (part == 1 ? s_k[j - a.dk] : s_v[j - 2 * a.dk])) = y;
        ss[0] += part == 0 ? y * y : 0.f;
        ss[1] += part == 1 ? y * y : 0.f;
    }
    ss[0] = warp_sum(ss[0]);
    ss[1] = warp_sum(ss[1]);
    if (lane == 0) {
        s_red[0][warp] = ss[0];
        s_red[1][warp] = ss[1];
    }
    __syncthreads();
    if (a.decay_w != nullptr) {
        const T *w = static_cast<const T *>(a.decay_w) + int64_t(head) * a.dk * a.decay_ld;
        const T *bias = static_cast<const T *>(a.dt_bias) + int64_t(head) * a.dk;
        for (int c0 = 0; c0 < a.dk; c0 += kDecodeThreads / 4) { // four lanes per channel
            const int c = c0 + (tid >> 2), cc = min(c, a.dk - 1);
            const float x = decay_product(w + int64_t(cc) * a.decay_ld, s_z, a.rank, wide_decay != 0, tid & 3) + to_f32(bias[cc]);
            if ((tid & 3) == 0 && c < a.dk) {
                s_a[c] = expf(delta_decay_log(a_log, x));
            }
        }
    } else {
        const float g = expf(delta_decay_log(a_log, to_f32(row[a.a_at + head]) + to_f32(static_cast<const T *>(a.dt_bias)[head])));
        for (int c = tid; c < a.dk; c += kDecodeThreads) {
            s_a[c] = g;
        }
    }
    {
        float unit[2] = {a.unit_eps, a.unit_eps};
#pragma unroll
        for (int w = 0; w < kDecodeThreads / 32; ++w) {
            unit[0] += s_red[0][w];
            unit[1] += s_red[1][w];
        }
        unit[0] = a.q_scale * rsqrtf(unit[0]);
        unit[1] = rsqrtf(unit[1]);
        for (int c = tid; c < a.dk; c += kDecodeThreads) {
            s_q[c] *= unit[0];
            s_k[c] *= unit[1];
        }
    }
    __syncthreads();

    // ---- the state, as many columns at a time as the CTA's threads cover ------------------------------------------------
    const int pass = col_groups * VEC;
    float so = 0.f; // squares of this thread's outputs
    for (int base = 0; base < a.dv; base += pass) {
        const int c0 = base + cg * VEC;
        if (base > 0) {
            load(c0);
        }
        F acc;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            acc.v[e] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < NR; ++u) {
            const int r = rg + u * row_groups;
            if (r < a.dk) {
                const float g = s_a[r], k = s_k[r];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[u].v[e] *= g;
                    acc.v[e] = fmaf(s[u].v[e], k, acc.v[e]);
                }
            }
        }
        F *mine = reinterpret_cast<F *>(s_part + rg * pass + cg * VEC);
        *mine = acc;
        auto column = [&](int c) {
            float sum = 0.f;
#pragma unroll 8
            for (int g = 0; g < row_groups; ++g) {
                sum += s_part[g * pass + c];
            }
            return sum;
        };
        __syncthreads();
        for (int c = tid; c < pass; c += kDecodeThreads) {
            s_u[c] = base + c < a.dv ? beta * (s_v[base + c] - column(c)) : 0.f;
        }
        __syncthreads();
        const F w = *reinterpret_cast<const F *>(s_u + cg * VEC);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            acc.v[e] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < NR; ++u) {
            const int r = rg + u * row_groups;
            if (r < a.dk && c0 < a.dv) {
                const float k = s_k[r], q = s_q[r];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[u].v[e] = fmaf(k, w.v[e], s[u].v[e]);
                    acc.v[e] = fmaf(q, s[u].v[e], acc.v[e]);
                }
                *reinterpret_cast<F *>(state + int64_t(r) * a.dv + c0) = s[u];
            }
        }
        *mine = acc;
        __syncthreads();
        for (int c = tid; c < pass && base + c < a.dv; c += kDecodeThreads) {
            const float o = column(c);
            s_o[base + c] = o;
            so = fmaf(o, o, so);
        }
        if (base + pass < a.dv) {
            __syncthreads(); // the next pass writes the partial sums
        }
    }

    // ---- norm, gate ------------------------------------------------------------------------------------------------------
    so = warp_sum(so);
    if (lane == 0) {
        s_red[2][warp] = so;
    }
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kDecodeThreads / 32; ++w) {
        tot += s_red[2][w];
    }
    const float inv = rsqrtf(tot / float(a.dv) + a.eps);
    T *out = static_cast<T *>(a.out) + int64_t(row_i) * a.out_stride + int64_t(head) * a.dv;
    for (int c = tid; c < a.dv; c += kDecodeThreads) {
        const float y = c == tid ? gate_in : to_f32(gate[c]);
        const float w = c == tid ? norm : to_f32(static_cast<const T *>(a.norm_w)[c]);
        out[c] = from_f32<T>(s_o[c] * inv * w * (a.gate_silu ? silu(y) : sigmoid_of(y)));
    }
}

constexpr int kStrip = 16, kPrepWarps = 8;

// One warp per head of q, k or v (and one for write strengths and decays of all heads) over a strip of kStrip rows; a lane owns
// VEC channels and keeps their newest inputs in registers from row to row (kTaps; 0: any number of taps, inputs read again).
template <typename T, int VEC, int kTaps>
__global__ void __launch_bounds__(kPrepWarps * 32, kTaps > 0 ? 4 : 2) gated_delta_prepare_kernel(GatedDeltaArgs a, DeltaScratch at) {
    const int lane = int(threadIdx.x) & 31, unit = int(blockIdx.y) * kPrepWarps + (int(threadIdx.x) >> 5);
    const int r0 = int(blockIdx.x) * kStrip, r1 = min(r0 + kStrip, a.n_rows);
    const int units = 2 * a.kv_heads + a.heads;
    if (unit > units) {
        return;
    }
    const T *proj = static_cast<const T *>(a.proj);
    if (unit == units) {
        for (int u = lane; u < (r1 - r0) * a.heads; u += 32) {
            const int row = r0 + u / a.heads, head = u % a.heads;
            const T *p = proj + int64_t(row) * a.row_stride;
            a.scratch[at.beta + int64_t(row) * a.heads + head] = sigmoid_of(to_f32(p[a.b_at + head]));
            if (a.decay_w == nullptr) {
                a.scratch[at.decay_log + int64_t(row) * a.heads + head] =
                    delta_decay_log(to_f32(static_cast<const T *>(a.a_log)[head]),
                                    to_f32(p[a.a_at + head]) + to_f32(static_cast<const T *>(a.dt_bias)[head]));
            }
        }
        return;
    }
    int seq0 = 0;
    {
        int hi = a.n_seqs - 1;
        while (seq0 < hi) { // last sequence that starts at or before r0
            const int mid = (seq0 + hi + 1) >> 1;
            if (a.q_starts[mid] <= r0) {
                seq0 = mid;
            } else {
                hi = mid - 1;
            }
        }
    }
    const bool is_v = unit >= 2 * a.kv_heads;
    const int size = is_v ? a.dv : a.dk, channels = a.channels();
    const int ch0 = is_v ? 2 * a.kv_heads * a.dk + (unit - 2 * a.kv_heads) * a.dv : unit * a.dk;
    using P = Pieces<T, VEC>;
    T *conv = reinterpret_cast<T *>(a.scratch);
    __shared__ float s_squares[kPrepWarps][kStrip][32]; // (a thread's own places: no barrier)
    float *ss = &s_squares[threadIdx.x >> 5][0][lane];
    for (int u = 0; u < kStrip; ++u) {
        ss[u * 32] = 0.f;
    }
    for (int c = lane * VEC; c < size; c += 32 * VEC) {
        const int ch = ch0 + c;
        const int64_t in_at = delta_input_at(a, ch);
        const T *w = delta_taps<T>(a, ch);
        constexpr int kHeld = kTaps > 0 ? kTaps : 1;
        float taps[kHeld][VEC], held[kHeld][VEC]; // by age: 0 = the current token's
        if constexpr (kTaps > 0) {
#pragma unroll
            for (int b = 0; b < kTaps; ++b) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    taps[b][e] = b < a.taps ? to_f32(w[e * a.taps + a.taps - 1 - b]) : 0.f;
                    held[b][e] = 0.f;
                }
            }
        }
        // the input `b` tokens before `row`, whose sequence starts its run at `start`, at position pos0
        auto input = [&](int row, int b, int start, int pos0, const float *ring, float (&x)[VEC]) {
            const int pos = pos0 + row - start - b;
            if (row - b >= start) {
                const P p = *reinterpret_cast<const P *>(proj + int64_t(row - b) * a.row_stride + in_at);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    x[e] = to_f32(p.v[e]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    x[e] = pos >= 0 && b < a.taps ? ring[int64_t(pos % a.taps) * channels + ch + e] : 0.f;
                }
            }
        };
        int seq = seq0, start = a.q_starts[seq], stop = a.q_starts[seq + 1];
        auto finish = [&](int row, const float (&acc)[VEC]) {
            P y;
            float sum = 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                y.v[e] = from_f32<T>(std::is_same_v<T, float> ? silu(acc[e]) : __fdividef(acc[e], 1.f + __expf(-acc[e])));
                sum = fmaf(to_f32(y.v[e]), to_f32(y.v[e]), sum);
            }
            *reinterpret_cast<P *>(conv + int64_t(row) * at.conv_stride + ch) = y;
            if (!is_v) {
                ss[(row - r0) * 32] += sum;
            }
        };
        if constexpr (kTaps > 0) {
            if (r0 >= start && r0 + kStrip <= stop) { // the strip lies inside one run: all its inputs are asked for eight rows at a time
                const float *ring = delta_ring(a, a.seq_ids[seq]);
                const int pos0 = a.kv_lens[seq] - (stop - start);
#pragma unroll
                for (int b = 1; b < kTaps; ++b) {
                    input(r0, b, start, pos0, ring, held[b]);
                }
                constexpr int kBatch = kStrip / 2;
#pragma unroll 1
                for (int u0 = 0; u0 < kStrip; u0 += kBatch) {
                    P raw[kBatch];
#pragma unroll
                    for (int u = 0; u < kBatch; ++u) {
                        raw[u] = *reinterpret_cast<const P *>(proj + int64_t(r0 + u0 + u) * a.row_stride + in_at);
                    }
#pragma unroll
                    for (int u = 0; u < kBatch; ++u) {
                        float acc[VEC];
#pragma unroll
                        for (int e = 0; e < VEC; ++e) {
                            held[0][e] = to_f32(raw[u].v[e]);
                            acc[e] = held[0][e] * taps[0][e];
#pragma unroll
                            for (int b = 1; b < kTaps; ++b) {
                                acc[e] = fmaf(held[b][e], taps[b][e], acc[e]);
                            }
#pragma unroll
                            for (int b = kTaps - 1; b > 0; --b) {
                                held[b][e] = held[b - 1][e];
                            }
                        }
                        finish(r0 + u0 + u, acc);
                    }
                }
                continue;
            }
        }
        bool refill = true;
#pragma unroll 1
        for (int row = r0; row < r1; ++row) {
            while (row >= stop && seq + 1 < a.n_seqs) {
                ++seq;
                start = stop;
                stop = a.q_starts[seq + 1];
                refill = true;
            }
            if (stop - start < 2) {
                continue; // single tokens are the decode kernel's
            }
            const int pos0 = a.kv_lens[seq] - (stop - start);
            const float *ring = delta_ring(a, a.seq_ids[seq]);
            float acc[VEC];
            if constexpr (kTaps > 0) {
                if (refill) {
#pragma unroll
                    for (int b = 1; b < kTaps; ++b) {
                        input(row, b, start, pos0, ring, held[b]);
                    }
                    refill = false;
                }
                input(row, 0, start, pos0, ring, held[0]);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    acc[e] = held[0][e] * taps[0][e];
#pragma unroll
                    for (int b = 1; b < kTaps; ++b) {
                        acc[e] = fmaf(held[b][e], taps[b][e], acc[e]);
                    }
#pragma unroll
                    for (int b = kTaps - 1; b > 0; --b) {
                        held[b][e] = held[b - 1][e];
                    }
                }
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    acc[e] = 0.f;
                }
                for (int b = 0; b < a.taps; ++b) {
                    input(row, b, start, pos0, ring, held[0]);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        acc[e] = fmaf(held[0][e], to_f32(w[e * a.taps + a.taps - 1 - b]), acc[e]);
                    }
                }
            }
            finish(row, acc);
        }
    }
    if (is_v) {
        return;
    }
    for (int u = 0; u < kStrip; ++u) {
        const float tot = warp_sum(ss[u * 32]);
        if (lane == u && r0 + u < r1) {
            a.scratch[at.unit + int64_t(r0 + u) * 2 * a.kv_heads + unit] = rsqrtf(tot + a.unit_eps) * (unit < a.kv_heads ? a.q_scale : 1.f);
        }
    }
}

// decay[row, h * dk + c] (not its logarithm), for the form that goes token by token
template <typename T>
__global__ void gated_delta_decay_kernel(GatedDeltaArgs a, DeltaScratch at) {
    extern __shared__ float s_zrow[];
    const int64_t row = blockIdx.x;
    const T *proj = static_cast<const T *>(a.proj) + row * a.row_stride;
    if (a.decay_w != nullptr) {
        for (int r = int(threadIdx.x); r < a.rank; r += int(blockDim.x)) {
            s_zrow[r] = to_f32(proj[a.a_at + r]);
        }
        __syncthreads();
    }
    const int n = a.heads * a.dk;
    for (int c = int(threadIdx.x); c < n; c += int(blockDim.x)) {
        const int head = c / a.dk;
        const float log = a.decay_w != nullptr
                              ? delta_decay_log(to_f32(static_cast<const T *>(a.a_log)[head]), delta_decay_input<T>(a, s_zrow, head, c - head * a.dk))
                              : a.scratch[at.decay_log + row * a.heads + head];
        a.scratch[at.decay + row * n + c] = expf(log);
    }
}

constexpr int kRecCols = 16, kRecRowGroups = 8, kRecThreads = kRecCols * kRecRowGroups;

// NR state rows per thread: row(j) = 4 * g + 32 * (j / 4) + j % 4 for row group g.
template <typename T, int NR>
__global__ void __launch_bounds__(kRecThreads) gated_delta_recurrent_kernel(GatedDeltaArgs a, DeltaScratch at) {
    constexpr int kRows = kRecRowGroups * NR;
    constexpr int kTok = NR > 32 ? 4 : 8; // tokens staged at a time
    __shared__ __align__(16) float s_q[kTok][kRows], s_k[kTok][kRows], s_a[kTok][kRows];
    __shared__ float s_v[kTok][kRecCols], s_beta[kTok];
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int tid = int(threadIdx.x), g = tid % kRecRowGroups, cl = tid / kRecRowGroups;
    const int col = int(blockIdx.y) * kRecCols + cl;
    const int row0 = a.q_starts[i], row1 = a.q_starts[i + 1];
    if (row1 - row0 < 2) {
        return; // single tokens are the decode kernel's
    }
    const bool fresh = a.kv_lens[i] == row1 - row0;
    float *state = a.state + int64_t(a.seq_ids[i]) * a.slot_stride + int64_t(head) * a.dk * a.dv;
    auto row_of = [&](int j) { return 4 * g + 32 * (j / 4) + j % 4; };
    float s[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        s[j] = !fresh && row_of(j) < a.dk && col < a.dv ? state[int64_t(row_of(j)) * a.dv + col] : 0.f;
    }
    const T *conv = reinterpret_cast<const T *>(a.scratch);
    const float *unit = a.scratch + at.unit;
    const int kvh = head / (a.heads / a.kv_heads), nq = a.kv_heads * a.dk;
    auto over_rows = [](float v) {
        v += __shfl_xor_sync(0xffffffffu, v, 1);
        v += __shfl_xor_sync(0xffffffffu, v, 2);
        return v + __shfl_xor_sync(0xffffffffu, v, 4);
    };
    for (int t0 = row0; t0 < row1; t0 += kTok) {
        __syncthreads();
        for (int u = tid; u < kTok * kRows; u += kRecThreads) {
            const int t = u / kRows, r = u - t * kRows;
            const bool in = t0 + t < row1 && r < a.dk;
            const T *x = conv + int64_t(t0 + t) * at.conv_stride + kvh * a.dk + r;
            const float *f = unit + int64_t(t0 + t) * 2 * a.kv_heads + kvh;
            s_q[t][r] = in ? to_f32(x[0]) * f[0] : 0.f;
            s_k[t][r] = in ? to_f32(x[nq]) * f[a.kv_heads] : 0.f;
            s_a[t][r] = in ? a.scratch[at.decay + (int64_t(t0 + t) * a.heads + head) * a.dk + r] : 1.f;
        }
        for (int u = tid; u < kTok * kRecCols; u += kRecThreads) {
            const int t = u / kRecCols, c = u - t * kRecCols + int(blockIdx.y) * kRecCols;
            s_v[t][u % kRecCols] =
                t0 + t < row1 && c < a.dv ? to_f32(conv[int64_t(t0 + t) * at.conv_stride + 2 * nq + int64_t(head) * a.dv + c]) : 0.f;
        }
        if (tid < kTok) {
            s_beta[tid] = t0 + tid < row1 ? a.scratch[at.beta + int64_t(t0 + tid) * a.heads + head] : 0.f;
        }
        __syncthreads();
        const int n = min(kTok, row1 - t0);
        for (int t = 0; t < n; ++t) {
            float d = 0.f, o = 0.f;
#pragma unroll
            for (int j = 0; j < NR; j += 4) {
                const float4 k4 = *reinterpret_cast<const float4 *>(&s_k[t][4 * g + 8 * j]);
                const float4 a4 = *reinterpret_cast<const float4 *>(&s_a[t][4 * g + 8 * j]);
                s[j] *= a4.x;
                s[j + 1] *= a4.y;
                s[j + 2] *= a4.z;
                s[j + 3] *= a4.w;
                d = fmaf(k4.x, s[j], d);
                d = fmaf(k4.y, s[j + 1], d);
                d = fmaf(k4.z, s[j + 2], d);
                d = fmaf(k4.w, s[j + 3], d);
            }
            const float w = s_beta[t] * (s_v[t][cl] - over_rows(d));
#pragma unroll
            for (int j = 0; j < NR; j += 4) {
                const float4 q4 = *reinterpret_cast<const float4 *>(&s_q[t][4 * g + 8 * j]);
                const float4 k4 = *reinterpret_cast<const float4 *>(&s_k[t][4 * g + 8 * j]);
                s[j] = fmaf(k4.x, w, s[j]);
                s[j + 1] = fmaf(k4.y, w, s[j + 1]);
                s[j + 2] = fmaf(k4.z, w, s[j + 2]);
                s[j + 3] = fmaf(k4.w, w, s[j + 3]);
                o = fmaf(q4.x, s[j], o);
                o = fmaf(q4.y, s[j + 1], o);
                o = fmaf(q4.z, s[j + 2], o);
                o = fmaf(q4.w, s[j + 3], o);
            }
            o = over_rows(o);
            if (g == 0 && col < a.dv) {
                a.scratch[at.raw + (int64_t(t0 + t) * a.heads + head) * a.dv + col] = o;
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

// out = rms_norm(raw) * gate: one warp per (row, head)
template <typename T>
__global__ void gated_delta_out_kernel(GatedDeltaArgs a, DeltaScratch at) {
    const int64_t item = int64_t(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = int(threadIdx.x) & 31;
    if (item >= int64_t(a.n_rows) * a.heads) {
        return;
    }
    const int64_t row = item / a.heads;
    const int head = int(item - row * a.heads);
    const float *o = a.scratch + at.raw + item * a.dv;
    float ss = 0.f;
    for (int c = lane; c < a.dv; c += 32) {
        ss = fmaf(o[c], o[c], ss);
    }
    const float inv = rsqrtf(warp_sum(ss) / float(a.dv) + a.eps);
    const T *gate = static_cast<const T *>(a.gate) + row * a.gate_stride + int64_t(head) * a.dv;
    const T *w = static_cast<const T *>(a.norm_w);
    T *out = static_cast<T *>(a.out) + row * a.out_stride + int64_t(head) * a.dv;
    for (int c = lane; c < a.dv; c += 32) {
        const float y = to_f32(gate[c]);
        out[c] = from_f32<T>(o[c] * inv * to_f32(w[c]) * (a.gate_silu ? silu(y) : sigmoid_of(y)));
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
void recurrent(cudaStream_t s, const GatedDeltaArgs &a, const DeltaScratch &at) {
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads), unsigned((a.dv + kRecCols - 1) / kRecCols));
    const int nr = (a.dk + kRecRowGroups - 1) / kRecRowGroups;
    if (nr <= 4) {
        gated_delta_recurrent_kernel<T, 4><<<grid, kRecThreads, 0, s>>>(a, at);
    } else if (nr <= 8) {
        gated_delta_recurrent_kernel<T, 8><<<grid, kRecThreads, 0, s>>>(a, at);
    } else if (nr <= 16) {
        gated_delta_recurrent_kernel<T, 16><<<grid, kRecThreads, 0, s>>>(a, at);
    } else if (nr <= 32) {
        gated_delta_recurrent_kernel<T, 32><<<grid, kRecThreads, 0, s>>>(a, at);
    } else {
        gated_delta_recurrent_kernel<T, 64><<<grid, kRecThreads, 0, s>>>(a, at);
    }
}

void check_args(const GatedDeltaArgs &a) {
    CHECK_ARGUMENT(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dk > 0 && a.dk <= 512 && a.dv > 0 && a.dv <= 2048 &&
                       a.taps > 0 && a.taps <= 1024 && (a.decay_w == nullptr || (a.rank > 0 && a.rank <= 2048)),
                   "gated delta rule: whole groups of heads, key size at most 512, value size and rank at most 2048");
    CHECK_ARGUMENT(int64_t(a.n_seqs) * a.heads <= 0x7fffffff, "gated delta rule: too many (sequence, head) pairs");
}

void single_tokens(stream_t stream, llaisysDataType_t dtype, const GatedDeltaArgs &a) {
    auto s = static_cast<cudaStream_t>(stream);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        const bool wide = a.dv % 4 == 0 && a.slot_stride % 4 == 0 && reinterpret_cast<uintptr_t>(a.state) % 16 == 0;
        const int groups = wide ? a.dv / 4 : a.dv;
        int row_groups = 1; // at least dk / 8, so that a thread holds at most 8 rows
        while (row_groups * 8 < a.dk) {
            row_groups *= 2;
        }
        int col_groups = 1;
        while (col_groups < groups && col_groups * row_groups < kDecodeThreads) {
            col_groups *= 2;
        }
        row_groups = kDecodeThreads / col_groups;
        const int nr = (a.dk + row_groups - 1) / row_groups;
        const int vec = wide ? 4 : 1;
        auto up4 = [](int n) { return size_t(n + 3) / 4 * 4; };
        const size_t floats = 3 * up4(a.dk) + 2 * up4(a.dv) + size_t(a.rank + 31) / 32 * 32 + up4(col_groups * vec) + size_t(kDecodeThreads) * vec;
        const bool wide_decay = a.decay_ld * sizeof(T) % 16 == 0 && reinterpret_cast<uintptr_t>(a.decay_w) % 16 == 0;
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3(unsigned(a.n_seqs) * unsigned(a.heads));
        cfg.blockDim = dim3(kDecodeThreads);
        cfg.dynamicSmemBytes = floats * sizeof(float); // at most 1536 + 4096 + 2048 + 2048 + 2048 floats
        cfg.stream = s;
        cudaLaunchAttribute attr{};
        attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr.val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = &attr;
        cfg.numAttrs = 1;
        auto pick = [&](auto vec) {
            constexpr int V = decltype(vec)::value;
            return nr <= 2 ? gated_delta_decode_kernel<T, V, 2>
                           : (nr <= 4 ? gated_delta_decode_kernel<T, V, 4> : gated_delta_decode_kernel<T, V, 8>);
        };
        auto kernel = wide ? pick(std::integral_constant<int, 4>{}) : pick(std::integral_constant<int, 1>{});
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, GatedDeltaArgs(a), int(col_groups), int(wide_decay)));
    });
}

} // namespace

size_t gated_delta_state_floats(size_t heads, size_t kv_heads, size_t dk, size_t dv, size_t taps) {
    return heads * dk * dv + taps * (2 * kv_heads * dk + heads * dv);
}

size_t gated_delta_scratch_floats(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t kv_heads, size_t dk, size_t dv) {
    return size_t(delta_scratch(dtype, int64_t(n_rows), int64_t(heads), int64_t(kv_heads), int64_t(dk), int64_t(dv)).total);
}

void gated_delta_decode(stream_t stream, llaisysDataType_t dtype, const GatedDeltaArgs &args) {
    if (args.n_seqs == 0) {
        return;
    }
    check_args(args);
    GatedDeltaArgs a = args;
    a.q_starts = nullptr; // row i is sequence i's
    single_tokens(stream, dtype, a);
    check_launch("gated_delta_decode");
}

void gated_delta_chunk(stream_t stream, llaisysDataType_t dtype, const GatedDeltaArgs &a) {
    if (a.n_seqs == 0 || a.n_rows == 0) {
        return;
    }
    check_args(a);
    const DeltaScratch at = delta_scratch(dtype, a.n_rows, a.heads, a.kv_heads, a.dk, a.dv);
    CHECK_ARGUMENT(a.scratch != nullptr && reinterpret_cast<uintptr_t>(a.scratch) % 16 == 0 && a.scratch_floats >= size_t(at.total),
                   "gated delta rule: scratch missing, unaligned or too small");
    auto s = static_cast<cudaStream_t>(stream);
    const bool tiles = gated_delta_tiles_fit(dtype, a.dk, a.dv);
    dispatch(dtype, [&](auto tag) {
        using T = decltype(tag);
        auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
        const bool wide = a.dk % 4 == 0 && a.dv % 4 == 0 && a.row_stride % 4 == 0 && a.q_at % 4 == 0 && a.k_at % 4 == 0 && a.v_at % 4 == 0 &&
                          aligned(a.proj);
        const dim3 grid(unsigned((a.n_rows + kStrip - 1) / kStrip), unsigned((2 * a.kv_heads + a.heads) / kPrepWarps + 1));
        auto prepare = a.taps <= 4 ? (wide ? gated_delta_prepare_kernel<T, 4, 4> : gated_delta_prepare_kernel<T, 1, 4>)
                                   : (wide ? gated_delta_prepare_kernel<T, 4, 0> : gated_delta_prepare_kernel<T, 1, 0>);
        prepare<<<grid, kPrepWarps * 32, 0, s>>>(a, at);
        if (tiles) {
            gated_delta_tiles(stream, a);
        } else {
            gated_delta_decay_kernel<T><<<unsigned(a.n_rows), 128, size_t(a.rank) * sizeof(float), s>>>(a, at);
            recurrent<T>(s, a, at);
        }
        if (!tiles || a.dv > 128) { // (rows of single tokens hold nothing yet: the next kernel writes them)
            const int64_t items = int64_t(a.n_rows) * a.heads;
            gated_delta_out_kernel<T><<<unsigned((items + 7) / 8), 256, 0, s>>>(a, at);
        }
    });
    single_tokens(stream, dtype, a); // and the newest convolution inputs of every run
    check_launch("gated_delta_chunk");
}

} // namespace llaisys::kernels
