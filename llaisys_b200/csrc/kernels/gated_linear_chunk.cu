// Gated linear attention over runs of tokens on the tensor cores, 64 tokens (a TILE) at a time.
//
// With b_t = sum of log2 decays up to token t (per key channel d) and a reference m_d between 0 and b_end,
//     q^_t = q_t 2^(b_t - m),   k^_s = k_s 2^(m - b_s),   S^ = 2^m S   (rows of S are key channels)
//     o_t  = S^T' q^_t + sum_{s <= t} (q^_t . k^_s) v_s,      S_end = 2^(b_end - m) (S^ + sum_s k^_s v_s^T)
// which is the recurrence exactly: every factor 2^(b_t - b_s) is split in two. The split is safe as long as no channel's
// decay over the tokens taken together exceeds 2^-kMaxDecay (the factors stay below 2^kMaxDecay, the masked products too); a
// tile whose decay is stronger is processed in PIECES, as few as its decays allow, down to single tokens (factor 1).
//
// Precision: the recurrence is f32. The tensor cores take 16-bit operands, so every f32 operand (q^, k^, S^, the scores)
// enters as the sum of two bf16 numbers, a product of two such operands as its three leading terms; v is bf16 already.
// What is left out is below 2^-16 of a term. Accumulators and the state are f32.
//
// A CTA owns up to 128 value columns of one (sequence, head): the transposed state S^T [dv, dk] lives in its warps'
// accumulator registers (16 value rows x half of the key channels each) from the first tile to the last, and doubles as the
// A operand of S^T q^. The two warps of a row block sum over different halves of the channels (and of the keys, in the
// score product); their outputs are added when they leave. Raw q, k, v and decay inputs of the next tile arrive by cp.async under
// the current tile's products. (The kernel is latency-bound: with one warp per row block it had two warps per scheduler and
// took 1.8 times as long.)
//
// Few (sequence, head) pairs leave SMs idle, so long runs are cut into SEGMENTS: a first launch computes what every segment
// adds to the state from zero and how much it decays, a scan turns that into every segment's starting state, and the main
// launch runs all segments at once.
#include "gated_linear.cuh"
#include "kernels.hpp"
#include "linear_tiles.cuh"

#include <algorithm>
#include <mutex>

namespace llaisys::kernels {

namespace {

constexpr int kTile = 64;
constexpr float kMaxDecay = 80.f; // log2 units
constexpr float kMaxTokenDecay = 160.f; // log2: one token's decay is cut here, where it is zero in f32
constexpr int kMaxRank = 128;
constexpr int kMaxCtas = 296;     // (pairs x segments) of a launch that is cut: a wave or two

template <int DK, int DV>
struct ChunkSmem { // byte offsets
    static constexpr int kOperands = 4 * kTile * DK * 2;        // q^ and k^, high and low each
    static constexpr int kOutputs = 2 * kTile * DV * 4;         // o of both channel halves
    static constexpr int kQ = 0;                                // raw q, k [64][DK] bf16
    static constexpr int kK = kQ + kTile * DK * 2;
    static constexpr int kB = kK + kTile * DK * 2;              // running sums of the tile's log2 decays [64][DK] f32
    static constexpr int kV = kB + kTile * DK * 4;              // v, two buffers [64][DV] bf16, swizzled
    static constexpr int kQh = kV + 2 * kTile * DV * 2;         // q^ high, low [64][DK] bf16, swizzled
    static constexpr int kKh = kQh + 2 * kTile * DK * 2;        // k^ high, low
    static constexpr int kO = kQh;                              // o [half][64][DV] f32 over q^ and k^ once they are used up
    static constexpr int kA = kQh + (kOperands > kOutputs ? kOperands : kOutputs); // scores high, low [64][64] bf16, swizzled
    static constexpr int kG = kA + 2 * kTile * kTile * 2;       // output gates of the tile [64][DV] bf16
    static constexpr int kPart = kG + kTile * DV * 2;           // decay sums of the token parts [4][DK] f32
    static constexpr int kRef = kPart + 4 * DK * 4;             // per channel: the reference m, and the factors of S
    static constexpr int kIn = kRef + DK * 4;                   // on the way into its frame
    static constexpr int kOut = kIn + DK * 4;                   // and out of it
    static constexpr int kZ = kOut + DK * 4;                    // low-rank decay inputs [64][rank, padded to 16] bf16
};

template <int DK, int DV, bool kStateOnly>
__global__ void __launch_bounds__(DV * 4)
    gated_linear_tile_kernel(GatedLinearArgs a, int segs, int seg_len, int dv_slices) {
    using M = ChunkSmem<DK, DV>;
    constexpr int kThreads = DV * 4, kWarps = DV / 8, kRowBlocks = DV / 16;
    constexpr int kHalf = DK / 2, kNt = kHalf / 8; // channels of a warp, in 8-channel groups
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ int s_limit;
    const uint32_t sm = smem_u32(smem);
    float *s_b = reinterpret_cast<float *>(smem + M::kB), *s_part = reinterpret_cast<float *>(smem + M::kPart);
    auto b_at = [](int t, int d) { return t * DK + (d ^ (((t >> 1) & 3) << 3)); };
    float *s_ref = reinterpret_cast<float *>(smem + M::kRef), *s_in = reinterpret_cast<float *>(smem + M::kIn);
    float *s_out = reinterpret_cast<float *>(smem + M::kOut);

    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, q4 = lane & 3, lr = lane & 7, lm = lane >> 3;
    const int rb = warp % kRowBlocks, half = warp / kRowBlocks, d0 = half * kHalf; // value rows 16 rb .., channels d0 ..
    int x = int(blockIdx.x);
    const int seg = x % segs;
    x /= segs;
    const int head = x % a.heads, i = x / a.heads;
    const int col0 = int(blockIdx.y) * DV, n_cols = min(DV, a.dv - col0);
    const int row0 = a.q_starts[i], row1 = a.q_starts[i + 1];
    if (row1 - row0 < 2) {
        return; // single tokens are the decode kernel's
    }
    const int begin = row0 + seg * seg_len;
    if (begin >= row1) {
        return;
    }
    const int end = min(row1, begin + seg_len);
    const bool last = end == row1;
    if (kStateOnly && last) {
        return; // nothing starts from what the last segment leaves
    }
    const bool fresh = a.kv_lens[i] == row1 - row0;
    float *state = a.state + int64_t(a.seq_ids[i]) * a.slot_stride + int64_t(head) * a.dk * a.dv;
    float *slot = a.segments != nullptr
                      ? a.segments + (int64_t(i) * a.heads * segs + int64_t(head) * segs + seg) * (int64_t(a.dk) * a.dv + a.dk)
                      : nullptr;

    // ---- the state: s[nt] = S^T rows 16 rb + g (+ 8), channels d0 + 8 nt + 2 q4 (+ 1) -------------------------------------
    const float *from = kStateOnly ? nullptr : (segs > 1 ? slot : (fresh ? nullptr : state));
    float s[kNt][4];
#pragma unroll
    for (int nt = 0; nt < kNt; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = d0 + nt * 8 + 2 * q4 + (e & 1), c = rb * 16 + g + 8 * (e >> 1);
            s[nt][e] = from != nullptr && d < a.dk && c < n_cols ? from[int64_t(d) * a.dv + col0 + c] : 0.f;
        }
    }
    float decayed = 0.f; // log2 decay of the whole segment (thread = channel)

    const __nv_bfloat16 *proj = static_cast<const __nv_bfloat16 *>(a.proj);
    const int rank_steps = (a.rank + 15) / 16;
    // what a warp needs of the decay projection: its 16 channels' biases and weights (the first 16 ranks stay in registers)
    constexpr int kParts = kWarps / (DK / 16), kPartTiles = 8 / kParts; // token parts of a tile, 8-token groups per part
    const int ch0 = (warp % (DK / 16)) * 16, part = warp / (DK / 16);
    auto decay_weights = [&](int ks, uint32_t (&wa)[4]) {
#pragma unroll
        for (int e = 0; e < 4; ++e) { // rows ch0 + g (+ 8), ranks 16 ks + 2 q4 (+ 8), two at a time
            const int d = ch0 + g + 8 * (e & 1), r = ks * 16 + 2 * q4 + 8 * (e >> 1);
            const uint16_t *w = reinterpret_cast<const uint16_t *>(a.decay_w) + (int64_t(head) * a.dk + d) * a.rank + r;
            wa[e] = d < a.dk && r < a.rank ? uint32_t(w[0]) | (r + 1 < a.rank ? uint32_t(w[1]) << 16 : 0u) : 0u;
        }
    };
    uint32_t first_w[4];
    decay_weights(0, first_w);
    const float to_log2 = 1.4426950408889634f / a.tau;
    float bias[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int d = ch0 + g + 8 * h;
        bias[h] = d < a.dk ? to_f32(static_cast<const __nv_bfloat16 *>(a.decay_b)[int64_t(head) * a.dk + d]) : 0.f;
    }
    auto load_tile = [&](int t0, int buf) {
        constexpr int kPieces = DK / 8, kVPieces = DV / 8;
        for (int u = tid; u < kTile * kPieces; u += kThreads) {
            const int t = u / kPieces, c = u - t * kPieces;
            const int bytes = t0 + t < end && c * 8 < a.dk ? 16 : 0;
            const __nv_bfloat16 *src = bytes ? proj + int64_t(t0 + t) * a.row_stride + int64_t(head) * a.dk + c * 8 : proj;
            if (!kStateOnly) {
                cp_async_16(sm + M::kQ + u * 16, bytes ? src + a.q_at : proj, bytes);
            }
            cp_async_16(sm + M::kK + u * 16, bytes ? src + a.k_at : proj, bytes);
        }
        const int z_pieces = rank_steps * 2;
        for (int u = tid; u < kTile * z_pieces; u += kThreads) {
            const int t = u / z_pieces, c = u - t * z_pieces;
            const int bytes = t0 + t < end ? max(0, min(16, (a.rank - c * 8) * 2)) : 0;
            cp_async_16(sm + M::kZ + u * 16, bytes ? proj + int64_t(t0 + t) * a.row_stride + a.z_at + c * 8 : proj, bytes);
        }
        for (int u = tid; u < kTile * kVPieces; u += kThreads) {
            const int t = u / kVPieces, c = u - t * kVPieces;
            const int bytes = t0 + t < end && c * 8 < n_cols ? 16 : 0;
            cp_async_16(sm + M::kV + buf * (kTile * DV * 2) + swz(t, c, DV * 2),
                        bytes ? proj + int64_t(t0 + t) * a.row_stride + a.v_at + int64_t(head) * a.dv + col0 + c * 8 : proj, bytes);
        }
        cp_async_commit();
    };
    // the gates of the CURRENT tile, needed at its end: asked for together with the next tile's operands
    auto load_gates = [&](int t0) {
        if (!kStateOnly && dv_slices == 1) {
            constexpr int kPieces = DV / 8;
            for (int u = tid; u < kTile * kPieces; u += kThreads) {
                const int t = u / kPieces, c = u - t * kPieces;
                const int bytes = t0 + t < end && c * 8 < n_cols ? 16 : 0;
                cp_async_16(sm + M::kG + u * 16,
                            bytes ? proj + int64_t(t0 + t) * a.row_stride + a.g_at + int64_t(head) * a.dv + c * 8 : proj, bytes);
            }
            cp_async_commit();
        }
    };
    constexpr int kPer = DV / 32; // value columns per lane when outputs leave
    float norm_w[kPer];
#pragma unroll
    for (int e = 0; e < kPer; ++e) {
        norm_w[e] = !kStateOnly && dv_slices == 1 && lane * kPer + e < n_cols
                        ? to_f32(static_cast<const __nv_bfloat16 *>(a.norm_w)[lane * kPer + e]) * a.out_scale
                        : 0.f;
    }
    load_tile(begin, 0);

    int buf = 0;
    for (int t0 = begin; t0 < end; t0 += kTile, buf ^= 1) {
        const int n = min(kTile, end - t0);
        const uint32_t v_u32 = sm + M::kV + buf * (kTile * DV * 2);
        float o[8][4]; // O^T rows 16 rb + g (+ 8), tokens 8 nt + 2 q4 (+ 1): this warp's share of the sum
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
        }
        cp_async_wait<0>();
        __syncthreads();
        // ---- running sums of the log2 decays: W z on the tensor cores (16 channels x 8 tokens at a time, bf16 products in f32
        //      are exact), then a scan along the tokens. A warp does 16 channels of one part of the tile's tokens. ----------
        {
            float acc[kPartTiles][4] = {};
            for (int ks = 0; ks < rank_steps; ++ks) {
                uint32_t wa[4];
                if (ks == 0) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        wa[e] = first_w[e];
                    }
                } else {
                    decay_weights(ks, wa);
                }
#pragma unroll
                for (int nt = 0; nt < kPartTiles; ++nt) {
                    const int t = (part * kPartTiles + nt) * 8 + g;
                    const uint32_t *z = reinterpret_cast<const uint32_t *>(smem + M::kZ + (t * rank_steps + ks) * 32);
                    mma_bf16(acc[nt], wa, z[q4], z[q4 + 4]);
                }
            }
            float carry[2] = {0.f, 0.f};
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = ch0 + g + 8 * h;
#pragma unroll
                for (int nt = 0; nt < kPartTiles; ++nt) {
                    float l0 = fmaxf(log_sigmoid_fast(acc[nt][2 * h] + bias[h]) * to_log2, -kMaxTokenDecay);
                    float l1 = fmaxf(log_sigmoid_fast(acc[nt][2 * h + 1] + bias[h]) * to_log2, -kMaxTokenDecay);
                    float incl = l0 + l1;
                    const float up1 = __shfl_up_sync(0xffffffffu, incl, 1, 4);
                    incl += q4 >= 1 ? up1 : 0.f;
                    const float up2 = __shfl_up_sync(0xffffffffu, incl, 2, 4);
                    incl += q4 >= 2 ? up2 : 0.f;
                    const float before = __shfl_up_sync(0xffffffffu, incl, 1, 4);
                    acc[nt][2 * h] = carry[h] + (q4 >= 1 ? before : 0.f) + l0;
                    acc[nt][2 * h + 1] = acc[nt][2 * h] + l1;
                    carry[h] += __shfl_sync(0xffffffffu, incl, 3, 4);
                }
                if (kParts > 1 && q4 == 0) {
                    s_part[part * DK + d] = carry[h];
                }
            }
            if (kParts > 1) {
                __syncthreads();
            }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = ch0 + g + 8 * h;
                float base = 0.f;
                for (int u = 0; u < part; ++u) {
                    base += s_part[u * DK + d];
                }
#pragma unroll
                for (int nt = 0; nt < kPartTiles; ++nt) {
                    const int t = (part * kPartTiles + nt) * 8 + 2 * q4;
                    // (channels the model does not have keep factor 1)
                    s_b[b_at(t, d)] = d < a.dk ? acc[nt][2 * h] + base : 0.f;
                    s_b[b_at(t + 1, d)] = d < a.dk ? acc[nt][2 * h + 1] + base : 0.f;
                }
            }
            __syncthreads();
        }
        for (int p0 = 0; p0 < n;) {
            // ---- how many tokens from p0 on go together; the piece's reference and the factors of S -----------------------
            int p1 = n;
            {
                const float base = tid < DK && p0 > 0 ? s_b[b_at(p0 - 1, tid)] : 0.f;
                auto set = [&](int stop) {
                    const float ref = s_b[b_at((p0 + stop - 1) / 2, tid)], last_sum = s_b[b_at(stop - 1, tid)];
                    s_ref[tid] = ref;
                    s_in[tid] = ex2(ref - base);
                    s_out[tid] = ex2(last_sum - ref);
                    return last_sum - base;
                };
                float total = 0.f;
                if (tid < DK) {
                    total = set(n);
                }
                if (!__syncthreads_and(total >= -kMaxDecay)) {
                    if (tid == 0) {
                        s_limit = n;
                    }
                    __syncthreads();
                    if (tid < DK && total < -kMaxDecay) {
                        int t = p0 + 1; // at least one token
                        while (t < n && s_b[b_at(t, tid)] - base >= -kMaxDecay) {
                            ++t;
                        }
                        atomicMin(&s_limit, t);
                    }
                    __syncthreads();
                    p1 = s_limit;
                    if (tid < DK) {
                        total = set(p1);
                    }
                    __syncthreads();
                }
                decayed += total;
            }
            // ---- q^ and k^, zero outside the piece -------------------------------------------------------------------
            for (int u = tid; u < kTile * (DK / 8); u += kThreads) {
                const int t = u / (DK / 8), c = u - t * (DK / 8);
                uint4 qh = make_uint4(0, 0, 0, 0), ql = qh, kh = qh, kl = qh;
                if (t >= p0 && t < p1) {
                    const uint4 kw = *reinterpret_cast<const uint4 *>(smem + M::kK + u * 16);
                    uint4 qw = make_uint4(0, 0, 0, 0);
                    if (!kStateOnly) {
                        qw = *reinterpret_cast<const uint4 *>(smem + M::kQ + u * 16);
                    }
                    const float4 b0 = *reinterpret_cast<const float4 *>(s_b + b_at(t, c * 8));
                    const float4 b1 = *reinterpret_cast<const float4 *>(s_b + b_at(t, c * 8) + 4);
                    const float4 r0 = *reinterpret_cast<const float4 *>(s_ref + c * 8);
                    const float4 r1 = *reinterpret_cast<const float4 *>(s_ref + c * 8 + 4);
                    auto pair = [&](uint32_t qp, uint32_t kp, float e0, float e1, uint32_t &qhi, uint32_t &qlo, uint32_t &khi,
                                    uint32_t &klo) {
                        if (!kStateOnly) {
                            split2(lo_half(qp) * a.q_scale * ex2(e0), hi_half(qp) * a.q_scale * ex2(e1), qhi, qlo);
                        }
                        split2(lo_half(kp) * ex2(-e0), hi_half(kp) * ex2(-e1), khi, klo);
                    };
                    pair(qw.x, kw.x, b0.x - r0.x, b0.y - r0.y, qh.x, ql.x, kh.x, kl.x);
                    pair(qw.y, kw.y, b0.z - r0.z, b0.w - r0.w, qh.y, ql.y, kh.y, kl.y);
                    pair(qw.z, kw.z, b1.x - r1.x, b1.y - r1.y, qh.z, ql.z, kh.z, kl.z);
                    pair(qw.w, kw.w, b1.z - r1.z, b1.w - r1.w, qh.w, ql.w, kh.w, kl.w);
                }
                const uint32_t at = swz(t, c, DK * 2);
                if (!kStateOnly) {
                    *reinterpret_cast<uint4 *>(smem + M::kQh + at) = qh;
                    *reinterpret_cast<uint4 *>(smem + M::kQh + kTile * DK * 2 + at) = ql;
                }
                *reinterpret_cast<uint4 *>(smem + M::kKh + at) = kh;
                *reinterpret_cast<uint4 *>(smem + M::kKh + kTile * DK * 2 + at) = kl;
            }
            __syncthreads();
            if (p1 == n) {
                load_gates(t0);
            }
            if (p1 == n && t0 + kTile < end) {
                load_tile(t0 + kTile, buf ^ 1); // raw q, k and z are used up; v goes to the other buffer
            }
            // ---- S^ = 2^m S ------------------------------------------------------------------------------------------
#pragma unroll
            for (int nt = 0; nt < kNt; ++nt) {
                const float f0 = s_in[d0 + nt * 8 + 2 * q4], f1 = s_in[d0 + nt * 8 + 2 * q4 + 1];
                s[nt][0] *= f0;
                s[nt][1] *= f1;
                s[nt][2] *= f0;
                s[nt][3] *= f1;
            }
            if constexpr (!kStateOnly) {
                // ---- O^T += S^T q^ over this warp's channels: the accumulators are the A operand ---------------------------
#pragma unroll
                for (int ks = 0; ks < kNt / 2; ++ks) {
                    uint32_t ah[4], al[4], bh[4][4], bl[4][4];
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        const uint32_t at =
                            sm + M::kQh + swz((np * 2 + (lm >> 1)) * 8 + lr, half * (kHalf / 8) + 2 * ks + (lm & 1), DK * 2);
                        ldmatrix_x4(bh[np], at);
                        ldmatrix_x4(bl[np], at + kTile * DK * 2);
                    }
                    split2(s[2 * ks][0], s[2 * ks][1], ah[0], al[0]);
                    split2(s[2 * ks][2], s[2 * ks][3], ah[1], al[1]);
                    split2(s[2 * ks + 1][0], s[2 * ks + 1][1], ah[2], al[2]);
                    split2(s[2 * ks + 1][2], s[2 * ks + 1][3], ah[3], al[3]);
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        mma_bf16(o[2 * np], ah, bh[np][0], bh[np][1]);
                        mma_bf16(o[2 * np + 1], ah, bh[np][2], bh[np][3]);
                    }
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        mma_bf16(o[2 * np], al, bh[np][0], bh[np][1]);
                        mma_bf16(o[2 * np + 1], al, bh[np][2], bh[np][3]);
                    }
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        mma_bf16(o[2 * np], ah, bl[np][0], bl[np][1]);
                        mma_bf16(o[2 * np + 1], ah, bl[np][2], bl[np][3]);
                    }
                }
                // ---- scores q^_t . k^_s, s <= t, as two bf16 terms: the ten 16 x 16 blocks on and below the diagonal -------
                for (int w = warp; w < 10; w += kWarps) {
                    const int tb = w < 1 ? 0 : (w < 3 ? 1 : (w < 6 ? 2 : 3)), sb = w - tb * (tb + 1) / 2;
                    float c[6][4] = {}; // three products x two 8-key halves, summed below: six independent chains
#pragma unroll
                    for (int ks = 0; ks < DK / 16; ++ks) {
                        const uint32_t qa = sm + M::kQh + swz(tb * 16 + lr + 8 * (lm & 1), 2 * ks + (lm >> 1), DK * 2);
                        const uint32_t ka = sm + M::kKh + swz(sb * 16 + (lm >> 1) * 8 + lr, 2 * ks + (lm & 1), DK * 2);
                        uint32_t ah[4], al[4], bh[4], bl[4];
                        ldmatrix_x4(ah, qa);
                        ldmatrix_x4(bh, ka);
                        ldmatrix_x4(al, qa + kTile * DK * 2);
                        ldmatrix_x4(bl, ka + kTile * DK * 2);
                        mma_bf16(c[0], ah, bh[0], bh[1]);
                        mma_bf16(c[1], ah, bh[2], bh[3]);
                        mma_bf16(c[2], al, bh[0], bh[1]);
                        mma_bf16(c[3], al, bh[2], bh[3]);
                        mma_bf16(c[4], ah, bl[0], bl[1]);
                        mma_bf16(c[5], ah, bl[2], bl[3]);
                    }
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
#pragma unroll
                        for (int e = 0; e < 4; e += 2) {
                            const int t = tb * 16 + g + 4 * e, sc = sb * 16 + h * 8 + 2 * q4;
                            const float x0 = c[h][e] + (c[2 + h][e] + c[4 + h][e]);
                            const float x1 = c[h][e + 1] + (c[2 + h][e + 1] + c[4 + h][e + 1]);
                            uint32_t hi, lo;
                            split2(sc <= t ? x0 : 0.f, sc + 1 <= t ? x1 : 0.f, hi, lo);
                            const uint32_t at = M::kA + swz(t, sb * 2 + h, kTile * 2) + q4 * 4;
                            *reinterpret_cast<uint32_t *>(smem + at) = hi;
                            *reinterpret_cast<uint32_t *>(smem + at + kTile * kTile * 2) = lo;
                        }
                    }
                }
            }
            // ---- S^T += V^T k^ over this warp's channels, then S = 2^(b_end - m) S^ ------------------------------------
#pragma unroll
            for (int ks = 0; ks < kTile / 16; ++ks) {
                uint32_t va[4], bh[kNt / 2][4], bl[kNt / 2][4];
                ldmatrix_x4_trans(va, v_u32 + swz(ks * 16 + (lm >> 1) * 8 + lr, rb * 2 + (lm & 1), DV * 2));
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    const uint32_t at = sm + M::kKh + swz(ks * 16 + (lm & 1) * 8 + lr, half * (kHalf / 8) + np * 2 + (lm >> 1), DK * 2);
                    ldmatrix_x4_trans(bh[np], at);
                    ldmatrix_x4_trans(bl[np], at + kTile * DK * 2);
                }
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    mma_bf16(s[2 * np], va, bh[np][0], bh[np][1]);
                    mma_bf16(s[2 * np + 1], va, bh[np][2], bh[np][3]);
                }
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    mma_bf16(s[2 * np], va, bl[np][0], bl[np][1]);
                    mma_bf16(s[2 * np + 1], va, bl[np][2], bl[np][3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < kNt; ++nt) {
                const float f0 = s_out[d0 + nt * 8 + 2 * q4], f1 = s_out[d0 + nt * 8 + 2 * q4 + 1];
                s[nt][0] *= f0;
                s[nt][1] *= f1;
                s[nt][2] *= f0;
                s[nt][3] *= f1;
            }
            if constexpr (!kStateOnly) {
                __syncthreads(); // the scores are there; q^ and k^ are used up
                // ---- O^T += V^T A^T: the two warps of a row block take two 16-key steps each --------------------------------
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int ks = u == 0 ? half : 3 - half; // 0 and 3, 1 and 2: five blocks each below the diagonal
                    uint32_t va[4];
                    ldmatrix_x4_trans(va, v_u32 + swz(ks * 16 + (lm >> 1) * 8 + lr, rb * 2 + (lm & 1), DV * 2));
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        if (np >= ks) { // tokens 16 np .. see keys 16 ks ..
                            const uint32_t at = sm + M::kA + swz((np * 2 + (lm >> 1)) * 8 + lr, 2 * ks + (lm & 1), kTile * 2);
                            uint32_t bh[4], bl[4];
                            ldmatrix_x4(bh, at);
                            ldmatrix_x4(bl, at + kTile * kTile * 2);
                            mma_bf16(o[2 * np], va, bh[0], bh[1]);
                            mma_bf16(o[2 * np + 1], va, bh[2], bh[3]);
                            mma_bf16(o[2 * np], va, bl[0], bl[1]);
                            mma_bf16(o[2 * np + 1], va, bl[2], bl[3]);
                        }
                    }
                }
            }
            if (p1 < n) {
                __syncthreads(); // the next piece rewrites the operands, the scores and the channel values
            }
            p0 = p1;
        }
        if constexpr (!kStateOnly) {
            // ---- o [token][value column] through shared memory: norm, gate, store ------------------------------------------
            float *s_o = reinterpret_cast<float *>(smem + M::kO);
            auto o_at = [](int t, int c) { return t * DV + (c ^ (((t >> 1) & 3) << 3)); };
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s_o[half * (kTile * DV) + o_at(nt * 8 + 2 * q4 + (e & 1), rb * 16 + g + 8 * (e >> 1))] = o[nt][e];
                }
            }
            cp_async_wait<0>(); // the gates
            __syncthreads();
            // a warp's tokens side by side: their sums and exponentials overlap
            constexpr int kRows = kTile / kWarps;
            using F = Pieces<float, kPer>; // (the swizzle moves whole groups of eight columns)
            using P = Pieces<__nv_bfloat16, kPer>;
            const int c = lane * kPer;
            F v[kRows];
            float ss[kRows];
#pragma unroll
            for (int u = 0; u < kRows; ++u) {
                const int t = warp + u * kWarps;
                v[u] = *reinterpret_cast<const F *>(s_o + o_at(t, c));
                const F other = *reinterpret_cast<const F *>(s_o + kTile * DV + o_at(t, c));
                ss[u] = 0.f;
#pragma unroll
                for (int e = 0; e < kPer; ++e) {
                    v[u].v[e] += other.v[e];
                    ss[u] = fmaf(v[u].v[e], v[u].v[e], ss[u]); // (columns past n_cols are zero)
                }
            }
            if (dv_slices > 1) { // the norm runs over more columns than this CTA has: a kernel of its own finishes
#pragma unroll
                for (int u = 0; u < kRows; ++u) {
                    const int t = warp + u * kWarps;
                    if (t < n && c < n_cols) {
                        *reinterpret_cast<F *>(a.raw + (int64_t(t0 + t) * a.heads + head) * a.dv + col0 + c) = v[u];
                    }
                }
            } else {
#pragma unroll
                for (int o2 = 16; o2 > 0; o2 >>= 1) {
#pragma unroll
                    for (int u = 0; u < kRows; ++u) {
                        ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o2);
                    }
                }
#pragma unroll
                for (int u = 0; u < kRows; ++u) {
                    const int t = warp + u * kWarps;
                    const float inv = rsqrtf(ss[u] / float(a.dv) + a.eps);
                    const P gate = *reinterpret_cast<const P *>(smem + M::kG + (t * DV + c) * 2);
                    P y;
#pragma unroll
                    for (int e = 0; e < kPer; ++e) {
                        y.v[e] = __float2bfloat16_rn(v[u].v[e] * inv * norm_w[e] * silu_fast(to_f32(gate.v[e])));
                    }
                    if (t < n && c < n_cols) { // (n_cols is a multiple of 8)
                        *reinterpret_cast<P *>(static_cast<__nv_bfloat16 *>(a.out) + int64_t(t0 + t) * a.out_stride +
                                               int64_t(head) * a.dv + c) = y;
                    }
                }
            }
        }
    }

    float *to = kStateOnly ? slot : (last ? state : nullptr);
    if (to != nullptr) {
#pragma unroll
        for (int nt = 0; nt < kNt; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = d0 + nt * 8 + 2 * q4 + (e & 1), c = rb * 16 + g + 8 * (e >> 1);
                if (d < a.dk && c < n_cols) {
                    to[int64_t(d) * a.dv + col0 + c] = s[nt][e];
                }
            }
        }
    }
    if (kStateOnly && blockIdx.y == 0 && tid < a.dk && tid < DK) {
        slot[int64_t(a.dk) * a.dv + tid] = decayed;
    }
}

// Slots of a sequence hold what each segment adds and how it decays; afterwards they hold each segment's starting state.
__global__ void gated_linear_scan_kernel(GatedLinearArgs a, int segs, int seg_len) {
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int len = a.q_starts[i + 1] - a.q_starts[i];
    const int64_t size = int64_t(a.dk) * a.dv, stride = size + a.dk;
    const int64_t e = int64_t(blockIdx.y) * blockDim.x + threadIdx.x;
    if (len < 2 || e >= size) {
        return;
    }
    const int n = (len + seg_len - 1) / seg_len, d = int(e / a.dv);
    float *slot = a.segments + (int64_t(i) * a.heads + head) * segs * stride;
    float s = a.kv_lens[i] == len ? 0.f : a.state[int64_t(a.seq_ids[i]) * a.slot_stride + int64_t(head) * size + e];
    constexpr int kAtOnce = 8; // segments fetched together: the sums are a chain, the loads are not
    for (int j0 = 0; j0 < n; j0 += kAtOnce) {
        float add[kAtOnce], decay[kAtOnce];
#pragma unroll
        for (int u = 0; u < kAtOnce; ++u) {
            const bool used = j0 + u + 1 < n; // (nothing starts from what the last segment leaves)
            add[u] = used ? slot[(j0 + u) * stride + e] : 0.f;
            decay[u] = used ? slot[(j0 + u) * stride + size + d] : 0.f;
        }
#pragma unroll
        for (int u = 0; u < kAtOnce; ++u) {
            if (j0 + u < n) {
                slot[(j0 + u) * stride + e] = s;
                s = fmaf(s, ex2(decay[u]), add[u]);
            }
        }
    }
}

template <int DK, int DV, bool kStateOnly>
void launch_tiles(cudaStream_t s, const GatedLinearArgs &a, int segs, int seg_len, int slices) {
    static std::once_flag once[64];
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    constexpr int kFixed = ChunkSmem<DK, DV>::kZ;
    constexpr int kMaxBytes = kFixed + kTile * kMaxRank * 2;
    static_assert(kMaxBytes <= 227 * 1024, "shared memory of one CTA");
    const int bytes = kFixed + kTile * ((a.rank + 15) / 16 * 16) * 2;
    std::call_once(once[dev & 63], [] {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(gated_linear_tile_kernel<DK, DV, kStateOnly>,
                                                cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxBytes));
    });
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads) * unsigned(segs), unsigned(slices));
    gated_linear_tile_kernel<DK, DV, kStateOnly><<<grid, DV * 4, bytes, s>>>(a, segs, seg_len, slices);
}

int slices_of(int dv) { return (dv + 127) / 128; }

} // namespace

size_t gated_linear_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv) {
    if (dtype != LLAISYS_DTYPE_BF16 || heads == 0 || dk > 128) {
        return 0;
    }
    return size_t(kMaxCtas) * (dk * dv + dk); // pairs x segments of a launch that is cut never exceed kMaxCtas
}

bool gated_linear_tiles_apply(llaisysDataType_t dtype, const GatedLinearArgs &a) {
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    return dtype == LLAISYS_DTYPE_BF16 && a.rank <= kMaxRank && a.z_at % 8 == 0 && a.dk <= 128 && a.dk % 8 == 0 && a.dv % 8 == 0 && a.row_stride % 8 == 0 && a.q_at % 8 == 0 &&
           a.k_at % 8 == 0 && a.v_at % 8 == 0 && a.g_at % 8 == 0 && a.out_stride % 8 == 0 && aligned(a.proj) && aligned(a.out) &&
           aligned(a.norm_w);
}

void gated_linear_tiles(stream_t stream, const GatedLinearArgs &a) {
    auto s = static_cast<cudaStream_t>(stream);
    const int slices = slices_of(a.dv);
    const int64_t pairs = int64_t(a.n_seqs) * a.heads;
    // segments: as many as a wave of CTAs and the scratch hold, down to one tile each (the extra pass over the states runs on
    // SMs that would be idle: it costs about 0.6 of the main pass, so two segments already pay)
    const int64_t slot = int64_t(a.dk) * a.dv + a.dk;
    const int64_t wave = a.dk <= 64 && a.dv <= 64 ? kMaxCtas : kMaxCtas / 2;
    int64_t segs = std::min<int64_t>(wave / (pairs * slices), (a.max_q_len + kTile - 1) / kTile);
    segs = a.segments == nullptr ? 1 : std::min(segs, int64_t(a.segment_floats) / (slot * pairs));
    segs = std::max<int64_t>(segs, 1);
    int seg_len = (a.max_q_len + kTile - 1) / kTile * kTile;
    if (segs > 1) {
        seg_len = int((a.max_q_len + segs * kTile - 1) / (segs * kTile)) * kTile;
        segs = (a.max_q_len + seg_len - 1) / seg_len;
    }
    auto run = [&](auto state_only) {
        constexpr bool kOnly = decltype(state_only)::value;
        if (a.dk <= 64) {
            a.dv <= 64 ? launch_tiles<64, 64, kOnly>(s, a, int(segs), seg_len, slices)
                       : launch_tiles<64, 128, kOnly>(s, a, int(segs), seg_len, slices);
        } else {
            a.dv <= 64 ? launch_tiles<128, 64, kOnly>(s, a, int(segs), seg_len, slices)
                       : launch_tiles<128, 128, kOnly>(s, a, int(segs), seg_len, slices);
        }
    };
    if (segs > 1) {
        run(std::true_type{});
        const dim3 grid(unsigned(pairs), unsigned((int64_t(a.dk) * a.dv + 255) / 256));
        gated_linear_scan_kernel<<<grid, 256, 0, s>>>(a, int(segs), seg_len);
    }
    run(std::false_type{});
    check_launch("gated_linear_tiles");
}

} // namespace llaisys::kernels
