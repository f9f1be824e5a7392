// Gated delta rule over runs of tokens on the tensor cores, 32 tokens (a TILE) at a time.
//
// With b_t = sum of log2 decays up to token t (per key channel) and a reference m between 0 and b_end,
//     q^_t = q_t 2^(b_t - m),  k~_t = k_t 2^(b_t - m),  k^_s = k_s 2^(m - b_s),  S^ = 2^m S   (rows of S are key channels)
//     u_t = beta_t (v_t - S^^T k~_t - sum_{s<t} (k~_t . k^_s) u_s)
//     o_t = S^^T q^_t + sum_{s<=t} (q^_t . k^_s) u_s,     S_end = 2^(b_end - m) (S^ + sum_s k^_s u_s^T)
// which is the recurrence exactly. The corrections u solve a unit lower triangular system that does not depend on the value
// column: with A_ts = beta_t (k~_t . k^_s), s < t, they are U = (I + A)^-1 diag(beta) (V - K~ S^). One warp inverts I + A by
// forward substitution while the others multiply by the state. The split of the decays, its limit and the PIECES of a tile that
// decays more strongly are those of gated_linear_chunk.cu.
//
// Three barriers of the whole CTA divide a tile: (1) decays and operands of this tile, each warp for its own channels, and what
// is left to do for the outputs of the tile before; (2) everything that reads the old state, the triangular system beside it;
// (3) corrections, new state, outputs.
//
// Precision: the recurrence is f32. The tensor cores take 16-bit operands, so every f32 operand enters as the sum of two bf16
// numbers, a product of two such operands as its three leading terms; what is left out is below 2^-16 of a term. Accumulators,
// the state and the triangular inverse are f32.
//
// A CTA owns up to 128 value columns of one (sequence, head). The transposed state S^T [dv, dk] lives in its warps'
// accumulators, 16 value rows x half of the key channels each, and doubles as the A operand of both products with it. The two
// warps of a row block ("half" 0 and 1) sum over different channels; half 0 turns both sums into the right-hand side V - K~ S^,
// each half solves for one 16-token block of U, and they pass operand fragments and sums to one another through shared memory
// in register order. The next tile's inputs arrive by cp.async under the current tile's products.
//
// Few (sequence, head) pairs leave SMs idle, so long runs are cut into SEGMENTS. What a segment does to the state is affine,
// S_end = M S_start + C: a first launch runs every segment from zero with its values (C) and from the identity without values
// (M), a scan over the segments gives their starting states, and the main launch runs all of them at once.
#include "gated_delta.cuh"
#include "kernels.hpp"
#include "linear_tiles.cuh"

#include <algorithm>
#include <mutex>
#include <type_traits>

namespace llaisys::kernels {

namespace {

constexpr int kTile = 32;
constexpr float kMaxDecay = 80.f;       // log2 units
constexpr float kMaxTokenDecay = 160.f; // log2: one token's decay is cut here, where it is zero in f32
constexpr int kMaxRank = 512;
constexpr int kMaxCtas = 148; // (pairs x segments) of a launch that is cut
constexpr int kMinSegments = 3; // M and C cost a pass each: fewer segments do not pay
constexpr int kAStride = 36;  // floats per column of A
constexpr float kLog2e = 1.4426950408889634f;

template <int DK, int DV>
struct DeltaSmem { // byte offsets
    static constexpr int kWarps = DV / 8, kRowBlocks = DV / 16;
    static constexpr int kSplit = kWarps == 16 ? 4 : 2;         // warps per 16 x 16 block of A, each with a share of the channels
    static constexpr int kOperand = 2 * kTile * DK * 2;         // high and low
    static constexpr int kQ = 0;                                // convolved q, k [32][DK] bf16, swizzled
    static constexpr int kK = kQ + kTile * DK * 2;
    static constexpr int kV = kK + kTile * DK * 2;              // v, two buffers [32][DV] bf16, swizzled
    static constexpr int kB = kV + 2 * kTile * DV * 2;          // running sums of the tile's log2 decays [channels / 8][32][8] f32
    static constexpr int kQh = kB + kTile * DK * 4;             // q^ [32][DK] bf16, swizzled, high and low
    static constexpr int kKh = kQh + kOperand;                  // k^
    static constexpr int kKt = kKh + kOperand;                  // k~
    static constexpr int kO = kKt + kOperand;                   // o [32][DV] f32
    static constexpr int kS = kO + kTile * DV * 4;              // q^ . k^ [32][32] bf16, high and low
    static constexpr int kT = kS + 2 * kTile * kTile * 2;       // (I + A)^-1 diag(beta), the same
    static constexpr int kInv = kT + 2 * kTile * kTile * 2;     // inverse of the second diagonal block, by columns [16][16] f32
    static constexpr int kX = kInv + 16 * 16 * 4;               // half 1's sums: [row block][8-token group][lane] float4
    static constexpr int kF = kX + kRowBlocks * 4 * 512;        // fragments, per row block: [R block 0 | U block 0 | U block 1][high, low][lane]
    static constexpr int kFragments = kRowBlocks * 3 * 2 * 512;
    static constexpr int kA = kF;                               // before them: shares of A, column s at kAStride s, f32
    static constexpr int kShare = kTile * kAStride * 4;
    static_assert(kSplit * kShare <= kFragments, "A fits where the fragments come later");
    static constexpr int kG = kF + kFragments;                  // output gates of the tile [32][DV] bf16
    static constexpr int kScal = kG + kTile * DV * 2;           // per token, two buffers: q factor, k factor, beta, log decay [4][32] f32
    static constexpr int kNorm = kScal + 2 * 4 * kTile * 4;     // output norm [DV] f32
    static constexpr int kBias = kNorm + DV * 4;                // decay biases [DK] f32
    static constexpr int kIn = kBias + DK * 4;                  // per channel: the factors of S on the way into the tile's frame
    static constexpr int kOut = kIn + DK * 4;                   // and out of it
    static constexpr int kZ = kOut + DK * 4;                    // low-rank decay inputs [32][rank, padded to 16] bf16, swizzled; then
                                                                // decay weights as fragments [16 ranks][8 channels][lane] 8 bytes
};

// 16-byte chunk `chunk` of row `row` of a matrix with 64-byte rows
__device__ __forceinline__ uint32_t swz64(int row, int chunk) { return uint32_t(row * 64 + ((chunk ^ ((row >> 1) & 3)) << 4)); }

__device__ __forceinline__ void cp_async_4(uint32_t dst, const void *src, int src_bytes) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}

// log2(1 + e^x) = max(x, 0) log2 e + log2(1 + 2^(-|x| log2 e)). Its error, a few 2^-24 of absolute size, is that of rounding the
// decay itself to f32.
__device__ __forceinline__ float softplus_log2(float x) {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(1.f + ex2(fabsf(x) * -kLog2e)));
    return fmaf(fmaxf(x, 0.f), kLog2e, y);
}

__device__ __forceinline__ void mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0,
                                     uint32_t bl1) {
    mma_bf16(d, ah, bh0, bh1);
    mma_bf16(d, al, bh0, bh1);
    mma_bf16(d, ah, bl0, bl1);
}

// T = (I + A)^-1 diag(beta) of 32 tokens by one warp. A / beta by columns in kSplit shares `share` floats apart (below the diagonal;
// the rest means nothing), summed into the first; two diagonal
// blocks of 16 by forward substitution (lane: one column of one block), then T_10 = -T_11 A_10 T_00. high / low: T as two bf16
// matrices, swizzled; the block above the diagonal is never read.
template <int kSplit>
__device__ __forceinline__ void invert(float *s_a, int share, float *s_inv, const float *s_beta, unsigned char *high, int lane) {
    const int blk = lane >> 4, c = lane & 15;
    auto put = [&](int t, int col, float v) {
        const uint32_t u = __float_as_uint(v);
        const uint32_t at = swz64(t, col >> 3) + (col & 7) * 2;
        *reinterpret_cast<uint16_t *>(high + at) = uint16_t(u >> 16);
        *reinterpret_cast<__nv_bfloat16 *>(high + kTile * kTile * 2 + at) = __float2bfloat16_rn(v - __uint_as_float(u & 0xffff0000u));
    };
#pragma unroll
    for (int u = 0; u < 6; ++u) { // columns 0 .. 15 have eight groups of four rows, columns 16 .. 31 the last four of them
        const int at = u * 32 + lane, s = at < 128 ? at >> 3 : 16 + ((at - 128) >> 2), t = (at < 128 ? at & 7 : 4 + (at & 3)) * 4;
        float *p = s_a + s * kAStride + t;
        float4 v = *reinterpret_cast<const float4 *>(p);
        const float4 b = *reinterpret_cast<const float4 *>(s_beta + t);
#pragma unroll
        for (int w = 1; w < kSplit; ++w) {
            const float4 more = *reinterpret_cast<const float4 *>(p + w * share);
            v.x += more.x, v.y += more.y, v.z += more.z, v.w += more.w;
        }
        *reinterpret_cast<float4 *>(p) = make_float4(v.x * b.x, v.y * b.y, v.z * b.z, v.w * b.w);
    }
    __syncwarp();
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
        x[t] = t == c ? 1.f : 0.f;
    }
#pragma unroll
    for (int s = 0; s < 15; ++s) {
        const float *col = s_a + (blk * 16 + s) * kAStride + blk * 16;
        float a[16];
#pragma unroll
        for (int t = (s + 1) / 4 * 4; t < 16; t += 4) {
            *reinterpret_cast<float4 *>(a + t) = *reinterpret_cast<const float4 *>(col + t);
        }
#pragma unroll
        for (int t = s + 1; t < 16; ++t) {
            x[t] = fmaf(-a[t], x[s], x[t]);
        }
    }
    const float beta = s_beta[blk * 16 + c];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
        put(blk * 16 + t, blk * 16 + c, x[t] * beta);
    }
    if (blk == 1) {
#pragma unroll
        for (int t = 0; t < 16; t += 4) {
            *reinterpret_cast<float4 *>(s_inv + c * 16 + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
        }
    }
    __syncwarp();
    // lane (blk, c): rows 8 blk .. 8 blk + 7 of column c of A_10 T_00, then of -T_11 times that
    float y[8] = {}, z[8] = {};
#pragma unroll
    for (int s = 0; s < 16; ++s) {
        const float xs = __shfl_sync(0xffffffffu, x[s], c);
        const float4 *a = reinterpret_cast<const float4 *>(s_a + s * kAStride + 16 + blk * 8);
        const float4 a0 = a[0], a1 = a[1];
        y[0] = fmaf(a0.x, xs, y[0]);
        y[1] = fmaf(a0.y, xs, y[1]);
        y[2] = fmaf(a0.z, xs, y[2]);
        y[3] = fmaf(a0.w, xs, y[3]);
        y[4] = fmaf(a1.x, xs, y[4]);
        y[5] = fmaf(a1.y, xs, y[5]);
        y[6] = fmaf(a1.z, xs, y[6]);
        y[7] = fmaf(a1.w, xs, y[7]);
    }
#pragma unroll
    for (int s = 0; s < 16; ++s) {
        const float ys = -__shfl_sync(0xffffffffu, y[s & 7], (s >> 3) * 16 + c);
        const float4 *a = reinterpret_cast<const float4 *>(s_inv + s * 16 + blk * 8);
        const float4 a0 = a[0], a1 = a[1];
        z[0] = fmaf(a0.x, ys, z[0]);
        z[1] = fmaf(a0.y, ys, z[1]);
        z[2] = fmaf(a0.z, ys, z[2]);
        z[3] = fmaf(a0.w, ys, z[3]);
        z[4] = fmaf(a1.x, ys, z[4]);
        z[5] = fmaf(a1.y, ys, z[5]);
        z[6] = fmaf(a1.z, ys, z[6]);
        z[7] = fmaf(a1.w, ys, z[7]);
    }
    const float beta0 = s_beta[c];
#pragma unroll
    for (int t = 0; t < 8; ++t) {
        put(16 + blk * 8 + t, c, z[t] * beta0);
    }
}

template <int DK, int DV, bool kStateOnly>
__global__ void __launch_bounds__(DV * 4)
    gated_delta_tile_kernel(GatedDeltaArgs a, DeltaScratch at, int segs, int seg_len, int dv_slices, int weights_in_smem) {
    using M = DeltaSmem<DK, DV>;
    constexpr int kThreads = DV * 4, kWarps = DV / 8, kRowBlocks = DV / 16;
    constexpr int kHalf = DK / 2, kNt = kHalf / 8; // channels of a warp in the products with the state, in 8-channel groups
    constexpr int kChunks = DK / 8;                // 8-channel groups of the decays and operands: one warp each, or two
    constexpr int kSplit = M::kSplit, kInvWarp = kWarps - 4; // the warp that inverts takes no share of A
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ int s_limit;
    const uint32_t sm = smem_u32(smem);
    float *s_b = reinterpret_cast<float *>(smem + M::kB);
    auto b_at = [](int t, int d) { return (d >> 3) * (kTile * 8) + t * 8 + ((d & 7) ^ (((t >> 2) & 1) << 2)); };
    float *s_in = reinterpret_cast<float *>(smem + M::kIn), *s_out = reinterpret_cast<float *>(smem + M::kOut);
    float *s_a = reinterpret_cast<float *>(smem + M::kA), *s_o = reinterpret_cast<float *>(smem + M::kO);
    float *s_norm = reinterpret_cast<float *>(smem + M::kNorm), *s_bias = reinterpret_cast<float *>(smem + M::kBias);
    auto o_at = [](int t, int c) { return t * DV + (c ^ (((t >> 1) & 3) << 3)); };

    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, q4 = lane & 3, lr = lane & 7, lm = lane >> 3;
    const int rb = warp % kRowBlocks, half = warp / kRowBlocks, d0 = half * kHalf; // value rows 16 rb .., channels d0 ..
    int x = int(blockIdx.x);
    const int seg = x % segs;
    x /= segs;
    const int head = x % a.heads, i = x / a.heads;
    // state-only launches: behind the value columns, the columns of the identity
    const bool identity = kStateOnly && int(blockIdx.y) >= dv_slices;
    const int col0 = (int(blockIdx.y) - (identity ? dv_slices : 0)) * DV, n_cols = min(DV, (identity ? a.dk : a.dv) - col0);
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
    float *slot = a.segments != nullptr ? a.segments + ((int64_t(i) * a.heads + head) * segs + seg) * (int64_t(a.dk) * a.dv + DK * DK)
                                        : nullptr;

    // ---- the state: s[nt] = S^T rows 16 rb + g (+ 8), channels d0 + 8 nt + 2 q4 (+ 1) -------------------------------------
    const float *from = kStateOnly ? nullptr : (segs > 1 ? slot : (fresh ? nullptr : state));
    float s[kNt][4];
#pragma unroll
    for (int nt = 0; nt < kNt; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = d0 + nt * 8 + 2 * q4 + (e & 1), c = rb * 16 + g + 8 * (e >> 1);
            s[nt][e] = from != nullptr && d < a.dk && c < n_cols ? from[int64_t(d) * a.dv + col0 + c]
                                                                 : (identity && d == col0 + c && c < n_cols ? 1.f : 0.f);
        }
    }

    const __nv_bfloat16 *conv = reinterpret_cast<const __nv_bfloat16 *>(a.scratch);
    const __nv_bfloat16 *z_rows = static_cast<const __nv_bfloat16 *>(a.proj) + a.a_at;
    const int kvh = head / (a.heads / a.kv_heads), nq = a.kv_heads * a.dk;
    const bool per_channel = a.decay_w != nullptr;
    const int rank_steps = per_channel ? (a.rank + 15) / 16 : 0;
    // decay weights of 8 channels x 16 ranks as a B fragment: channel 8 c + g, ranks 16 ks + 2 q4 (+ 8), two at a time
    auto decay_weights = [&](int ks, int c, uint32_t (&wb)[2]) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int d = c * 8 + g, r = ks * 16 + 2 * q4 + 8 * e;
            const uint16_t *w = reinterpret_cast<const uint16_t *>(a.decay_w) + (int64_t(head) * a.dk + d) * a.decay_ld + r;
            wb[e] = d < a.dk && r < a.rank ? uint32_t(w[0]) | (r + 1 < a.rank ? uint32_t(w[1]) << 16 : 0u) : 0u;
        }
    };
    unsigned char *s_w = smem + M::kZ + kTile * rank_steps * 32 + lane * 8;
    // place of 16-byte piece `chunk` of a token's decay inputs: eight rows in a row fall on different banks
    auto z_at = [&](int t, int chunk) {
        const int key = (rank_steps & 3) == 0 ? t & 7 : ((rank_steps & 1) == 0 ? (t >> 1) & 3 : (t >> 2) & 1);
        return uint32_t(M::kZ + t * rank_steps * 32 + ((chunk ^ key) << 4));
    };
    if (per_channel) {
        if (weights_in_smem) {
            for (int u = warp; u < rank_steps * kChunks; u += kWarps) {
                uint32_t wb[2];
                decay_weights(u / kChunks, u % kChunks, wb);
                *reinterpret_cast<uint2 *>(s_w + u * 256) = make_uint2(wb[0], wb[1]);
            }
        }
        for (int d = tid; d < DK; d += kThreads) {
            s_bias[d] = d < a.dk ? to_f32(static_cast<const __nv_bfloat16 *>(a.dt_bias)[int64_t(head) * a.dk + d]) : 0.f;
        }
    }
    if (!kStateOnly && dv_slices == 1) {
        for (int c = tid; c < DV; c += kThreads) {
            s_norm[c] = c < n_cols ? to_f32(static_cast<const __nv_bfloat16 *>(a.norm_w)[c]) : 0.f;
        }
    }
    const float minus_a = per_channel ? -expf(to_f32(static_cast<const __nv_bfloat16 *>(a.a_log)[head])) : 0.f;
    // inputs of a tile, by threads first, first + 1, .. of `threads`
    auto load_tile = [&](int t0, int buf, int first, int threads) {
        constexpr int kPieces = DK / 8, kVPieces = DV / 8;
        for (int u = first; u < kTile * kPieces; u += threads) {
            const int t = u / kPieces, c = u - t * kPieces;
            const int bytes = t0 + t < end && c * 8 < a.dk ? 16 : 0;
            const __nv_bfloat16 *src = bytes ? conv + int64_t(t0 + t) * at.conv_stride + int64_t(kvh) * a.dk + c * 8 : conv;
            const uint32_t to = swz(t, c, DK * 2);
            if (!kStateOnly) {
                cp_async_16(sm + M::kQ + to, src, bytes);
            }
            cp_async_16(sm + M::kK + to, bytes ? src + nq : conv, bytes);
        }
        if (per_channel) {
            const int z_pieces = rank_steps * 2;
            for (int u = first; u < kTile * z_pieces; u += threads) {
                const int t = u / z_pieces, c = u - t * z_pieces;
                const int bytes = t0 + t < end ? max(0, min(16, (a.rank - c * 8) * 2)) : 0;
                cp_async_16(sm + z_at(t, c), bytes ? z_rows + int64_t(t0 + t) * a.row_stride + c * 8 : z_rows, bytes);
            }
        }
        if (!identity) {
            for (int u = first; u < kTile * kVPieces; u += threads) {
                const int t = u / kVPieces, c = u - t * kVPieces;
                const int bytes = t0 + t < end && c * 8 < n_cols ? 16 : 0;
                cp_async_16(sm + M::kV + buf * (kTile * DV * 2) + swz(t, c, DV * 2),
                            bytes ? conv + int64_t(t0 + t) * at.conv_stride + 2 * nq + int64_t(head) * a.dv + col0 + c * 8 : conv, bytes);
            }
        }
        if (first < 4 * kTile) {
            const int which = first / kTile, t = first - which * kTile;
            const int64_t row = t0 + t;
            const int bytes = t0 + t < end ? 4 : 0;
            const float *src = which < 2 ? a.scratch + at.unit + row * 2 * a.kv_heads + which * a.kv_heads + kvh
                                         : a.scratch + (which == 2 ? at.beta : at.decay_log) + row * a.heads + head;
            cp_async_4(sm + M::kScal + (buf * 4 * kTile + first) * 4, bytes ? src : a.scratch, which == 3 && per_channel ? 0 : bytes);
        }
        cp_async_commit();
    };
    // the gates of the CURRENT tile, needed at its end: asked for together with the next tile's operands
    auto load_gates = [&](int t0, int first, int threads) {
        if (!kStateOnly && dv_slices == 1) {
            constexpr int kPieces = DV / 8;
            const __nv_bfloat16 *gate = static_cast<const __nv_bfloat16 *>(a.gate);
            for (int u = first; u < kTile * kPieces; u += threads) {
                const int t = u / kPieces, c = u - t * kPieces;
                const int bytes = t0 + t < end && c * 8 < n_cols ? 16 : 0;
                cp_async_16(sm + M::kG + u * 16, bytes ? gate + int64_t(t0 + t) * a.gate_stride + int64_t(head) * a.dv + c * 8 : gate, bytes);
            }
            cp_async_commit();
        }
    };
    if (identity) { // no values: both buffers stay zero
        for (int u = tid; u < 2 * kTile * DV / 8; u += kThreads) {
            *reinterpret_cast<uint4 *>(smem + M::kV + u * 16) = make_uint4(0, 0, 0, 0);
        }
    }
    load_tile(begin, 0, tid, kThreads);

    const int frag = rb * 3 * 2 * 512 + lane * 16; // this lane's place in the row block's fragments
    auto put_frag = [&](int which, const uint32_t (&hi)[4], const uint32_t (&lo)[4]) {
        unsigned char *p = smem + M::kF + frag + which * 1024;
        *reinterpret_cast<uint4 *>(p) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4 *>(p + 512) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    };
    auto get_frag = [&](int which, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
        const unsigned char *p = smem + M::kF + frag + which * 1024;
        const uint4 h = *reinterpret_cast<const uint4 *>(p), l = *reinterpret_cast<const uint4 *>(p + 512);
        hi[0] = h.x, hi[1] = h.y, hi[2] = h.z, hi[3] = h.w;
        lo[0] = l.x, lo[1] = l.y, lo[2] = l.z, lo[3] = l.w;
    };
    // accumulators of 16 value rows x two 8-token groups as A fragments of a 16-token step
    auto split_frag = [](const float (&c0)[4], const float (&c1)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
        split2(c0[0], c0[1], hi[0], lo[0]);
        split2(c0[2], c0[3], hi[1], lo[1]);
        split2(c1[0], c1[1], hi[2], lo[2]);
        split2(c1[2], c1[3], hi[3], lo[3]);
    };

    // running sums of the tile's log2 decays for 8 channels, by one warp: W z on the tensor cores (bf16 products in f32 are exact)
    // or the tokens' own, then a scan along the tokens
    auto decays = [&](int c, const float *s_scal) {
        if (per_channel) {
            float v[4][2]; // tokens 8 j + g, channels 8 c + 2 q4 (+ 1)
            {
                float acc[2][4] = {};
                for (int ks = 0; ks < rank_steps; ++ks) {
                    uint32_t wb[2];
                    if (weights_in_smem) {
                        const uint2 w = *reinterpret_cast<const uint2 *>(s_w + (ks * kChunks + c) * 256);
                        wb[0] = w.x, wb[1] = w.y;
                    } else {
                        decay_weights(ks, c, wb);
                    }
#pragma unroll
                    for (int mt = 0; mt < 2; ++mt) {
                        uint32_t za[4];
                        ldmatrix_x4(za, sm + z_at(mt * 16 + lr + 8 * (lm & 1), 2 * ks + (lm >> 1)));
                        mma_bf16(acc[mt], za, wb[0], wb[1]);
                    }
                }
                const float2 bias = *reinterpret_cast<const float2 *>(s_bias + c * 8 + 2 * q4);
                const bool real = c * 8 < a.dk; // (channels the model does not have keep factor 1; dk is a multiple of 8)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const float x = acc[j >> 1][2 * (j & 1) + e] + (e == 0 ? bias.x : bias.y);
                        v[j][e] = real ? fmaxf(softplus_log2(x) * minus_a, -kMaxTokenDecay) : 0.f;
                    }
                }
            }
#pragma unroll
            for (int off = 1; off < 8; off *= 2) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const float up = __shfl_up_sync(0xffffffffu, v[j][e], off * 4);
                        v[j][e] += g >= off ? up : 0.f;
                    }
                }
            }
            float base[2] = {0.f, 0.f};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float2 sum;
                sum.x = v[j][0] + base[0];
                sum.y = v[j][1] + base[1];
                *reinterpret_cast<float2 *>(s_b + b_at(8 * j + g, c * 8 + 2 * q4)) = sum;
                if (j < 3) {
                    base[0] += __shfl_sync(0xffffffffu, v[j][0], 28 + q4);
                    base[1] += __shfl_sync(0xffffffffu, v[j][1], 28 + q4);
                }
            }
        } else {
            float v = fmaxf(s_scal[3 * kTile + lane] * kLog2e, -kMaxTokenDecay);
#pragma unroll
            for (int off = 1; off < 32; off *= 2) {
                const float up = __shfl_up_sync(0xffffffffu, v, off);
                v += lane >= off ? up : 0.f;
            }
            const float4 all = make_float4(v, v, v, v);
            *reinterpret_cast<float4 *>(s_b + b_at(lane, c * 8)) = all;
            *reinterpret_cast<float4 *>(s_b + b_at(lane, c * 8 + 4)) = all;
        }
        __syncwarp();
    };
    // q^, k^ and k~ of 8 channels and tokens [p0, p1) (zero elsewhere), by one warp, and the factors of S; -> whether the piece's
    // decays are within the limit
    auto operands = [&](int c, int p0, int p1, const float *s_scal) {
        const int t = lane, mid = (p0 + p1 - 1) / 2;
        uint4 qh = make_uint4(0, 0, 0, 0), ql = qh, kh = qh, kl = qh, th = qh, tl = qh;
        const uint32_t to = swz(t, c, DK * 2);
        if (t >= p0 && t < p1) {
            const uint4 kw = *reinterpret_cast<const uint4 *>(smem + M::kK + to);
            uint4 qw = make_uint4(0, 0, 0, 0);
            if (!kStateOnly) {
                qw = *reinterpret_cast<const uint4 *>(smem + M::kQ + to);
            }
            const float fq = s_scal[t], fk = s_scal[kTile + t];
            const float4 b0 = *reinterpret_cast<const float4 *>(s_b + b_at(t, c * 8)), b1 = *reinterpret_cast<const float4 *>(s_b + b_at(t, c * 8 + 4));
            const float4 r0 = *reinterpret_cast<const float4 *>(s_b + b_at(mid, c * 8)), r1 = *reinterpret_cast<const float4 *>(s_b + b_at(mid, c * 8 + 4));
            auto pair = [&](uint32_t qp, uint32_t kp, float e0, float e1, uint32_t &qhi, uint32_t &qlo, uint32_t &khi, uint32_t &klo, uint32_t &thi,
                            uint32_t &tlo) {
                const float f0 = ex2(e0), f1 = ex2(e1), k0 = lo_half(kp) * fk, k1 = hi_half(kp) * fk;
                if (!kStateOnly) {
                    split2(lo_half(qp) * fq * f0, hi_half(qp) * fq * f1, qhi, qlo);
                }
                split2(k0 * f0, k1 * f1, thi, tlo);
                split2(k0 * ex2(-e0), k1 * ex2(-e1), khi, klo);
            };
            pair(qw.x, kw.x, b0.x - r0.x, b0.y - r0.y, qh.x, ql.x, kh.x, kl.x, th.x, tl.x);
            pair(qw.y, kw.y, b0.z - r0.z, b0.w - r0.w, qh.y, ql.y, kh.y, kl.y, th.y, tl.y);
            pair(qw.z, kw.z, b1.x - r1.x, b1.y - r1.y, qh.z, ql.z, kh.z, kl.z, th.z, tl.z);
            pair(qw.w, kw.w, b1.z - r1.z, b1.w - r1.w, qh.w, ql.w, kh.w, kl.w, th.w, tl.w);
        }
        if (!kStateOnly) {
            *reinterpret_cast<uint4 *>(smem + M::kQh + to) = qh;
            *reinterpret_cast<uint4 *>(smem + M::kQh + kTile * DK * 2 + to) = ql;
        }
        *reinterpret_cast<uint4 *>(smem + M::kKh + to) = kh;
        *reinterpret_cast<uint4 *>(smem + M::kKh + kTile * DK * 2 + to) = kl;
        *reinterpret_cast<uint4 *>(smem + M::kKt + to) = th;
        *reinterpret_cast<uint4 *>(smem + M::kKt + kTile * DK * 2 + to) = tl;
        bool ok = true;
        if (lane < 8) {
            const int d = c * 8 + lane;
            const float base = p0 > 0 ? s_b[b_at(p0 - 1, d)] : 0.f, ref = s_b[b_at(mid, d)], last_sum = s_b[b_at(p1 - 1, d)];
            s_in[d] = ex2(ref - base);
            s_out[d] = ex2(last_sum - ref);
            ok = last_sum - base >= -kMaxDecay;
        }
        return ok;
    };
    // norm, gate and store of a finished tile's o [token][value column]
    auto outputs = [&](int t0, int n) {
        constexpr int kRows = kTile / kWarps, kPer = DV / 32; // a warp's tokens side by side: their sums and exponentials overlap
        using F = Pieces<float, kPer>; // (the swizzle moves whole groups of eight columns)
        using P = Pieces<__nv_bfloat16, kPer>;
        const int c = lane * kPer;
        F v[kRows];
        float ss[kRows];
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            v[u] = *reinterpret_cast<const F *>(s_o + o_at(warp + u * kWarps, c));
            ss[u] = 0.f;
#pragma unroll
            for (int e = 0; e < kPer; ++e) {
                ss[u] = fmaf(v[u].v[e], v[u].v[e], ss[u]); // (columns past n_cols are zero)
            }
        }
        if (dv_slices > 1) { // the norm runs over more columns than this CTA has: a kernel of its own finishes
#pragma unroll
            for (int u = 0; u < kRows; ++u) {
                const int t = warp + u * kWarps;
                if (t < n && c < n_cols) {
                    *reinterpret_cast<F *>(a.scratch + at.raw + (int64_t(t0 + t) * a.heads + head) * a.dv + col0 + c) = v[u];
                }
            }
            return;
        }
#pragma unroll
        for (int o2 = 16; o2 > 0; o2 >>= 1) {
#pragma unroll
            for (int u = 0; u < kRows; ++u) {
                ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o2);
            }
        }
        const F norm = *reinterpret_cast<const F *>(s_norm + c);
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            const int t = warp + u * kWarps;
            const float inv = rsqrtf(ss[u] / float(a.dv) + a.eps);
            const P gate = *reinterpret_cast<const P *>(smem + M::kG + (t * DV + c) * 2);
            P y;
#pragma unroll
            for (int e = 0; e < kPer; ++e) {
                const float z = to_f32(gate.v[e]);
                y.v[e] = __float2bfloat16_rn(v[u].v[e] * inv * norm.v[e] * __fdividef(a.gate_silu ? z : 1.f, 1.f + ex2(fminf(z * -kLog2e, 120.f))));
            }
            if (t < n && c < n_cols) { // (n_cols is a multiple of 8)
                *reinterpret_cast<P *>(static_cast<__nv_bfloat16 *>(a.out) + int64_t(t0 + t) * a.out_stride + int64_t(head) * a.dv + c) = y;
            }
        }
    };

    int buf = 0;
    for (int t0 = begin; t0 < end; t0 += kTile, buf ^= 1) {
        const int n = min(kTile, end - t0);
        const uint32_t v_u32 = sm + M::kV + buf * (kTile * DV * 2);
        const float *s_scal = reinterpret_cast<const float *>(smem + M::kScal) + buf * 4 * kTile;
        float o[4][4]; // O^T rows 16 rb + g (+ 8), tokens 8 nt + 2 q4 (+ 1): this warp's share of the sum
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
        }
        cp_async_wait<0>();
        __syncthreads();
        bool ok = true;
        for (int c = warp; c < kChunks; c += kWarps) {
            decays(c, s_scal);
            ok = operands(c, 0, n, s_scal) && ok;
        }
        if (!kStateOnly && t0 > begin) {
            outputs(t0 - kTile, kTile);
        }
        const bool whole = __syncthreads_and(ok);
        for (int p0 = 0; p0 < n;) {
            int p1 = n;
            if (!whole) { // how many tokens from p0 on go together, and their operands
                if (tid == 0) {
                    s_limit = n;
                }
                __syncthreads();
                if (tid < DK) {
                    const float base = p0 > 0 ? s_b[b_at(p0 - 1, tid)] : 0.f;
                    int t = p0 + 1; // at least one token
                    while (t < n && s_b[b_at(t, tid)] - base >= -kMaxDecay) {
                        ++t;
                    }
                    atomicMin(&s_limit, t);
                }
                __syncthreads();
                p1 = s_limit;
                for (int c = warp; c < kChunks; c += kWarps) {
                    operands(c, p0, p1, s_scal);
                }
                __syncthreads();
            }
            // ---- the 16 x 16 blocks on and below the diagonal of k~ . k^ (a share of the channels per warp) and q^ . k^ -----------
            constexpr int kBlockTasks = 3 * kSplit;
            const int share_of = warp < kInvWarp ? warp : (warp == kInvWarp ? kBlockTasks : warp - 1);
            const int q_block = kWarps == 16 ? warp - 13 : (warp + 1) % 8;
            // one 16-channel step of a block: three products x two 8-key halves, six independent chains
            auto block_step = [&](int operand, int tb, int sb, int ks, float (&c)[6][4]) {
                const uint32_t qa = sm + operand + swz(tb * 16 + lr + 8 * (lm & 1), 2 * ks + (lm >> 1), DK * 2);
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
            };
            if (share_of < kBlockTasks) {
                const int w = share_of / kSplit, part = share_of % kSplit, tb = w > 0, sb = w > 1;
                constexpr int kSteps = DK / 16 / kSplit;
                float c[6][4] = {};
#pragma unroll
                for (int k1 = 0; k1 < kSteps; ++k1) {
                    block_step(M::kKt, tb, sb, part * kSteps + k1, c);
                }
#pragma unroll
                for (int h = 0; h < 2; ++h) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int t = tb * 16 + g + 8 * (e >> 1), sc = sb * 16 + h * 8 + 2 * q4 + (e & 1);
                        s_a[part * (M::kShare / 4) + sc * kAStride + t] = c[h][e] + (c[2 + h][e] + c[4 + h][e]);
                    }
                }
                named_barrier_arrive(1, (kBlockTasks + 1) * 32);
            } else if (warp == kInvWarp) {
                named_barrier_sync(1, (kBlockTasks + 1) * 32); // A is complete
                invert<kSplit>(s_a, M::kShare / 4, reinterpret_cast<float *>(smem + M::kInv), s_scal + 2 * kTile, smem + M::kT, lane);
            }
            if (!kStateOnly && q_block >= 0 && q_block < 3) {
                const int tb = q_block > 0, sb = q_block > 1;
                float c[6][4] = {};
#pragma unroll
                for (int ks = 0; ks < DK / 16; ++ks) {
                    block_step(M::kQh, tb, sb, ks, c);
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
                        const uint32_t to = M::kS + swz64(t, sb * 2 + h) + q4 * 4;
                        *reinterpret_cast<uint32_t *>(smem + to) = hi;
                        *reinterpret_cast<uint32_t *>(smem + to + kTile * kTile * 2) = lo;
                    }
                }
            }
            // ---- S^ = 2^m S, then S^^T k~ and O^T += S^^T q^ over this warp's channels: the accumulators are the A operand ----
#pragma unroll
            for (int nt = 0; nt < kNt; ++nt) {
                const float f0 = s_in[d0 + nt * 8 + 2 * q4], f1 = s_in[d0 + nt * 8 + 2 * q4 + 1];
                s[nt][0] *= f0;
                s[nt][1] *= f1;
                s[nt][2] *= f0;
                s[nt][3] *= f1;
            }
            float r[4][4] = {};
#pragma unroll
            for (int ks = 0; ks < kNt / 2; ++ks) {
                uint32_t ah[4], al[4];
                split_frag(s[2 * ks], s[2 * ks + 1], ah, al);
                auto product = [&](int operand, float (&d)[4][4]) {
                    uint32_t bh[2][4], bl[2][4];
#pragma unroll
                    for (int np = 0; np < 2; ++np) {
                        const uint32_t from_at = sm + operand + swz((np * 2 + (lm >> 1)) * 8 + lr, half * (kHalf / 8) + 2 * ks + (lm & 1), DK * 2);
                        ldmatrix_x4(bh[np], from_at);
                        ldmatrix_x4(bl[np], from_at + kTile * DK * 2);
                    }
#pragma unroll
                    for (int np = 0; np < 2; ++np) {
                        mma_bf16(d[2 * np], ah, bh[np][0], bh[np][1]);
                        mma_bf16(d[2 * np + 1], ah, bh[np][2], bh[np][3]);
                    }
#pragma unroll
                    for (int np = 0; np < 2; ++np) {
                        mma_bf16(d[2 * np], al, bh[np][0], bh[np][1]);
                        mma_bf16(d[2 * np + 1], al, bh[np][2], bh[np][3]);
                    }
#pragma unroll
                    for (int np = 0; np < 2; ++np) {
                        mma_bf16(d[2 * np], ah, bl[np][0], bl[np][1]);
                        mma_bf16(d[2 * np + 1], ah, bl[np][2], bl[np][3]);
                    }
                };
                product(M::kKt, r);
                if constexpr (!kStateOnly) {
                    product(M::kQh, o);
                }
            }
            float4 *s_x = reinterpret_cast<float4 *>(smem + M::kX) + rb * 4 * 32 + lane;
            if (half == 1) {
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    s_x[nt * 32] = make_float4(r[nt][0], r[nt][1], r[nt][2], r[nt][3]);
                }
            }
            __syncthreads();
            // ---- R = V - K~ S^ (half 0), U^T = R^T T^T: half 0 has tokens 16 .., half 1 tokens 0 .. 15 ---------------------------
            uint32_t uh[2][4], ul[2][4]; // by 16-token block
            {
                uint32_t rh[2][4], rl[2][4];
                if (half == 0) {
#pragma unroll
                    for (int nt = 0; nt < 4; ++nt) {
                        const float4 other = s_x[nt * 32];
                        r[nt][0] += other.x;
                        r[nt][1] += other.y;
                        r[nt][2] += other.z;
                        r[nt][3] += other.w;
                    }
#pragma unroll
                    for (int ks = 0; ks < 2; ++ks) {
                        uint32_t va[4];
                        ldmatrix_x4_trans(va, v_u32 + swz(ks * 16 + (lm >> 1) * 8 + lr, rb * 2 + (lm & 1), DV * 2));
#pragma unroll
                        for (int e = 0; e < 4; ++e) { // fragment register e: group 2 ks + e / 2, rows g + 8 (e % 2)
                            float(&c)[4] = r[2 * ks + (e >> 1)];
                            c[2 * (e & 1)] = lo_half(va[e]) - c[2 * (e & 1)];
                            c[2 * (e & 1) + 1] = hi_half(va[e]) - c[2 * (e & 1) + 1];
                        }
                        split_frag(r[2 * ks], r[2 * ks + 1], rh[ks], rl[ks]);
                    }
                    put_frag(0, rh[0], rl[0]);
                }
                if (half == 1 && p1 == n) { // half 1 waits for half 0 here: time to ask for what comes next
                    load_gates(t0, tid - kThreads / 2, kThreads / 2);
                    if (t0 + kTile < end) {
                        load_tile(t0 + kTile, buf ^ 1, tid - kThreads / 2, kThreads / 2); // q, k and z are used up; v and the scalars
                    }                                                                     // go to the other buffer
                }
                named_barrier_sync(2 + rb, 64); // the two warps of the row block
                if (half == 1) {
                    get_frag(0, rh[0], rl[0]);
                }
                const int mine = 1 - half;
                float u[2][4] = {};
#pragma unroll
                for (int ks = 0; ks < 2; ++ks) {
                    if (ks <= mine) {
                        const uint32_t from_at = sm + M::kT + swz64(mine * 16 + (lm >> 1) * 8 + lr, 2 * ks + (lm & 1));
                        uint32_t bh[4], bl[4];
                        ldmatrix_x4(bh, from_at);
                        ldmatrix_x4(bl, from_at + kTile * kTile * 2);
                        mma3(u[0], rh[ks], rl[ks], bh[0], bh[1], bl[0], bl[1]);
                        mma3(u[1], rh[ks], rl[ks], bh[2], bh[3], bl[2], bl[3]);
                    }
                }
                if (half == 0) {
                    split_frag(u[0], u[1], uh[1], ul[1]);
                    put_frag(2, uh[1], ul[1]);
                } else {
                    split_frag(u[0], u[1], uh[0], ul[0]);
                    put_frag(1, uh[0], ul[0]);
                }
                named_barrier_sync(2 + rb, 64);
                if (half == 0) {
                    get_frag(1, uh[0], ul[0]);
                } else {
                    get_frag(2, uh[1], ul[1]);
                }
            }
            // ---- S^T += U^T k^ over this warp's channels, then S = 2^(b_end - m) S^ ------------------------------------
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                uint32_t bh[kNt / 2][4], bl[kNt / 2][4];
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    const uint32_t from_at = sm + M::kKh + swz(ks * 16 + (lm & 1) * 8 + lr, half * (kHalf / 8) + np * 2 + (lm >> 1), DK * 2);
                    ldmatrix_x4_trans(bh[np], from_at);
                    ldmatrix_x4_trans(bl[np], from_at + kTile * DK * 2);
                }
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    mma_bf16(s[2 * np], uh[ks], bh[np][0], bh[np][1]);
                    mma_bf16(s[2 * np + 1], uh[ks], bh[np][2], bh[np][3]);
                }
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    mma_bf16(s[2 * np], ul[ks], bh[np][0], bh[np][1]);
                    mma_bf16(s[2 * np + 1], ul[ks], bh[np][2], bh[np][3]);
                }
#pragma unroll
                for (int np = 0; np < kNt / 2; ++np) {
                    mma_bf16(s[2 * np], uh[ks], bl[np][0], bl[np][1]);
                    mma_bf16(s[2 * np + 1], uh[ks], bl[np][2], bl[np][3]);
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
                // ---- O^T += U^T (q^ . k^)^T: half 0 adds the keys 16 .., half 1 the keys 0 .. 15 ---------------------------------
                auto scores = [&](const uint32_t (&h)[4], const uint32_t (&l)[4], int tb, int sb) {
                    const uint32_t from_at = sm + M::kS + swz64(tb * 16 + (lm >> 1) * 8 + lr, 2 * sb + (lm & 1));
                    uint32_t bh[4], bl[4];
                    ldmatrix_x4(bh, from_at);
                    ldmatrix_x4(bl, from_at + kTile * kTile * 2);
                    mma3(o[2 * tb], h, l, bh[0], bh[1], bl[0], bl[1]);
                    mma3(o[2 * tb + 1], h, l, bh[2], bh[3], bl[2], bl[3]);
                };
                if (half == 0) {
                    scores(uh[1], ul[1], 1, 1);
                } else {
                    scores(uh[0], ul[0], 0, 0);
                    scores(uh[0], ul[0], 1, 0);
                }
            }
            if (p1 < n) {
                __syncthreads(); // the next piece rewrites the operands, the scores and the channel values
            }
            p0 = p1;
        }
        if constexpr (!kStateOnly) {
            // ---- o of both halves, [token][value column]; norm, gate and store follow behind the next barrier -----------------------
            float4 *s_x = reinterpret_cast<float4 *>(smem + M::kX) + rb * 4 * 32 + lane;
            if (half == 1) {
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    s_x[nt * 32] = make_float4(o[nt][0], o[nt][1], o[nt][2], o[nt][3]);
                }
            }
            named_barrier_sync(2 + rb, 64);
            if (half == 0) {
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    const float4 other = s_x[nt * 32];
                    const int t = nt * 8 + 2 * q4, c = rb * 16 + g;
                    s_o[o_at(t, c)] = o[nt][0] + other.x;
                    s_o[o_at(t + 1, c)] = o[nt][1] + other.y;
                    s_o[o_at(t, c + 8)] = o[nt][2] + other.z;
                    s_o[o_at(t + 1, c + 8)] = o[nt][3] + other.w;
                }
            }
        }
    }
    if constexpr (!kStateOnly) {
        cp_async_wait<0>(); // the last tile's gates
        __syncthreads();
        const int t0 = begin + (end - 1 - begin) / kTile * kTile;
        outputs(t0, end - t0);
    }

    if (identity) { // M as A fragments (high, low), behind the segment's C: pairs along its columns, transposed across the warp
        uint4 *m = reinterpret_cast<uint4 *>(slot + int64_t(a.dk) * a.dv) + lane;
#pragma unroll
        for (int u = 0; u < kNt / 2; ++u) {
            uint32_t hi[4], lo[4];
            split2(s[2 * u][0], s[2 * u][1], hi[0], lo[0]);
            split2(s[2 * u + 1][0], s[2 * u + 1][1], hi[1], lo[1]);
            split2(s[2 * u][2], s[2 * u][3], hi[2], lo[2]);
            split2(s[2 * u + 1][2], s[2 * u + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                hi[e] = movmatrix_trans(hi[e]);
                lo[e] = movmatrix_trans(lo[e]);
            }
            const int at16 = ((half * (kNt / 2) + u) * (DK / 16) + col0 / 16 + rb) * 2; // 16 rows x 16 columns of M
            if (col0 + rb * 16 < DK) {
                m[at16 * 32] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                m[(at16 + 1) * 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        }
        return;
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
}

// Slots of a sequence hold what each segment does to the state, C [dk, dv] f32 and M as operand fragments; afterwards their first
// part holds each segment's starting state. A CTA follows 16 value columns through all segments, a warp per 16 rows of the
// state: S_{j+1} = M_j S_j + C_j with both factors as two bf16 numbers. A fragment of M is replaced by the next segment's as soon
// as it has been used.
template <int DK>
__global__ void __launch_bounds__(DK * 2) gated_delta_scan_kernel(GatedDeltaArgs a, int segs, int seg_len) {
    constexpr int kSteps = DK / 16;
    __shared__ uint2 s_s[2][kSteps][2][2][32]; // S as B fragments: two buffers, [16 rows][8 columns][high, low][lane]
    const int head = int(blockIdx.x) % a.heads, i = int(blockIdx.x) / a.heads;
    const int len = a.q_starts[i + 1] - a.q_starts[i];
    if (len < 2) {
        return;
    }
    const int n = (len + seg_len - 1) / seg_len;
    const int64_t size = int64_t(a.dk) * a.dv, stride = size + DK * DK;
    float *slots = a.segments + (int64_t(i) * a.heads + head) * segs * stride;
    const float *state = a.state + int64_t(a.seq_ids[i]) * a.slot_stride + int64_t(head) * size;
    const bool fresh = a.kv_lens[i] == len;
    const int warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31, g = lane >> 2, q4 = lane & 3;
    const int col = int(blockIdx.y) * 16 + 2 * q4;
    // this lane's rows 16 warp + g (+ 8), columns col (+ 1) of both 8-column groups
    auto each = [&](auto &&body) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = warp * 16 + g + 8 * h, c = col + nt * 8;
                body(nt, h, int64_t(d) * a.dv + c, d < a.dk && c < a.dv);
            }
        }
    };
    auto load = [&](const float *p, bool there, float (&x)[2][4]) { // (dv is even: both columns are there, or neither)
        each([&](int nt, int h, int64_t at, bool in) {
            const float2 v = in && there ? *reinterpret_cast<const float2 *>(p + at) : make_float2(0.f, 0.f);
            x[nt][2 * h] = v.x, x[nt][2 * h + 1] = v.y;
        });
    };
    auto fragments = [&](int j, int ks) { return reinterpret_cast<const uint4 *>(slots + j * stride + size) + ((warp * kSteps + ks) * 2) * 32 + lane; };
    float s[2][4], next[2][4];
    load(state, !fresh, s);
    load(slots, n > 1, next);
    uint4 mh[kSteps], ml[kSteps];
#pragma unroll
    for (int ks = 0; ks < kSteps; ++ks) {
        mh[ks] = n > 1 ? fragments(0, ks)[0] : make_uint4(0, 0, 0, 0);
        ml[ks] = n > 1 ? fragments(0, ks)[32] : make_uint4(0, 0, 0, 0);
    }
    for (int j = 0; j < n; ++j) {
        each([&](int nt, int h, int64_t at, bool in) {
            if (in) {
                *reinterpret_cast<float2 *>(slots + j * stride + at) = make_float2(s[nt][2 * h], s[nt][2 * h + 1]);
            }
        });
        if (j + 1 == n) {
            break; // (nothing starts from what the last segment leaves)
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) { // rows of S become the summed dimension: transpose the pairs across the warp
            uint32_t h0, l0, h1, l1;
            split2(s[nt][0], s[nt][1], h0, l0);
            split2(s[nt][2], s[nt][3], h1, l1);
            s_s[j & 1][warp][nt][0][lane] = make_uint2(movmatrix_trans(h0), movmatrix_trans(h1));
            s_s[j & 1][warp][nt][1][lane] = make_uint2(movmatrix_trans(l0), movmatrix_trans(l1));
        }
        float after[2][4];
        load(slots + (j + 1) * stride, j + 2 < n, after); // C of the next segment
        __syncthreads();
        float low[2][4] = {}, high[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < kSteps; ++ks) {
            const uint32_t ah[4] = {mh[ks].x, mh[ks].y, mh[ks].z, mh[ks].w}, al[4] = {ml[ks].x, ml[ks].y, ml[ks].z, ml[ks].w};
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const uint2 bh = s_s[j & 1][ks][nt][0][lane], bl = s_s[j & 1][ks][nt][1][lane];
                mma_bf16(next[nt], ah, bh.x, bh.y);
                mma_bf16(low[nt], al, bh.x, bh.y);
                mma_bf16(high[nt], ah, bl.x, bl.y);
            }
            if (j + 2 < n) {
                mh[ks] = fragments(j + 1, ks)[0];
                ml[ks] = fragments(j + 1, ks)[32];
            }
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[nt][e] = next[nt][e] + (low[nt][e] + high[nt][e]);
                next[nt][e] = after[nt][e];
            }
        }
    }
}

template <int DK>
void launch_scan(cudaStream_t s, const GatedDeltaArgs &a, int segs, int seg_len) {
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads), unsigned((a.dv + 15) / 16));
    gated_delta_scan_kernel<DK><<<grid, DK * 2, 0, s>>>(a, segs, seg_len);
}

int64_t slot_floats(int64_t dk, int64_t dv) { return dk * dv + (dk <= 64 ? 64 * 64 : 128 * 128); }

template <int DK, int DV, bool kStateOnly>
void launch_tiles(cudaStream_t s, const GatedDeltaArgs &a, const DeltaScratch &at, int segs, int seg_len, int slices) {
    static std::once_flag once[64];
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    constexpr int kFixed = DeltaSmem<DK, DV>::kZ;
    constexpr int kMaxBytes = 227 * 1024 - 1024; // (the static shared memory beside it)
    static_assert(kFixed + kTile * kMaxRank * 2 <= kMaxBytes, "shared memory of one CTA");
    const int rank = a.decay_w != nullptr ? (a.rank + 15) / 16 * 16 : 0;
    const int without = kFixed + kTile * rank * 2, with = without + DK * rank * 2;
    const bool weights_in_smem = rank > 0 && with <= kMaxBytes && (kFixed > 113 * 1024 || with <= 113 * 1024); // (or one CTA less per SM)
    const int bytes = weights_in_smem ? with : without;
    std::call_once(once[dev & 63], [] {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(gated_delta_tile_kernel<DK, DV, kStateOnly>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxBytes));
    });
    const int extra = kStateOnly ? (a.dk + DV - 1) / DV : 0;
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads) * unsigned(segs), unsigned(slices + extra));
    gated_delta_tile_kernel<DK, DV, kStateOnly><<<grid, DV * 4, bytes, s>>>(a, at, segs, seg_len, slices, weights_in_smem ? 1 : 0);
}

} // namespace

size_t gated_delta_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv) {
    if (heads == 0 || !gated_delta_tiles_fit(dtype, int64_t(dk), int64_t(dv))) {
        return 0;
    }
    return size_t(kMaxCtas) * size_t(slot_floats(int64_t(dk), int64_t(dv))); // pairs x segments of a launch that is cut never exceed kMaxCtas
}

void gated_delta_tiles(stream_t stream, const GatedDeltaArgs &a) {
    auto s = static_cast<cudaStream_t>(stream);
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    CHECK_ARGUMENT(aligned(a.gate) && a.gate_stride % 8 == 0 && aligned(a.out) && a.out_stride % 8 == 0, "gated delta rule: gate and output rows must be 16-byte aligned");
    CHECK_ARGUMENT(a.decay_w == nullptr || (a.rank <= kMaxRank && aligned(a.proj) && a.row_stride % 8 == 0 && a.a_at % 8 == 0),
                   "gated delta rule: decay inputs must be 16-byte aligned, at most 512 per token");
    const DeltaScratch at = delta_scratch(LLAISYS_DTYPE_BF16, a.n_rows, a.heads, a.kv_heads, a.dk, a.dv);
    const int slices = (a.dv + 127) / 128;
    const int64_t pairs = int64_t(a.n_seqs) * a.heads;
    int64_t segs = std::min<int64_t>(kMaxCtas / (pairs * slices), (a.max_q_len + kTile - 1) / kTile);
    segs = a.segments == nullptr ? 1 : std::min(segs, int64_t(a.segment_floats) / (slot_floats(a.dk, a.dv) * pairs));
    int seg_len = (a.max_q_len + kTile - 1) / kTile * kTile;
    if (segs >= kMinSegments) {
        seg_len = int((a.max_q_len + segs * kTile - 1) / (segs * kTile)) * kTile;
        segs = (a.max_q_len + seg_len - 1) / seg_len;
    } else {
        segs = 1;
    }
    auto run = [&](auto state_only) {
        constexpr bool kOnly = decltype(state_only)::value;
        if (a.dk <= 64) {
            a.dv <= 64 ? launch_tiles<64, 64, kOnly>(s, a, at, int(segs), seg_len, slices)
                       : launch_tiles<64, 128, kOnly>(s, a, at, int(segs), seg_len, slices);
        } else {
            a.dv <= 64 ? launch_tiles<128, 64, kOnly>(s, a, at, int(segs), seg_len, slices)
                       : launch_tiles<128, 128, kOnly>(s, a, at, int(segs), seg_len, slices);
        }
    };
    if (segs > 1) {
        run(std::true_type{});
        a.dk <= 64 ? launch_scan<64>(s, a, int(segs), seg_len) : launch_scan<128>(s, a, int(segs), seg_len);
    }
    run(std::false_type{});
    check_launch("gated_delta_tiles");
}

} // namespace llaisys::kernels
