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
// A CTA owns 16 * warps value columns of one (sequence, head): the transposed state S^T [dv, dk] lives in its warps'
// accumulator registers (16 rows each) from the first tile to the last, and doubles as the A operand of S^T q^. Raw q, k,
// decays and v of the next tile arrive by cp.async under the current tile's products.
//
// Few (sequence, head) pairs leave SMs idle, so long runs are cut into SEGMENTS: a first launch computes what every segment
// adds to the state from zero and how much it decays, a scan turns that into every segment's starting state, and the main
// launch runs all segments at once.
#include "gated_linear.cuh"
#include "kernels.hpp"
#include "mma_utils.cuh"

#include <algorithm>
#include <mutex>

namespace llaisys::kernels {

namespace {

constexpr int kTile = 64;
constexpr float kMaxDecay = 80.f; // log2 units
constexpr int kMaxCtas = 296;     // (pairs x segments) of a launch that is cut: a wave or two

template <int DK, int DV>
struct ChunkSmem { // byte offsets
    static constexpr int kQ = 0;                                // raw q, k [64][DK] bf16
    static constexpr int kK = kQ + kTile * DK * 2;
    static constexpr int kB = kK + kTile * DK * 2;              // log2 decays, then their running sums [64][DK] f32
    static constexpr int kV = kB + kTile * DK * 4;              // v, two buffers [64][DV] bf16, swizzled
    static constexpr int kQh = kV + 2 * kTile * DV * 2;         // q^ high, low [64][DK] bf16, swizzled
    static constexpr int kKh = kQh + 2 * kTile * DK * 2;        // k^ high, low
    static constexpr int kO = kQh;                              // o [64][DV] f32 over q^ and k^ once they are used up
    static constexpr int kA = kKh + 2 * kTile * DK * 2;         // scores high, low [64][64] bf16, swizzled
    static constexpr int kRef = kA + 2 * kTile * kTile * 2;     // m and b_end per channel
    static constexpr int kEnd = kRef + DK * 4;
    static constexpr int kBytes = kEnd + DK * 4;
    static_assert(kTile * DV * 4 <= 4 * kTile * DK * 2, "o fits over q^ and k^");
};

__device__ __forceinline__ uint32_t swz(int row, int chunk, int row_bytes) { // 16-byte chunk `chunk` of row `row`
    return uint32_t(row * row_bytes + ((chunk ^ (row & 7)) << 4));
}
// x0, x1 as packed bf16 (x0 low half) and what is left of them after that rounding
__device__ __forceinline__ void split2(float x0, float x1, uint32_t &hi, uint32_t &lo) {
    hi = pack2<true>(x0, x1);
    lo = pack2<true>(x0 - __uint_as_float(hi << 16), x1 - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ float lo_half(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float hi_half(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

template <int DK, int DV, bool kStateOnly>
__global__ void __launch_bounds__(DV * 2)
    gated_linear_tile_kernel(GatedLinearArgs a, int segs, int seg_len, int dv_slices) {
    using M = ChunkSmem<DK, DV>;
    constexpr int kThreads = DV * 2, kWarps = DV / 16;
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ int s_limit;
    const uint32_t sm = smem_u32(smem);
    float *s_b = reinterpret_cast<float *>(smem + M::kB);
    float *s_ref = reinterpret_cast<float *>(smem + M::kRef), *s_end = reinterpret_cast<float *>(smem + M::kEnd);

    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, q4 = lane & 3, lr = lane & 7, lm = lane >> 3;
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

    // ---- the state: s[nt] = S^T rows 16 warp + g (+ 8), channels 8 nt + 2 q4 (+ 1) -------------------------------------
    const float *from = kStateOnly ? nullptr : (segs > 1 ? slot : (fresh ? nullptr : state));
    float s[DK / 8][4];
#pragma unroll
    for (int nt = 0; nt < DK / 8; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = nt * 8 + 2 * q4 + (e & 1), c = warp * 16 + g + 8 * (e >> 1);
            s[nt][e] = from != nullptr && d < a.dk && c < n_cols ? from[int64_t(d) * a.dv + col0 + c] : 0.f;
        }
    }
    float decayed = 0.f; // log2 decay of the whole segment (thread = channel)

    const __nv_bfloat16 *proj = static_cast<const __nv_bfloat16 *>(a.proj);
    auto load_tile = [&](int t0, int buf) {
        constexpr int kPieces = DK / 8, kVPieces = DV / 8, kBPieces = DK / 4;
        for (int u = tid; u < kTile * kPieces; u += kThreads) {
            const int t = u / kPieces, c = u - t * kPieces;
            const int bytes = t0 + t < end && c * 8 < a.dk ? 16 : 0;
            const __nv_bfloat16 *src = bytes ? proj + int64_t(t0 + t) * a.row_stride + int64_t(head) * a.dk + c * 8 : proj;
            if (!kStateOnly) {
                cp_async_16(sm + M::kQ + u * 16, bytes ? src + a.q_at : proj, bytes);
            }
            cp_async_16(sm + M::kK + u * 16, bytes ? src + a.k_at : proj, bytes);
        }
        for (int u = tid; u < kTile * kBPieces; u += kThreads) {
            const int t = u / kBPieces, c = u - t * kBPieces;
            const int bytes = t0 + t < end && c * 4 < a.dk ? 16 : 0;
            cp_async_16(sm + M::kB + u * 16, bytes ? a.decay + (int64_t(t0 + t) * a.heads + head) * a.dk + c * 4 : a.decay, bytes);
        }
        for (int u = tid; u < kTile * kVPieces; u += kThreads) {
            const int t = u / kVPieces, c = u - t * kVPieces;
            const int bytes = t0 + t < end && c * 8 < n_cols ? 16 : 0;
            cp_async_16(sm + M::kV + buf * (kTile * DV * 2) + swz(t, c, DV * 2),
                        bytes ? proj + int64_t(t0 + t) * a.row_stride + a.v_at + int64_t(head) * a.dv + col0 + c * 8 : proj, bytes);
        }
        cp_async_commit();
    };
    load_tile(begin, 0);

    int buf = 0;
    for (int t0 = begin; t0 < end; t0 += kTile, buf ^= 1) {
        const int n = min(kTile, end - t0);
        const uint32_t v_u32 = sm + M::kV + buf * (kTile * DV * 2);
        float o[8][4]; // O^T rows 16 warp + g (+ 8), tokens 8 nt + 2 q4 (+ 1)
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
        }
        cp_async_wait<0>();
        __syncthreads();
        for (int p0 = 0; p0 < n;) {
            // ---- how many tokens from p0 on go together ----------------------------------------------------------------
            int p1 = n;
            {
                float total = 0.f;
                if (tid < DK) {
#pragma unroll 8
                    for (int t = p0; t < n; ++t) {
                        total += s_b[t * DK + tid];
                    }
                }
                if (!__syncthreads_and(total >= -kMaxDecay)) {
                    if (tid == 0) {
                        s_limit = n;
                    }
                    __syncthreads();
                    if (tid < DK && total < -kMaxDecay) {
                        float run = 0.f;
                        int t = p0;
                        do { // at least one token
                            run += s_b[t * DK + tid];
                            ++t;
                        } while (t < n && run + s_b[t * DK + tid] >= -kMaxDecay);
                        atomicMin(&s_limit, t);
                    }
                    __syncthreads();
                    p1 = s_limit;
                }
            }
            // ---- running sums of the piece, its reference and its end ------------------------------------------------
            if (tid < DK) {
                const int mid = (p0 + p1 - 1) / 2;
                float run = 0.f, ref = 0.f;
#pragma unroll 8
                for (int t = p0; t < p1; ++t) {
                    run += s_b[t * DK + tid];
                    s_b[t * DK + tid] = run;
                    ref = t == mid ? run : ref;
                }
                s_ref[tid] = ref;
                s_end[tid] = run;
                decayed += run;
            }
            __syncthreads();
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
                    const float4 b0 = *reinterpret_cast<const float4 *>(s_b + t * DK + c * 8);
                    const float4 b1 = *reinterpret_cast<const float4 *>(s_b + t * DK + c * 8 + 4);
                    const float4 r0 = *reinterpret_cast<const float4 *>(s_ref + c * 8);
                    const float4 r1 = *reinterpret_cast<const float4 *>(s_ref + c * 8 + 4);
                    auto pair = [&](uint32_t qp, uint32_t kp, float d0, float d1, uint32_t &qhi, uint32_t &qlo, uint32_t &khi,
                                    uint32_t &klo) {
                        if (!kStateOnly) {
                            split2(lo_half(qp) * a.q_scale * fast_exp2(d0), hi_half(qp) * a.q_scale * fast_exp2(d1), qhi, qlo);
                        }
                        split2(lo_half(kp) * fast_exp2(-d0), hi_half(kp) * fast_exp2(-d1), khi, klo);
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
            if (p1 == n && t0 + kTile < end) {
                load_tile(t0 + kTile, buf ^ 1); // raw q, k and decays are used up; v goes to the other buffer
            }
            // ---- S^ = 2^m S ------------------------------------------------------------------------------------------
#pragma unroll
            for (int nt = 0; nt < DK / 8; ++nt) {
                const float f0 = fast_exp2(s_ref[nt * 8 + 2 * q4]), f1 = fast_exp2(s_ref[nt * 8 + 2 * q4 + 1]);
                s[nt][0] *= f0;
                s[nt][1] *= f1;
                s[nt][2] *= f0;
                s[nt][3] *= f1;
            }
            if constexpr (!kStateOnly) {
                // ---- O^T += S^T q^ : the accumulators are the A operand --------------------------------------------------
#pragma unroll
                for (int ks = 0; ks < DK / 16; ++ks) {
                    uint32_t ah[4], al[4];
                    split2(s[2 * ks][0], s[2 * ks][1], ah[0], al[0]);
                    split2(s[2 * ks][2], s[2 * ks][3], ah[1], al[1]);
                    split2(s[2 * ks + 1][0], s[2 * ks + 1][1], ah[2], al[2]);
                    split2(s[2 * ks + 1][2], s[2 * ks + 1][3], ah[3], al[3]);
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        const uint32_t at = sm + M::kQh + swz((np * 2 + (lm >> 1)) * 8 + lr, 2 * ks + (lm & 1), DK * 2);
                        uint32_t bh[4], bl[4];
                        ldmatrix_x4(bh, at);
                        ldmatrix_x4(bl, at + kTile * DK * 2);
                        mma_16816<true>(o[2 * np], ah, bh[0], bh[1]);
                        mma_16816<true>(o[2 * np + 1], ah, bh[2], bh[3]);
                        mma_16816<true>(o[2 * np], al, bh[0], bh[1]);
                        mma_16816<true>(o[2 * np + 1], al, bh[2], bh[3]);
                        mma_16816<true>(o[2 * np], ah, bl[0], bl[1]);
                        mma_16816<true>(o[2 * np + 1], ah, bl[2], bl[3]);
                    }
                }
                // ---- scores (q^_t . k^_s), s <= t, as two bf16 terms: warps share the 4 x 4 pairs of 16 tokens -------------
                for (int w = warp; w < 10; w += kWarps) { // the ten blocks on and below the diagonal
                    const int tb = w < 1 ? 0 : (w < 3 ? 1 : (w < 6 ? 2 : 3)), sb = w - tb * (tb + 1) / 2;
                    float c[2][4] = {};
#pragma unroll
                    for (int ks = 0; ks < DK / 16; ++ks) {
                        const uint32_t qa = sm + M::kQh + swz(tb * 16 + lr + 8 * (lm & 1), 2 * ks + (lm >> 1), DK * 2);
                        const uint32_t ka = sm + M::kKh + swz(sb * 16 + (lm >> 1) * 8 + lr, 2 * ks + (lm & 1), DK * 2);
                        uint32_t ah[4], al[4], bh[4], bl[4];
                        ldmatrix_x4(ah, qa);
                        ldmatrix_x4(al, qa + kTile * DK * 2);
                        ldmatrix_x4(bh, ka);
                        ldmatrix_x4(bl, ka + kTile * DK * 2);
                        mma_16816<true>(c[0], ah, bh[0], bh[1]);
                        mma_16816<true>(c[1], ah, bh[2], bh[3]);
                        mma_16816<true>(c[0], al, bh[0], bh[1]);
                        mma_16816<true>(c[1], al, bh[2], bh[3]);
                        mma_16816<true>(c[0], ah, bl[0], bl[1]);
                        mma_16816<true>(c[1], ah, bl[2], bl[3]);
                    }
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
#pragma unroll
                        for (int e = 0; e < 4; e += 2) {
                            const int t = tb * 16 + g + 4 * e, sc = sb * 16 + h * 8 + 2 * q4;
                            uint32_t hi, lo;
                            split2(sc <= t ? c[h][e] : 0.f, sc + 1 <= t ? c[h][e + 1] : 0.f, hi, lo);
                            const uint32_t at = M::kA + swz(t, sb * 2 + h, kTile * 2) + q4 * 4;
                            *reinterpret_cast<uint32_t *>(smem + at) = hi;
                            *reinterpret_cast<uint32_t *>(smem + at + kTile * kTile * 2) = lo;
                        }
                    }
                }
                __syncthreads();
            }
            // ---- O^T += V^T A^T and S^T += V^T k^ ---------------------------------------------------------------------
#pragma unroll
            for (int ks = 0; ks < kTile / 16; ++ks) {
                uint32_t va[4];
                ldmatrix_x4_trans(va, v_u32 + swz(ks * 16 + (lm >> 1) * 8 + lr, warp * 2 + (lm & 1), DV * 2));
                if constexpr (!kStateOnly) {
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        if (np >= ks) { // tokens 16 np .. see keys 16 ks ..
                            const uint32_t at = sm + M::kA + swz((np * 2 + (lm >> 1)) * 8 + lr, 2 * ks + (lm & 1), kTile * 2);
                            uint32_t bh[4], bl[4];
                            ldmatrix_x4(bh, at);
                            ldmatrix_x4(bl, at + kTile * kTile * 2);
                            mma_16816<true>(o[2 * np], va, bh[0], bh[1]);
                            mma_16816<true>(o[2 * np + 1], va, bh[2], bh[3]);
                            mma_16816<true>(o[2 * np], va, bl[0], bl[1]);
                            mma_16816<true>(o[2 * np + 1], va, bl[2], bl[3]);
                        }
                    }
                }
#pragma unroll
                for (int np = 0; np < DK / 16; ++np) {
                    const uint32_t at = sm + M::kKh + swz(ks * 16 + (lm & 1) * 8 + lr, np * 2 + (lm >> 1), DK * 2);
                    uint32_t bh[4], bl[4];
                    ldmatrix_x4_trans(bh, at);
                    ldmatrix_x4_trans(bl, at + kTile * DK * 2);
                    mma_16816<true>(s[2 * np], va, bh[0], bh[1]);
                    mma_16816<true>(s[2 * np + 1], va, bh[2], bh[3]);
                    mma_16816<true>(s[2 * np], va, bl[0], bl[1]);
                    mma_16816<true>(s[2 * np + 1], va, bl[2], bl[3]);
                }
            }
            // ---- S = 2^(b_end - m) S^ -----------------------------------------------------------------------------------
#pragma unroll
            for (int nt = 0; nt < DK / 8; ++nt) {
                const int d = nt * 8 + 2 * q4;
                const float f0 = fast_exp2(s_end[d] - s_ref[d]), f1 = fast_exp2(s_end[d + 1] - s_ref[d + 1]);
                s[nt][0] *= f0;
                s[nt][1] *= f1;
                s[nt][2] *= f0;
                s[nt][3] *= f1;
            }
            __syncthreads(); // q^, k^, the scores and the channel values are used up
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
                    s_o[o_at(nt * 8 + 2 * q4 + (e & 1), warp * 16 + g + 8 * (e >> 1))] = o[nt][e];
                }
            }
            __syncthreads();
            constexpr int kPer = DV / 32; // value columns per lane
            for (int t = warp; t < n; t += kWarps) {
                const int64_t row = t0 + t;
                float v[kPer];
                float ss = 0.f;
                const int c = lane * kPer;
#pragma unroll
                for (int e = 0; e < kPer; ++e) {
                    v[e] = s_o[o_at(t, c + e)];
                    ss = fmaf(v[e], v[e], ss); // (columns past n_cols are zero)
                }
                if (dv_slices > 1) { // the norm runs over more columns than this CTA has: a kernel of its own finishes
                    if (c < n_cols) {
#pragma unroll
                        for (int e = 0; e < kPer; ++e) {
                            a.raw[(row * a.heads + head) * a.dv + col0 + c + e] = v[e];
                        }
                    }
                    continue;
                }
#pragma unroll
                for (int u = 16; u > 0; u >>= 1) {
                    ss += __shfl_xor_sync(0xffffffffu, ss, u);
                }
                const float inv = rsqrtf(ss / float(a.dv) + a.eps) * a.out_scale;
                if (c < n_cols) { // (n_cols is a multiple of 8)
                    using P = Pieces<__nv_bfloat16, kPer>;
                    const P gate = *reinterpret_cast<const P *>(proj + row * a.row_stride + a.g_at + int64_t(head) * a.dv + c);
                    const P w = *reinterpret_cast<const P *>(static_cast<const __nv_bfloat16 *>(a.norm_w) + c);
                    P y;
#pragma unroll
                    for (int e = 0; e < kPer; ++e) {
                        y.v[e] = __float2bfloat16_rn(v[e] * inv * to_f32(w.v[e]) * silu(to_f32(gate.v[e])));
                    }
                    *reinterpret_cast<P *>(static_cast<__nv_bfloat16 *>(a.out) + row * a.out_stride + int64_t(head) * a.dv + c) = y;
                }
            }
        }
    }

    float *to = kStateOnly ? slot : (last ? state : nullptr);
    if (to != nullptr) {
#pragma unroll
        for (int nt = 0; nt < DK / 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = nt * 8 + 2 * q4 + (e & 1), c = warp * 16 + g + 8 * (e >> 1);
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
    for (int j = 0; j < n; ++j) {
        float *p = slot + j * stride;
        const float add = j + 1 < n ? p[e] : 0.f, decay = j + 1 < n ? fast_exp2(p[size + d]) : 0.f;
        p[e] = s;
        s = fmaf(s, decay, add);
    }
}

// decay[row, channel] = log2 a. A CTA does 32 rows x 128 channels; a thread keeps 16 weights of its channel in registers.
constexpr int kDecayRows = 32, kDecayCols = 128, kDecayRank = 16;
__global__ void __launch_bounds__(kDecayCols) gated_linear_log_decay_kernel(GatedLinearArgs a) {
    __shared__ __align__(16) float s_z[kDecayRows][kDecayRank];
    const __nv_bfloat16 *proj = static_cast<const __nv_bfloat16 *>(a.proj);
    const int n = a.heads * a.dk, c = int(blockIdx.y) * kDecayCols + int(threadIdx.x);
    const int64_t row0 = int64_t(blockIdx.x) * kDecayRows;
    const int rows = int(min(int64_t(kDecayRows), int64_t(a.n_rows) - row0));
    float acc[kDecayRows];
    const float bias = c < n ? to_f32(static_cast<const __nv_bfloat16 *>(a.decay_b)[c]) : 0.f;
#pragma unroll
    for (int t = 0; t < kDecayRows; ++t) {
        acc[t] = bias;
    }
    for (int r0 = 0; r0 < a.rank; r0 += kDecayRank) {
        __syncthreads();
        for (int u = int(threadIdx.x); u < kDecayRows * kDecayRank; u += kDecayCols) {
            const int t = u / kDecayRank, r = r0 + u % kDecayRank;
            s_z[t][u % kDecayRank] = t < rows && r < a.rank ? to_f32(proj[(row0 + t) * a.row_stride + a.z_at + r]) : 0.f;
        }
        __syncthreads();
        float w[kDecayRank];
#pragma unroll
        for (int r = 0; r < kDecayRank; ++r) {
            w[r] = c < n && r0 + r < a.rank ? to_f32(static_cast<const __nv_bfloat16 *>(a.decay_w)[int64_t(c) * a.rank + r0 + r]) : 0.f;
        }
#pragma unroll
        for (int t = 0; t < kDecayRows; ++t) {
#pragma unroll
            for (int r = 0; r < kDecayRank; r += 4) {
                const float4 z = *reinterpret_cast<const float4 *>(&s_z[t][r]);
                acc[t] = fmaf(w[r], z.x, acc[t]);
                acc[t] = fmaf(w[r + 1], z.y, acc[t]);
                acc[t] = fmaf(w[r + 2], z.z, acc[t]);
                acc[t] = fmaf(w[r + 3], z.w, acc[t]);
            }
        }
    }
    if (c < n) {
        const float f = 1.4426950408889634f / a.tau;
#pragma unroll
        for (int t = 0; t < kDecayRows; ++t) {
            if (t < rows) {
                a.decay[(row0 + t) * n + c] = log_sigmoid(acc[t]) * f;
            }
        }
    }
}

template <int DK, int DV, bool kStateOnly>
void launch_tiles(cudaStream_t s, const GatedLinearArgs &a, int segs, int seg_len, int slices) {
    static std::once_flag once[64];
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    constexpr int kBytes = ChunkSmem<DK, DV>::kBytes;
    std::call_once(once[dev & 63], [] {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(gated_linear_tile_kernel<DK, DV, kStateOnly>,
                                                cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes));
    });
    const dim3 grid(unsigned(a.n_seqs) * unsigned(a.heads) * unsigned(segs), unsigned(slices));
    gated_linear_tile_kernel<DK, DV, kStateOnly><<<grid, DV * 2, kBytes, s>>>(a, segs, seg_len, slices);
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
    return dtype == LLAISYS_DTYPE_BF16 && a.dk <= 128 && a.dk % 8 == 0 && a.dv % 8 == 0 && a.row_stride % 8 == 0 && a.q_at % 8 == 0 &&
           a.k_at % 8 == 0 && a.v_at % 8 == 0 && a.g_at % 8 == 0 && a.out_stride % 8 == 0 && aligned(a.proj) && aligned(a.out) &&
           aligned(a.norm_w) && aligned(a.decay);
}

void gated_linear_tiles(stream_t stream, const GatedLinearArgs &a) {
    auto s = static_cast<cudaStream_t>(stream);
    const dim3 decay_grid(unsigned((a.n_rows + kDecayRows - 1) / kDecayRows),
                          unsigned((a.heads * a.dk + kDecayCols - 1) / kDecayCols));
    gated_linear_log_decay_kernel<<<decay_grid, kDecayCols, 0, s>>>(a);
    const int slices = slices_of(a.dv);
    const int64_t pairs = int64_t(a.n_seqs) * a.heads;
    // segments: enough of them for a wave of CTAs, none shorter than 256 tokens, as many as the scratch holds
    const int64_t slot = int64_t(a.dk) * a.dv + a.dk;
    const int64_t wave = a.dk <= 64 && a.dv <= 64 ? kMaxCtas : kMaxCtas / 2;
    int64_t segs = std::min<int64_t>(wave / (pairs * slices), a.max_q_len / 256);
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
