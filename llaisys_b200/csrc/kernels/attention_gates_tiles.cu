// Attention without a softmax (GateArgs) on the tensor cores: bf16, K and V rows of at most 128 in whole 16-element steps, 16-token
// pages, any causal batch from single tokens to long chunks.
//
// The weights of all heads meet in every output, so a CTA takes a block of queries with ALL heads. Per kv head c, the pairs (query,
// head of c's group) are columns; 8 columns are a unit. Per tile of keys:
//   scores   S^T[key, column] = K_c q^T by mma.sync, queries in registers; gates in f32; weights to shared memory as f16
//            [query][key][head], times 2^15 (they lie in [0, 1]; so f16 holds them down to 2^-29 at full precision)
//   mixing   [head, key] = talk . weights of one query by mma.sync with f16 operands; to shared memory as bf16 [c][column][key]
//   values   O^T[value dim, column] += V_c^T . mixed by mma.sync, O in registers through all tiles
// Sums need no running maximum, so the tiles of all query blocks form one list that is cut into equal shares, one per SM; a block
// that is cut leaves partial sums in the scratch, and the last of its CTAs to arrive adds them in a fixed order.
//
// K and V tiles come by cp.async through two buffers each. Between two barriers a warp adds the values of tile t and scores tile t + 1,
// while K of tile t + 2 and V of tile t + 1 are under way; between the next two it mixes tile t + 1. Where two do not fit (many wide kv
// heads) there is one buffer each, and both loads stand between the barriers of the mixing.
#include "kernels.hpp"
#include "linear_tiles.cuh"

#include <algorithm>

namespace llaisys::kernels {

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32, kMaxUnits = 24, kMaxHeads = 64, kMaxSeqs = 1024;
constexpr float kLog2e = 1.4426950408889634f, kWeightUnit = 32768.f;

struct TileArgs {
    KVView kv;
    AttnBatch batch;
    const __nv_bfloat16 *q;
    __nv_bfloat16 *out;
    int64_t out_stride;
    GateArgs gates;
    float scale;
    int32_t bq, bk;          // queries of a block, keys of a tile
    int32_t bufs;            // buffers per operand, 1 or 2
    int32_t units_per_group; // of one kv head
    int32_t hp;              // heads padded to 16
    float *partials;         // [CTA][2][units * 8 * dv]
    int32_t *counters;       // [CTA]
    int32_t *error_flag;
};

// Byte offsets of the parts of shared memory. Rows are padded by 16 bytes: ldmatrix then meets every bank once.
struct TileSmem {
    int k, v, w, m, t, row_of, pages, prefix, total, k_bytes, v_bytes; // of one buffer

    __host__ __device__ TileSmem(const KVView &kv, int bufs, int bq, int bk, int units_per_group, int hp, int n_seqs) {
        int at = 0;
        auto take = [&](int bytes) {
            const int here = at;
            at += (bytes + 15) / 16 * 16;
            return here;
        };
        k_bytes = kv.nkvh * bk * (kv.d + 8) * 2;
        v_bytes = kv.nkvh * bk * (kv.vDim() + 8) * 2;
        k = take(bufs * k_bytes);
        v = take(bufs * v_bytes);
        w = take(bq * bk * (hp + 8) * 2);
        m = take(kv.nkvh * units_per_group * 8 * (bk + 8) * 2);
        t = take(hp * (hp + 8) * 2);
        row_of = take(hp * 4);
        pages = take(4 * bk / 16 * 4);
        prefix = take((n_seqs + 1) * 4);
        total = at;
    }
};

__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t &r0, uint32_t &r1, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// 1 / x_i for four numbers in [1, 2^31 + 1] with one reciprocal, times unit, plus c_i
__device__ __forceinline__ void rcp4(float (&x)[4], float unit, const float (&c)[4]) {
    const float p01 = x[0] * x[1], p23 = x[2] * x[3], r = rcp(p01 * p23) * unit, r01 = r * p23, r23 = r * p01;
    const float y0 = fmaf(r01, x[1], c[0]), y1 = fmaf(r01, x[0], c[1]), y2 = fmaf(r23, x[3], c[2]), y3 = fmaf(r23, x[2], c[3]);
    x[0] = y0;
    x[1] = y1;
    x[2] = y2;
    x[3] = y3;
}

struct Block { // a block of queries
    int q0, n_q;        // first query within its chunk, queries
    int pos0, kv_end;   // position of the first query, keys that the last one sees
    int tile0, n_tiles; // key tiles
};

__device__ __forceinline__ int q_first(const AttnBatch &b, int seq) { return b.q_starts != nullptr ? b.q_starts[seq] : seq; }
__device__ __forceinline__ int q_count(const AttnBatch &b, int seq) { return b.q_starts != nullptr ? b.q_starts[seq + 1] - b.q_starts[seq] : 1; }
__device__ __forceinline__ Block block_of(const TileArgs &a, int q_len, int kv_len, int index) {
    Block o;
    o.q0 = index * a.bq;
    o.n_q = min(a.bq, q_len - o.q0);
    o.pos0 = kv_len - q_len + o.q0;
    o.kv_end = o.n_q > 0 ? max(0, o.pos0 + o.n_q) : 0;
    o.tile0 = a.batch.window > 0 ? max(0, o.pos0 - a.batch.window + 1) / a.bk : 0;
    o.n_tiles = o.n_q > 0 ? max(0, (o.kv_end + a.bk - 1) / a.bk - o.tile0) : 0;
    return o;
}

// K or V rows of tile `tile`, its page ids in `ids`: a warp per (kv head, page). Keys from kv_end on become zero.
template <int STEPS>
__device__ __forceinline__ void load_tile(const TileArgs &a, const void *base, int64_t head_stride, int64_t token_stride, int width, uint32_t dst,
                                          const int *ids, int tile, int kv_end) {
    const int warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31, pages = a.bk / 16, row_bytes = (width + 8) * 2;
    const auto *src0 = static_cast<const __nv_bfloat16 *>(base);
    for (int item = warp; item < a.kv.nkvh * pages; item += kWarps) {
        const int c = item / pages, p = item - c * pages, page = ids[p];
        const int n = page < 0 ? 0 : min(16, kv_end - tile * a.bk - p * 16); // rows that exist
        const __nv_bfloat16 *src = src0 + int64_t(max(page, 0)) * a.kv.page_stride + c * head_stride;
        const uint32_t rows = dst + uint32_t((c * a.bk + p * 16) * row_bytes);
        if (width == STEPS * 16) {
            constexpr int kChunks = STEPS * 2, kStride = 32 / kChunks;
            const int r0 = lane / kChunks;
            const __nv_bfloat16 *from = src + r0 * token_stride + lane % kChunks * 8;
            uint32_t to = rows + uint32_t(r0 * row_bytes + lane % kChunks * 16);
#pragma unroll
            for (int r = 0; r < 16; r += kStride) {
                const bool ok = r + r0 < n;
                cp_async_16(to, ok ? from : src0, ok ? 16 : 0);
                from += kStride * token_stride;
                to += uint32_t(kStride * row_bytes);
            }
        } else {
            const int chunks = width / 8;
            for (int i = lane; i < 16 * chunks; i += 32) {
                const int r = i / chunks, chunk = i - r * chunks;
                const bool ok = r < n;
                cp_async_16(rows + uint32_t(r * row_bytes + chunk * 16), ok ? src + r * token_stride + chunk * 8 : src0, ok ? 16 : 0);
            }
        }
    }
    cp_async_commit();
}

// UNITS: per warp. SHARE: warps that share units -- they split a tile's keys for the scores and the value dims for the values.
// STEPS: 16-element steps of a K row at most (4 or 8); V rows likewise. ONE: the units of a warp belong to one kv head.
template <int UNITS, int SHARE, int STEPS, bool ONE>
__global__ void __launch_bounds__(kThreads, 1) attention_gates_tiles_kernel(const __grid_constant__ TileArgs a) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int kDims = (STEPS + SHARE - 1) / SHARE; // 16-dim blocks of V per warp
    const int nh = a.batch.nh, groups = a.kv.nkvh, share = nh / groups, d = a.kv.d, dv = a.kv.vDim(), bk = a.bk;
    const TileSmem lay(a.kv, a.bufs, a.bq, bk, a.units_per_group, a.hp, a.batch.n_seqs);
    const uint32_t base = smem_u32(smem);
    const int warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31;
    const int unit0 = warp / SHARE * UNITS, part = warp % SHARE, n_units = groups * a.units_per_group;
    int *prefix = reinterpret_cast<int *>(smem + lay.prefix), *page_ids = reinterpret_cast<int *>(smem + lay.pages), *row_of = reinterpret_cast<int *>(smem + lay.row_of);

    // ---- the list of tiles, and this CTA's share of it ----
    for (int s = warp; s < a.batch.n_seqs; s += kWarps) {
        const int q_len = q_count(a.batch, s), kv_len = a.batch.kv_lens[s], blocks = (q_len + a.bq - 1) / a.bq;
        int sum = 0;
        for (int b = lane; b < blocks; b += 32) {
            sum += block_of(a, q_len, kv_len, b).n_tiles;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            sum += __shfl_xor_sync(0xffffffffu, sum, o);
        }
        if (lane == 0) {
            prefix[s + 1] = sum;
        }
    }
    // talk as f16, identity without one, zero in the padding; weights of padding heads are zero throughout
    __half *talk = reinterpret_cast<__half *>(smem + lay.t);
    for (int i = threadIdx.x; i < a.hp * (a.hp + 8); i += kThreads) {
        const int h = i / (a.hp + 8), g = i % (a.hp + 8);
        float v = 0.f;
        if (h < nh && g < nh) {
            v = a.gates.talk != nullptr ? to_f32(static_cast<const __nv_bfloat16 *>(a.gates.talk)[h * nh + g]) : float(h == g);
        }
        talk[i] = __float2half_rn(v);
    }
    for (int i = threadIdx.x; i < a.bq * bk * (a.hp + 8) / 2; i += kThreads) {
        reinterpret_cast<uint32_t *>(smem + lay.w)[i] = 0u;
    }
    for (int h = threadIdx.x; h < a.hp; h += kThreads) {
        row_of[h] = h < nh ? h / share * a.units_per_group * 8 + h % share : -1; // row of query 0 in the mixed weights
    }
    __syncthreads();
    if (warp == 0) {
        int carry = 0;
        for (int s0 = 0; s0 < a.batch.n_seqs; s0 += 32) {
            int v = s0 + lane < a.batch.n_seqs ? prefix[s0 + lane + 1] : 0;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, v, o);
                v += lane >= o ? up : 0;
            }
            __syncwarp();
            if (s0 + lane < a.batch.n_seqs) {
                prefix[s0 + lane + 1] = carry + v;
            }
            carry += __shfl_sync(0xffffffffu, v, 31);
        }
        if (lane == 0) {
            prefix[0] = 0;
        }
    }
    __syncthreads();
    const int64_t total = prefix[a.batch.n_seqs], ctas = min(int64_t(gridDim.x), total); // (every share holds a tile)
    grid_dependency_wait(); // (the index arrays above are older than the kernel before this one)
    if (int64_t(blockIdx.x) >= ctas) {
        return;
    }
    const int begin = int(total * blockIdx.x / ctas), end = int(total * (blockIdx.x + 1) / ctas);
    int seq = 0, index = 0, block_begin = 0; // of the block that holds tile `begin`; its first tile in the list
    {
        int lo = 0, hi = a.batch.n_seqs - 1;
        while (lo < hi) { // last sequence with prefix[seq] <= begin
            const int mid = (lo + hi + 1) >> 1;
            if (prefix[mid] <= begin) {
                lo = mid;
            } else {
                hi = mid - 1;
            }
        }
        seq = lo;
        block_begin = prefix[seq];
        const int q_len = q_count(a.batch, seq), kv_len = a.batch.kv_lens[seq], blocks = (q_len + a.bq - 1) / a.bq;
        for (int b0 = 0; b0 < blocks; b0 += 32) { // every warp finds the same
            const int mine = b0 + lane < blocks ? block_of(a, q_len, kv_len, b0 + lane).n_tiles : 0;
            int v = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, v, o);
                v += lane >= o ? up : 0;
            }
            const unsigned past = __ballot_sync(0xffffffffu, block_begin + v > begin);
            if (past != 0u) {
                const int at = __ffs(int(past)) - 1;
                block_begin += __shfl_sync(0xffffffffu, v - mine, at);
                index = b0 + at;
                break;
            }
            block_begin += __shfl_sync(0xffffffffu, v, 31);
        }
    }

    const bool capped = a.gates.softcap > 0.f;
    const float to_exp = capped ? 2.f * kLog2e * a.scale / a.gates.softcap : -kLog2e * a.scale; // of a raw score
    const float cap2 = 2.f * kLog2e * a.gates.softcap;
    int group_of[UNITS];
#pragma unroll
    for (int u = 0; u < UNITS; ++u) {
        group_of[u] = min(unit0 + u, n_units - 1) / a.units_per_group;
    }

    for (int at = begin; at < end;) {
        const int q_len = q_count(a.batch, seq), blocks = (q_len + a.bq - 1) / a.bq;
        const Block blk = block_of(a, q_len, a.batch.kv_lens[seq], index);
        const int from = at - block_begin, upto = min(blk.n_tiles, end - block_begin); // tiles of the block in this share
        const int next_index = index + 1 < blocks ? index + 1 : 0, next_seq = index + 1 < blocks ? seq : seq + 1;
        if (upto <= from) { // (an empty sequence)
            index = next_index;
            seq = next_seq;
            continue;
        }
        const int32_t *table = a.kv.block_table + int64_t(a.batch.seq_ids != nullptr ? a.batch.seq_ids[seq] : seq) * a.kv.table_stride;
        const int64_t row0 = q_first(a.batch, seq) + blk.q0;
        const int pages = bk / 16;
        auto page_id = [&](int tile, int p) { // -1: past the end, or out of range
            const int at_block = tile * pages + p;
            int id = -1;
            if (at_block * 16 < blk.kv_end) {
                id = table[at_block];
                if (id < 0 || id >= a.kv.num_pages) {
                    atomicOr(a.error_flag, kErrBadPage);
                    id = -1;
                }
            }
            return id;
        };
        auto load_k = [&](int t) {
            if (t < upto) {
                load_tile<STEPS>(a, a.kv.k_base, a.kv.head_stride, a.kv.token_stride, d, base + lay.k + (t & (a.bufs - 1)) * lay.k_bytes,
                                 page_ids + (t & 3) * pages, blk.tile0 + t, blk.kv_end);
            } else {
                cp_async_commit(); // (an empty group keeps the count)
            }
        };
        auto load_v = [&](int t) {
            if (t < upto) {
                load_tile<STEPS>(a, a.kv.v_base, a.kv.vHeadStride(), a.kv.vTokenStride(), dv, base + lay.v + (t & (a.bufs - 1)) * lay.v_bytes,
                                 page_ids + (t & 3) * pages, blk.tile0 + t, blk.kv_end);
            } else {
                cp_async_commit();
            }
        };
        if (int(threadIdx.x) < 3 * pages) {
            const int t = from + int(threadIdx.x) / pages, p = int(threadIdx.x) % pages;
            page_ids[(t & 3) * pages + p] = page_id(blk.tile0 + t, p);
        }
        __syncthreads();
        load_k(from);
        load_v(from);
        load_k(a.bufs == 2 ? from + 1 : upto); // (upto: an empty group)

        // queries, and what a column needs for its gate
        uint32_t qf[UNITS][STEPS][2];
        int place[UNITS][2];                    // of the column's weight at key 0 in shared memory, -1: no such column
        float slope[UNITS][2], shift[UNITS][2], q_pos[UNITS][2];
#pragma unroll
        for (int u = 0; u < UNITS; ++u) {
            const int first_col = (unit0 + u - group_of[u] * a.units_per_group) * 8, col = first_col + (lane >> 2);
            const int qi = col / share, h = group_of[u] * share + col % share;
            const bool on = unit0 + u < n_units && qi < blk.n_q;
            const __nv_bfloat16 *src = a.q + ((row0 + qi) * nh + h) * d + 2 * (lane & 3);
#pragma unroll
            for (int ks = 0; ks < STEPS; ++ks) {
                const bool in = on && ks * 16 < d;
                qf[u][ks][0] = in ? *reinterpret_cast<const uint32_t *>(src + ks * 16) : 0u;
                qf[u][ks][1] = in ? *reinterpret_cast<const uint32_t *>(src + ks * 16 + 8) : 0u;
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int c2 = first_col + 2 * (lane & 3) + e, q2 = c2 / share, h2 = group_of[u] * share + c2 % share;
                const bool on2 = unit0 + u < n_units && q2 < blk.n_q;
                place[u][e] = on2 ? q2 * bk * (a.hp + 8) + h2 : -1;
                slope[u][e] = on2 && a.gates.slopes != nullptr ? kLog2e * a.gates.slopes[h2] : 0.f;
                const float b = on2 && a.gates.bias != nullptr ? to_f32(static_cast<const __nv_bfloat16 *>(a.gates.bias)[h2]) : 0.f;
                shift[u][e] = -kLog2e * (b + (capped ? a.gates.softcap : 0.f));
                q_pos[u][e] = float(blk.pos0 + q2);
            }
        }
        float o[UNITS][kDims][4];
#pragma unroll
        for (int u = 0; u < UNITS; ++u) {
#pragma unroll
            for (int b = 0; b < kDims; ++b) {
                o[u][b][0] = o[u][b][1] = o[u][b][2] = o[u][b][3] = 0.f;
            }
        }
        const float window = a.batch.window > 0 ? float(a.batch.window) : INFINITY;
        const bool pairs = share % 2 == 0; // the two columns of a thread are neighbouring heads of one query
        __half *w_s = reinterpret_cast<__half *>(smem + lay.w);

        // scores and gates of NK blocks of 16 keys of tile t (kb0, kb0 + SHARE, ..); `edge`: some keys are out of sight
        auto score = [&](auto nk, int t, int kb0, bool edge) {
            constexpr int NK = decltype(nk)::value;
            const uint32_t k_s = base + uint32_t(lay.k + (t & (a.bufs - 1)) * lay.k_bytes);
            float s[NK][UNITS][4];
#pragma unroll
            for (int b = 0; b < NK; ++b) {
#pragma unroll
                for (int u = 0; u < UNITS; ++u) {
                    s[b][u][0] = s[b][u][1] = s[b][u][2] = s[b][u][3] = 0.f;
                }
            }
#pragma unroll
            for (int ks = 0; ks < STEPS; ++ks) {
                if (ks * 16 < d) {
#pragma unroll
                    for (int b = 0; b < NK; ++b) {
                        uint32_t kf[4];
#pragma unroll
                        for (int u = 0; u < UNITS; ++u) {
                            if (u == 0 || (!ONE && group_of[u] != group_of[u - 1])) {
                                ldmatrix_x4(kf, k_s + uint32_t(((group_of[u] * bk + (kb0 + b * SHARE) * 16 + (lane & 15)) * (d + 8) + ks * 16 +
                                                                (lane >> 4) * 8) * 2));
                            }
                            mma_bf16(s[b][u], kf, qf[u][ks][0], qf[u][ks][1]);
                        }
                    }
                }
            }
#pragma unroll
            for (int b = 0; b < NK; ++b) {
                const int key = (kb0 + b * SHARE) * 16 + (lane >> 2);
                const float j = float((blk.tile0 + t) * bk + key);
#pragma unroll
                for (int u = 0; u < UNITS; ++u) {
                    float x[4], ago[4], c[4]; // element i: key + 8 (i / 2), column i % 2
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        ago[i] = q_pos[u][i & 1] - (j + float(i >> 1) * 8.f);
                        c[i] = fmaf(slope[u][i & 1], ago[i], shift[u][i & 1]);
                    }
                    if (capped) { // softcap tanh(y) = softcap - 2 softcap / (1 + e^(2 y))
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            x[i] = 1.f + ex2(fminf(s[b][u][i] * to_exp, 31.f));
                        }
                        rcp4(x, cap2, c);
                    } else {
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            x[i] = fmaf(s[b][u][i], to_exp, c[i]);
                        }
                    }
                    const float zero[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        x[i] = 1.f + ex2(fminf(x[i], 31.f));
                    }
                    rcp4(x, kWeightUnit, zero);
                    if (edge) {
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            x[i] = ago[i] >= 0.f && ago[i] < window ? x[i] : 0.f;
                        }
                    }
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const int row = (key + 8 * r) * (a.hp + 8);
                        if (pairs) {
                            if (place[u][0] >= 0) {
                                *reinterpret_cast<uint32_t *>(w_s + place[u][0] + row) = pack2<false>(x[2 * r], x[2 * r + 1]);
                            }
                        } else {
                            if (place[u][0] >= 0) {
                                w_s[place[u][0] + row] = __float2half_rn(x[2 * r]);
                            }
                            if (place[u][1] >= 0) {
                                w_s[place[u][1] + row] = __float2half_rn(x[2 * r + 1]);
                            }
                        }
                    }
                }
            }
        };
        auto scores = [&](int t) {
            const int first = (blk.tile0 + t) * bk;
            const bool edge = first + bk > blk.pos0 + 1 || (a.batch.window > 0 && first + a.batch.window < blk.pos0 + blk.n_q);
            int kb = part;
            for (; kb + SHARE < bk / 16; kb += 2 * SHARE) {
                score(std::integral_constant<int, 2>{}, t, kb, edge);
            }
            if (kb < bk / 16) {
                score(std::integral_constant<int, 1>{}, t, kb, edge);
            }
        };
        auto values = [&](int t) {
            const uint32_t v_s = base + uint32_t(lay.v + (t & (a.bufs - 1)) * lay.v_bytes);
            for (int kb = 0; kb < bk / 16; ++kb) {
                uint32_t mf[UNITS][2];
#pragma unroll
                for (int u = 0; u < UNITS; ++u) {
                    const int row = min(unit0 + u, n_units - 1) * 8 + (lane & 7);
                    ldmatrix_x2(mf[u][0], mf[u][1], base + uint32_t(lay.m + (row * (bk + 8) + kb * 16 + ((lane >> 3) & 1) * 8) * 2));
                }
#pragma unroll
                for (int b = 0; b < kDims; ++b) {
                    const int dim = (part + b * SHARE) * 16;
                    if (dim < dv) {
                        uint32_t vf[4];
#pragma unroll
                        for (int u = 0; u < UNITS; ++u) {
                            if (u == 0 || (!ONE && group_of[u] != group_of[u - 1])) {
                                ldmatrix_x4_trans(vf, v_s + uint32_t(((group_of[u] * bk + kb * 16 + (lane & 7) + (lane >> 4) * 8) * (dv + 8) + dim +
                                                                      ((lane >> 3) & 1) * 8) * 2));
                            }
                            mma_bf16(o[u][b], vf, mf[u][0], mf[u][1]);
                        }
                    }
                }
            }
        };
        auto mix = [&]() { // a warp per (query, 16 keys, 16 heads)
            const int tiles_h = a.hp / 16, per_q = pages * tiles_h;
            for (int item = warp; item < blk.n_q * per_q; item += kWarps) {
                const int qi = item / per_q, rest = item - qi * per_q, kb = rest / tiles_h, mt = rest - kb * tiles_h;
                float y0[4] = {0.f, 0.f, 0.f, 0.f}, y1[4] = {0.f, 0.f, 0.f, 0.f};
                for (int kt = 0; kt < tiles_h; ++kt) {
                    uint32_t tf[4], wf[4];
                    ldmatrix_x4(tf, base + uint32_t(lay.t + ((mt * 16 + (lane & 15)) * (a.hp + 8) + kt * 16 + (lane >> 4) * 8) * 2));
                    ldmatrix_x4(wf, base + uint32_t(lay.w + (((qi * bk + kb * 16 + (lane & 7) + (lane >> 4) * 8) * (a.hp + 8)) + kt * 16 +
                                                             ((lane >> 3) & 1) * 8) * 2));
                    mma_f16(y0, tf, wf[0], wf[1]);
                    mma_f16(y1, tf, wf[2], wf[3]);
                }
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int row = row_of[mt * 16 + (lane >> 2) + 8 * r];
                    if (row >= 0) {
                        auto *dst = reinterpret_cast<uint32_t *>(smem + lay.m + ((row + qi * share) * (bk + 8) + kb * 16 + 2 * (lane & 3)) * 2);
                        dst[0] = pack2<true>(y0[2 * r], y0[2 * r + 1]);
                        dst[4] = pack2<true>(y1[2 * r], y1[2 * r + 1]);
                    }
                }
            }
        };

        cp_async_wait<2>(); // K of the first tile
        __syncthreads();
        scores(from);
        __syncthreads();
        if (a.bufs == 1) {
            load_k(from + 1);
        }
        mix();
        for (int t = from; t < upto; ++t) {
            cp_async_wait<0>(); // V of tile t, K of tile t + 1
            __syncthreads();
            int next_page = 0;
            if (int(threadIdx.x) < pages) {
                next_page = page_id(blk.tile0 + t + 3, int(threadIdx.x));
            }
            if (a.bufs == 2) {
                load_k(t + 2);
                load_v(t + 1);
            }
            values(t);
            if (t + 1 < upto) {
                scores(t + 1);
                if (int(threadIdx.x) < pages) {
                    page_ids[((t + 3) & 3) * pages + int(threadIdx.x)] = next_page;
                }
                __syncthreads();
                if (a.bufs == 1) {
                    load_k(t + 2);
                    load_v(t + 1);
                }
                mix();
            }
        }

        // ---- the block's output, whole or in pieces ----
        bool writes = true;
        if (from != 0 || upto != blk.n_tiles) {
            const int64_t slot = int64_t(n_units) * 8 * dv;
            auto piece = [&](float *slot_base, int u, int b) {
                return reinterpret_cast<float4 *>(slot_base) + (int64_t(unit0 + u) * (dv / 16) + (part + b * SHARE)) * 32 + lane;
            };
            auto slot_of = [&](int cta, bool first) { return a.partials + (int64_t(cta) * 2 + (first ? 1 : 0)) * slot; };
            float *own = slot_of(int(blockIdx.x), from == 0);
#pragma unroll
            for (int u = 0; u < UNITS; ++u) {
#pragma unroll
                for (int b = 0; b < kDims; ++b) {
                    if (unit0 + u < n_units && (part + b * SHARE) * 16 < dv) {
                        *piece(own, u, b) = make_float4(o[u][b][0], o[u][b][1], o[u][b][2], o[u][b][3]);
                    }
                }
            }
            // CTAs whose shares touch the block: share c holds tile t iff c is the largest with c * total < (t + 1) * ctas
            const int first_cta = int(((int64_t(block_begin) + 1) * ctas - 1) / total);
            const int last_cta = int((int64_t(block_begin + blk.n_tiles) * ctas - 1) / total);
            __shared__ int last;
            __threadfence();
            __syncthreads();
            if (threadIdx.x == 0) {
                last = atomicAdd(a.counters + first_cta, 1) == last_cta - first_cta;
                if (last) {
                    a.counters[first_cta] = 0;
                }
            }
            __syncthreads();
            writes = last != 0;
            if (writes) {
                __threadfence();
#pragma unroll
                for (int u = 0; u < UNITS; ++u) {
#pragma unroll
                    for (int b = 0; b < kDims; ++b) {
                        if (unit0 + u < n_units && (part + b * SHARE) * 16 < dv) {
                            float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
                            for (int c = first_cta; c <= last_cta; ++c) {
                                const float4 v = __ldcg(piece(slot_of(c, c == first_cta), u, b));
                                sum.x += v.x;
                                sum.y += v.y;
                                sum.z += v.z;
                                sum.w += v.w;
                            }
                            o[u][b][0] = sum.x;
                            o[u][b][1] = sum.y;
                            o[u][b][2] = sum.z;
                            o[u][b][3] = sum.w;
                        }
                    }
                }
            }
        }
        if (writes) {
#pragma unroll
            for (int u = 0; u < UNITS; ++u) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (place[u][e] >= 0) {
                        const int c2 = (unit0 + u - group_of[u] * a.units_per_group) * 8 + 2 * (lane & 3) + e;
                        __nv_bfloat16 *dst = a.out + (row0 + c2 / share) * a.out_stride + int64_t(group_of[u] * share + c2 % share) * dv + (lane >> 2);
#pragma unroll
                        for (int b = 0; b < kDims; ++b) {
                            const int dim = (part + b * SHARE) * 16;
                            if (dim < dv) {
                                dst[dim] = __float2bfloat16_rn(o[u][b][e] * (1.f / kWeightUnit));
                                dst[dim + 8] = __float2bfloat16_rn(o[u][b][2 + e] * (1.f / kWeightUnit));
                            }
                        }
                    }
                }
            }
        }
        cp_async_wait<0>();
        __syncthreads();
        at += upto - from;
        block_begin += blk.n_tiles;
        index = next_index;
        seq = next_seq;
    }
}

constexpr int kMaxSmem = 226 * 1024;

int sm_count() {
    static int n = [] {
        int dev = 0, v = 0;
        LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
        LLAISYS_CUDA_CHECK(cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev));
        return v;
    }();
    return n;
}

template <int UNITS, int SHARE, int STEPS>
void launch(cudaStream_t s, const TileArgs &args, size_t smem, int grid, bool overlap) {
    auto kernel = args.units_per_group % UNITS == 0 ? attention_gates_tiles_kernel<UNITS, SHARE, STEPS, true>
                                                    : attention_gates_tiles_kernel<UNITS, SHARE, STEPS, UNITS == 1>;
    LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem));
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned(grid));
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = overlap ? 1 : 0;
    LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, args));
}

} // namespace

void attention_gates_tiles_scratch(size_t longest_v_row, size_t *floats, size_t *counters) {
    *floats = size_t(sm_count()) * 2 * kMaxUnits * 8 * ((longest_v_row + 15) / 16 * 16);
    *counters = size_t(sm_count());
}

int attention_gates_tiles(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                          const GateArgs &gates, const AttnOut &out, const AttnScratch &scratch) {
    const int d = kv.d, dv = kv.vDim();
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    if (dtype != LLAISYS_DTYPE_BF16 || d % 16 != 0 || dv % 16 != 0 || d > 128 || dv > 128 || kv.page_size != 16 || kv.block_table == nullptr ||
        batch.kv_lens == nullptr || kv.nkvh <= 0 || kv.nkvh > kMaxUnits || batch.nh > kMaxHeads || batch.nh % kv.nkvh != 0 ||
        batch.n_seqs > kMaxSeqs || batch.keep_first != 0 || out.out == nullptr || out.part != nullptr || out.row_scale != nullptr ||
        !aligned(kv.k_base) || !aligned(kv.v_base) || kv.token_stride % 8 != 0 || kv.vTokenStride() % 8 != 0 ||
        (batch.q_starts == nullptr && batch.const_q_len != 1) || reinterpret_cast<uintptr_t>(q) % 4 != 0) {
        return -1;
    }
    if (batch.n_seqs <= 0 || batch.total_q <= 0) {
        return 0;
    }
    const int share = batch.nh / kv.nkvh;
    TileArgs a{};
    a.kv = kv;
    a.batch = batch;
    a.q = static_cast<const __nv_bfloat16 *>(q);
    a.out = static_cast<__nv_bfloat16 *>(out.out);
    a.out_stride = out.row_stride ? out.row_stride : int64_t(batch.nh) * dv;
    a.gates = gates;
    a.scale = scale;
    a.hp = (batch.nh + 15) / 16 * 16;
    a.partials = scratch.partials;
    a.counters = scratch.counters;
    a.error_flag = scratch.error_flag;
    // the largest block of queries whose columns fit the warps' registers (whole units preferred), and the longest tile of keys
    // that fits shared memory
    const int most_q = batch.q_starts == nullptr ? 1 : std::min(std::max(batch.max_q_len, 1), 32);
    auto units = [&](int bq) { return (bq * share + 7) / 8; };
    int best = 0;
    for (int bq = 1; bq <= most_q; ++bq) {
        if (kv.nkvh * units(bq) <= kMaxUnits && (best == 0 || bq * share % 8 == 0 || best * share % 8 != 0)) {
            best = bq;
        }
    }
    if (best == 0) {
        return -1;
    }
    size_t smem = 0;
    for (int bufs = 2, bq = best; bufs >= 1 && smem == 0; bq > 1 ? bq /= 2 : (bq = best, --bufs)) {
        for (int bk = bq == 1 ? 128 : 64; bk >= 16; bk /= 2) {
            const TileSmem lay(kv, bufs, bq, bk, units(bq), a.hp, batch.n_seqs);
            if (lay.total <= kMaxSmem) {
                a.bufs = bufs;
                a.bq = bq;
                a.bk = bk;
                a.units_per_group = units(bq);
                smem = size_t(lay.total);
                break;
            }
        }
    }
    const int grid = sm_count(), n_units = smem != 0 ? kv.nkvh * a.units_per_group : 0;
    if (smem == 0 || scratch.partials == nullptr || scratch.counters == nullptr || scratch.error_flag == nullptr ||
        scratch.partials_floats < size_t(grid) * 2 * size_t(n_units) * 8 * size_t(dv) || scratch.counters_len < size_t(grid)) {
        return -1;
    }
    auto s = static_cast<cudaStream_t>(stream);
    auto go = [&](auto steps) {
        constexpr int kSteps = decltype(steps)::value;
        if (n_units > 16) {
            launch<3, 1, kSteps>(s, a, smem, grid, kv.overlap_launch);
        } else if (n_units > 8) {
            launch<2, 1, kSteps>(s, a, smem, grid, kv.overlap_launch);
        } else if (n_units > 4) {
            launch<1, 1, kSteps>(s, a, smem, grid, kv.overlap_launch);
        } else if (n_units > 2) {
            launch<1, 2, kSteps>(s, a, smem, grid, kv.overlap_launch);
        } else {
            launch<1, 4, kSteps>(s, a, smem, grid, kv.overlap_launch);
        }
    };
    if (d <= 64 && dv <= 64) {
        go(std::integral_constant<int, 4>{});
    } else {
        go(std::integral_constant<int, 8>{});
    }
    check_launch("attention_gates_tiles");
    return 0;
}

} // namespace llaisys::kernels
