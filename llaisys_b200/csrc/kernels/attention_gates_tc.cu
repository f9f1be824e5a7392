// Attention without a softmax (GateArgs) over chunks of queries, on the 5th-generation tensor cores (tcgen05 + TMEM): bf16, K and V
// rows of 128, 16-token pages, at most 32 heads and 16 kv heads.
//
// Roofline: tensor; 4 * nh * 128 flops per visible (query, key) pair as for softmax attention. What bounds it is the multi-function
// unit: a capped score and its sigmoid take two exponentials and half a reciprocal where a softmax takes one exponential.
//
// A CTA takes a block of bq queries with ALL heads, because the weights of all heads meet in every output, and visits its visible keys
// 128 at a time (a TILE). A kv head's columns are the pairs (query, head of its group), padded to n_c, a multiple of 16; both products
// are transposed, so that the long sides (keys, value dims) fill the 128 rows of an MMA and a kv head's few columns are its N:
//   S_c[key, column]   = K_c q^T          A = K tile (K-major), B = queries in shared memory
//   O_c[dim, column]  += V_c^T P_c        A = V tile (MN-major, as the pages hold it), B = P_c [column][key]
// S_c and O_c of all kv heads live in TMEM (256 columns each).
//
//   warps 0-15   read S as mma fragments (a thread has four keys of two neighbouring columns in every eight), compute the weights, store them as f16 times 2^15 into the buffer that becomes P; when all heads
//                are there, mix them IN PLACE: 16 keys of one query, all heads, are read as mma.sync operands, multiplied by the talk
//                matrix (in registers) and stored as bf16 to the same places
//   warps 16, 18 TMA of K and V tiles into a ring of 32 KiB slots, half of a tile's pages each (as in warp 17, an elected lane issues:
//                a warp between busy ones needs about 1000 clocks for a tile's 16 boxes)
//   warp 17      issues the MMAs (the whole warp walks, an elected lane issues: descriptors then stay in uniform registers, which made
//                a batch of eight small MMAs 3.7 times as fast as a loop run by one thread): S of tile t + 1 kv head by kv head as the scores of tile t have been read, then O of tile t.
//                Weights of tile t + 1 go where P_c of tile t was as soon as O_c has taken it.
//
// The tiles of all blocks form one line that is cut into equal shares, one per CTA; a block that is cut leaves partial sums in the
// scratch (nothing is rescaled: sums add), and the last of its CTAs to arrive adds them in a fixed order.
//
// Every wait is bounded: one that runs out sets bit 8 of the error word and the CTA winds down. No cluster launch, no multicast.
#include "kernels.hpp"
#include "linear_tiles.cuh"
#include "tcgen05_utils.cuh"

#include <cuda.h>

#include <algorithm>
#include <cstring>

namespace llaisys::kernels {

namespace {

constexpr int kD = 128, kBk = 128, kPages = kBk / 16;
constexpr int kWorkers = 16, kProducer = 16, kIssuer = 17, kProducer2 = 18, kThreads = 19 * 32;
constexpr int kChunk = 32; // columns of one kv head that a warp turns into weights at a time
constexpr int kSlot = kBk * kD * 2, kMaxStages = 6, kMaxColumns = 256, kMaxGroups = 16;
// What a block costs besides its tiles (queries in, products drained, outputs out), in tiles. The line that is cut into equal shares
// counts every block as this many units and then its tiles.
constexpr int kBlockCost = 1;
constexpr int kSmemLimit = 227 * 1024, kErrTimeout = 8;
constexpr float kLog2e = 1.4426950408889634f, kWeightUnit = 32768.f;

// A shared-memory descriptor that starts `bytes` further on (the address field counts 16-byte steps and does not overflow).
__device__ __forceinline__ uint64_t desc_at(uint64_t desc, uint32_t bytes) {
    return (desc & 0xffffffff00000000ull) | uint32_t(uint32_t(desc) + (bytes >> 4));
}

// A cursor over the ring: the next slot, and the parity of its barriers' phases in this round. (No division: the warps that hold one
// run between busy ones, and every instruction of theirs counts.)
struct Cursor {
    int slot = 0;
    uint32_t parity = 0;
    __device__ __forceinline__ void next(int stages) {
        ++slot;
        if (slot == stages) {
            slot = 0;
            parity ^= 1u;
        }
    }
};

struct Params {
    AttnBatch batch;
    GateArgs gates;
    const __nv_bfloat16 *q;
    __nv_bfloat16 *out;
    int64_t out_stride;
    float scale;
    int64_t page0;
    const int32_t *block_table;
    int32_t table_stride, num_pages;
    int32_t groups, share, bq, n_c, stages; // n_c: columns of a kv head, padded
    float *partials; // [CTA][2][groups * n_c][128]
    int32_t *counters;
    int32_t *error_flag;
};

struct Block { // a block of queries
    int q0, n_q;        // first query within its chunk, queries
    int pos0, kv_end;   // position of the first query, keys that the last one sees
    int tile0, n_tiles; // key tiles
    __device__ __forceinline__ int units() const { return n_tiles > 0 ? kBlockCost + n_tiles : 0; }
};

__device__ __forceinline__ Block block_of(const Params &p, int q_len, int kv_len, int index) {
    Block o;
    o.q0 = index * p.bq;
    o.n_q = min(p.bq, q_len - o.q0);
    o.pos0 = kv_len - q_len + o.q0;
    o.kv_end = o.n_q > 0 ? max(0, o.pos0 + o.n_q) : 0;
    o.tile0 = p.batch.window > 0 ? max(0, o.pos0 - p.batch.window + 1) / kBk : 0;
    o.n_tiles = o.n_q > 0 ? max(0, (o.kv_end + kBk - 1) / kBk - o.tile0) : 0;
    return o;
}

// A CTA's walk over its share [at, end) of the line: every role walks the same fragments.
struct Walk {
    int at, end, seq, index, block_begin; // (at: kept within the block at `index`)
};
struct Fragment {
    Block block;
    int seq, from, upto, block_begin; // tiles of the block
    int64_t row0;                     // first query row
};
__device__ __forceinline__ bool next_fragment(const Params &p, Walk &w, Fragment &f) {
    while (w.at < w.end) {
        const int first = p.batch.q_starts[w.seq], q_len = p.batch.q_starts[w.seq + 1] - first;
        f.block = block_of(p, q_len, p.batch.kv_lens[w.seq], w.index);
        f.seq = w.seq;
        f.block_begin = w.block_begin;
        f.from = max(0, w.at - w.block_begin - kBlockCost);
        f.upto = min(f.block.n_tiles, w.end - w.block_begin - kBlockCost);
        f.row0 = first + f.block.q0;
        w.block_begin += f.block.units();
        w.at = max(w.at, w.block_begin);
        w.index += 1;
        if (w.index * p.bq >= q_len) {
            w.index = 0;
            w.seq += 1;
        }
        if (f.upto > f.from) {
            return true;
        }
    }
    return false;
}

__device__ __forceinline__ void tmem_ld8(uint32_t taddr, float (&v)[8]) {
    uint32_t r[8];
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        v[i] = __uint_as_float(r[i]);
    }
}
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// Pairs of f32 in one register pair: two of these operations go out as one instruction.
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair(float x, float y) {
    Pair p;
    asm("mov.b64 %0, {%1, %2};\n" : "=l"(p) : "f"(x), "f"(y));
    return p;
}
__device__ __forceinline__ void unpair(Pair p, float &x, float &y) { asm("mov.b64 {%0, %1}, %2;\n" : "=f"(x), "=f"(y) : "l"(p)); }
__device__ __forceinline__ Pair mul2(Pair a, Pair b) {
    Pair d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ Pair add2(Pair a, Pair b) {
    Pair d;
    asm("add.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ Pair fma2(Pair a, Pair b, Pair c) {
    Pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
// 1 + 2^min(x, 31), element by element
__device__ __forceinline__ Pair one_plus_ex2(Pair x, Pair ones) {
    float a, b;
    unpair(x, a, b);
    return add2(ones, pair(ex2(fminf(a, 31.f)), ex2(fminf(b, 31.f))));
}
// (unit / the four numbers of x and y), which lie in [1, 2^31 + 1], with one reciprocal: p times y is for x, p times x for y
__device__ __forceinline__ Pair rcp4(Pair x, Pair y, float unit) {
    float a, b;
    unpair(mul2(x, y), a, b);
    const float r = rcp(a * b) * unit;
    return pair(r * b, r * a);
}
// n / d for 0 <= n < 2^15, inv = 1 / d rounded
__device__ __forceinline__ int small_div(int n, float inv) { return int((float(n) + 0.5f) * inv); }
// 32 columns of 16 lanes as m16n8 fragments: of columns 8 j + 2 (lane % 4) and the next, r[4 j ..] holds those of lane / 4, then those of lane / 4 + 8
__device__ __forceinline__ void tmem_ld_fragments(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
                   "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr));
}
__device__ __forceinline__ void stmatrix_x4_trans(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
    asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};\n" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
}
__device__ __forceinline__ void stmatrix_x4(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
    asm volatile("stmatrix.sync.aligned.m8n8.x4.shared.b16 [%0], {%1, %2, %3, %4};\n" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
}

// Shared memory: ring | queries | weights (all 1024-byte aligned) | per-column constants | barriers | small words.
struct Layout {
    int q, w, columns, bars, misc, total;
    __host__ __device__ Layout(int stages, int n_columns) {
        q = stages * kSlot;
        w = q + n_columns * kD * 2;
        columns = w + n_columns * kBk * 2;
        bars = columns + n_columns * 8;
        misc = bars + (2 * kMaxStages + 5 * kMaxGroups + 3) * 8;
        misc = (misc + 15) / 16 * 16;
        total = misc + 32; // [0, 16) zeros, then abort flag, TMEM base, `last`
    }
};
// barriers
constexpr int kBarFull = 0;                            // [stages] producers -> issuer: a tile has landed
constexpr int kBarFree = kBarFull + kMaxStages;        // [stages] MMAs -> producers: it has been used
constexpr int kBarS = kBarFree + kMaxStages;           // [2][groups] S_c of a tile is written
constexpr int kBarPV = kBarS + 2 * kMaxGroups;         // [2][groups] O_c has taken a tile (P_c is free)
constexpr int kBarRead = kBarPV + 2 * kMaxGroups;      // [groups] workers -> issuer: S_c has been read (a warp per chunk and quarter)
constexpr int kBarP = kBarRead + kMaxGroups;           // workers -> issuer: P of a tile is complete
constexpr int kBarQ = kBarP + 1;                       // workers -> issuer: queries of a fragment are in place
constexpr int kBarO = kBarQ + 1;                       // workers -> issuer: O has been read

template <int MT> // heads in whole 16s
__global__ void __launch_bounds__(kThreads, 1)
    attention_gates_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                              const __grid_constant__ Params p) {
    extern __shared__ __align__(1024) unsigned char smem[];
    const int groups = p.groups, share = p.share, n_c = p.n_c, nh = p.batch.nh, n_columns = groups * n_c;
    const Layout lay(p.stages, n_columns);
    const uint32_t base = smem_u32(smem);
    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    int *misc = reinterpret_cast<int *>(smem + lay.misc);
    volatile int *s_abort = misc + 4;
    auto bar = [&](int which) { return base + uint32_t(lay.bars + which * 8); };
    auto s_bar = [&](int n, int c) { return bar(kBarS + (n & 1) * kMaxGroups + c); };
    auto pv_bar = [&](int n, int c) { return bar(kBarPV + (n & 1) * kMaxGroups + c); };
    auto give_up = [&]() {
        *s_abort = 1;
        atomicOr(p.error_flag, kErrTimeout);
    };

    // ---- the line of tiles (its prefix sums lie in the ring, which nothing uses yet) ----
    int *prefix = reinterpret_cast<int *>(smem);
    for (int s = warp; s < p.batch.n_seqs; s += kThreads / 32) {
        const int q_len = p.batch.q_starts[s + 1] - p.batch.q_starts[s], kv_len = p.batch.kv_lens[s], blocks = (q_len + p.bq - 1) / p.bq;
        int sum = 0;
        for (int b = lane; b < blocks; b += 32) {
            sum += block_of(p, q_len, kv_len, b).units();
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            sum += __shfl_xor_sync(0xffffffffu, sum, o);
        }
        if (lane == 0) {
            prefix[s + 1] = sum;
        }
    }
    if (tid == 0) {
        prefix[0] = 0;
        for (int i = 0; i < kBarO + 1; ++i) {
            mbar_init(bar(i), i < kBarFree ? 2 : i < kBarRead ? 1 : (i < kBarP ? 4 * ((n_c + kChunk - 1) / kChunk) : kWorkers));
        }
        misc[0] = misc[1] = misc[2] = misc[3] = 0;
        *s_abort = 0;
        mbar_init_fence();
    }
    __syncthreads();
    if (warp == 0) {
        int carry = 0;
        for (int s0 = 0; s0 < p.batch.n_seqs; s0 += 32) {
            int v = s0 + lane < p.batch.n_seqs ? prefix[s0 + lane + 1] : 0;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, v, o);
                v += lane >= o ? up : 0;
            }
            __syncwarp();
            if (s0 + lane < p.batch.n_seqs) {
                prefix[s0 + lane + 1] = carry + v;
            }
            carry += __shfl_sync(0xffffffffu, v, 31);
        }
    }
    __syncthreads();
    const int64_t total = prefix[p.batch.n_seqs], ctas = min(int64_t(gridDim.x), total); // (every share holds a unit)
    grid_dependency_wait(); // (the index arrays above are older than the kernel before this one)
    if (int64_t(blockIdx.x) >= ctas) {
        return;
    }
    Walk walk{int(total * blockIdx.x / ctas), int(total * (blockIdx.x + 1) / ctas), 0, 0, 0};
    {
        int lo = 0, hi = p.batch.n_seqs - 1;
        while (lo < hi) { // last sequence with prefix[seq] <= walk.at
            const int mid = (lo + hi + 1) >> 1;
            if (prefix[mid] <= walk.at) {
                lo = mid;
            } else {
                hi = mid - 1;
            }
        }
        walk.seq = lo;
        walk.block_begin = prefix[lo];
        const int q_len = p.batch.q_starts[lo + 1] - p.batch.q_starts[lo], kv_len = p.batch.kv_lens[lo], blocks = (q_len + p.bq - 1) / p.bq;
        for (int b0 = 0; b0 < blocks; b0 += 32) { // every warp finds the same
            const int mine = b0 + lane < blocks ? block_of(p, q_len, kv_len, b0 + lane).units() : 0;
            int v = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, v, o);
                v += lane >= o ? up : 0;
            }
            const unsigned past = __ballot_sync(0xffffffffu, walk.block_begin + v > walk.at);
            if (past != 0u) {
                const int at = __ffs(int(past)) - 1;
                walk.block_begin += __shfl_sync(0xffffffffu, v - mine, at);
                walk.index = b0 + at;
                break;
            }
            walk.block_begin += __shfl_sync(0xffffffffu, v, 31);
        }
    }
    __syncthreads(); // the prefix sums have been read
    // rows of a tile past the last page keep what they held: their weights are zero, so they only have to be finite
    for (int i = tid; i < p.stages * kSlot / 16; i += kThreads) {
        reinterpret_cast<uint4 *>(smem)[i] = make_uint4(0, 0, 0, 0);
    }
    // what a column adds to the exponent of its gate at distance x from the block's first query, a * x + b: for a pair of columns a, a, b, b
    const bool capped = p.gates.softcap > 0.f;
    float *columns = reinterpret_cast<float *>(smem + lay.columns);
    const float inv_share = 1.f / float(share), inv_n_c = 1.f / float(n_c);
    for (int i = tid; i < n_columns; i += kThreads) {
        const int c = i / n_c, r = i - c * n_c, qi = r / share, h = c * share + r - qi * share;
        float2 v = make_float2(0.f, 0.f);
        if (qi < p.bq) {
            const float b = p.gates.bias != nullptr ? to_f32(static_cast<const __nv_bfloat16 *>(p.gates.bias)[h]) : 0.f;
            v.x = p.gates.slopes != nullptr ? kLog2e * p.gates.slopes[h] : 0.f;
            v.y = fmaf(v.x, float(qi), -kLog2e * (b + (capped ? p.gates.softcap : 0.f)));
        }
        columns[i / 2 * 4 + i % 2] = v.x;
        columns[i / 2 * 4 + i % 2 + 2] = v.y;
    }
    if (warp == kIssuer) {
        tmem_alloc(base + uint32_t(lay.misc + 20), 512);
        tmem_relinquish();
    }
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = uint32_t(misc[5]), tmem_o = tmem + kMaxColumns;

    if (warp == kProducer || warp == kProducer2) {
        // ================================ K and V tiles ==================================================
        bool alive = true;
        const int page0 = warp == kProducer ? 0 : kPages / 2; // this warp's pages of a tile
        Cursor at;
        bool first_round = true; // nothing has used the slots yet
        Fragment f;
        while (alive && next_fragment(p, walk, f)) {
            const int32_t *table = p.block_table + int64_t(p.batch.seq_ids != nullptr ? p.batch.seq_ids[f.seq] : f.seq) * p.table_stride;
            const int n_pages = (f.block.kv_end + 15) / 16, count = f.upto - f.from;
            auto page_of = [&](int t) { // of lane's page in tile t of the block; -1: none
                const int i = (f.block.tile0 + t) * kPages + (lane & (kPages - 1));
                int page = t < f.upto && i < n_pages ? table[i] : -1;
                if (t < f.upto && i < n_pages && (page < 0 || page >= p.num_pages)) {
                    atomicOr(p.error_flag, kErrBadPage);
                    page = 0;
                }
                return page;
            };
            // the operand of every kv head of one tile
            auto load = [&](int page, bool is_v) {
                const int here = min(max(__popc(__ballot_sync(0xffffffffu, lane < kPages && page >= 0)) - page0, 0), kPages / 2); // (the first ones)
                int c3[kPages / 2];
#pragma unroll
                for (int i = 0; i < kPages / 2; ++i) {
                    c3[i] = int((p.page0 + max(__shfl_sync(0xffffffffu, page, page0 + i), 0)) * 2) + (is_v ? 1 : 0);
                }
                for (int c = 0; c < groups && alive; ++c) {
                    if (!first_round && !__all_sync(0xffffffffu, wait_or_abort(bar(kBarFree + at.slot), at.parity ^ 1u, s_abort))) {
                        alive = false;
                        break;
                    }
                    const uint32_t dst = base + uint32_t(at.slot * kSlot), full = bar(kBarFull + at.slot);
                    if (elect_one()) {
                        mbar_arrive_expect_tx(full, uint32_t(here) * 4096);
#pragma unroll
                        for (int i = 0; i < kPages / 2; ++i) {
                            if (i < here) {
                                if (is_v) { // one box per page: [half of the dims][16 tokens][128 B]
                                    tma_load_5d(dst + uint32_t((page0 + i) * 4096), &map_v, 0, 0, 0, c, c3[i], full);
                                } else { // [half of the dims][128 tokens][128 B]
                                    tma_load_4d(dst + uint32_t((page0 + i) * 2048), &map_k, 0, 0, c, c3[i], full);
                                    tma_load_4d(dst + uint32_t(kSlot / 2 + (page0 + i) * 2048), &map_k, 64, 0, c, c3[i], full);
                                }
                            }
                        }
                    }
                    __syncwarp();
                    at.next(p.stages);
                    first_round = first_round && at.slot != 0;
                }
            };
            int page = page_of(f.from), ahead = page_of(f.from + 1);
            load(page, false);
            for (int i = 0; i < count && alive; ++i) {
                const int two_ahead = page_of(f.from + i + 2);
                if (i + 1 < count) {
                    load(ahead, false);
                }
                load(page, true);
                page = ahead;
                ahead = two_ahead;
            }
        }
        if (!alive && lane == 0) {
            give_up();
        }
    } else if (warp == kIssuer) {
        // ================================ MMAs ===========================================================
        auto wait = [&](uint32_t at, int parity) { return __all_sync(0xffffffffu, wait_or_abort(at, uint32_t(parity), s_abort)) != 0; };
        const uint32_t idesc_s = make_idesc(true, false, kBk, n_c), idesc_o = make_idesc(true, false, kD, n_c) | (1u << 15); // A MN-major
        // low words of the operands' descriptors count 16-byte steps; the high words are the same for all
        const uint64_t slots_k = smem_desc_sw128(base, 0, 1024), slots_v = smem_desc_sw128(base, 2048, 1024);
        const uint64_t q_desc = smem_desc_sw128(base + uint32_t(lay.q), 0, 1024), p_desc = smem_desc_sw128(base + uint32_t(lay.w), 0, 1024);
        const uint32_t group_bytes = uint32_t(n_c) * 256, half_bytes = uint32_t(n_c) * 128;
        bool ok = true;
        Cursor at;
        int n = 0, n_fragments = 0;
        auto scores = [&](int tile_no, bool waits) { // S of tile tile_no; waits: until the tile before it has been read
            uint64_t b = q_desc;
            uint32_t d = tmem, done = s_bar(tile_no, 0), read = bar(kBarRead);
            for (int c = 0; c < groups && ok; ++c, b = desc_at(b, group_bytes), d += uint32_t(n_c), done += 8, read += 8) {
                ok = (!waits || wait(read, (tile_no - 1) & 1)) && wait(bar(kBarFull + at.slot), int(at.parity));
                tc_fence_after();
                const uint64_t a = desc_at(slots_k, uint32_t(at.slot * kSlot)), b2 = desc_at(b, half_bytes);
                if (ok && elect_one()) {
#pragma unroll
                    for (int ks = 0; ks < kD / 16; ++ks) {
                        umma_f16(d, desc_at(a, (ks >> 2) * (kSlot / 2) + (ks & 3) * 32), desc_at(ks < 4 ? b : b2, (ks & 3) * 32), idesc_s, ks > 0 ? 1u : 0u);
                    }
                    umma_commit(done);
                    umma_commit(bar(kBarFree + at.slot));
                }
                __syncwarp();
                at.next(p.stages);
            }
        };
        Fragment f;
        for (; ok && next_fragment(p, walk, f); ++n_fragments) {
            const int count = f.upto - f.from;
            ok = wait(bar(kBarQ), n_fragments & 1);
            scores(n, n > 0);
            for (int i = 0; i < count && ok; ++i, ++n) {
                if (i + 1 < count) {
                    scores(n + 1, true);
                }
                ok = ok && wait(bar(kBarP), n & 1);
                if (i == 0 && n_fragments > 0) {
                    ok = ok && wait(bar(kBarO), (n_fragments - 1) & 1);
                }
                uint64_t b = p_desc;
                uint32_t d = tmem_o, done = pv_bar(n, 0);
                for (int c = 0; c < groups && ok; ++c, b = desc_at(b, group_bytes), d += uint32_t(n_c), done += 8) {
                    ok = wait(bar(kBarFull + at.slot), int(at.parity));
                    tc_fence_after();
                    const uint64_t a = desc_at(slots_v, uint32_t(at.slot * kSlot)), b2 = desc_at(b, half_bytes);
                    if (ok && elect_one()) {
#pragma unroll
                        for (int kk = 0; kk < kBk / 16; ++kk) { // 16 keys: one page
                            umma_f16(d, desc_at(a, kk * 4096), desc_at(kk < 4 ? b : b2, (kk & 3) * 32), idesc_o, i > 0 || kk > 0 ? 1u : 0u);
                        }
                        umma_commit(done);
                        umma_commit(bar(kBarFree + at.slot));
                    }
                    __syncwarp();
                    at.next(p.stages);
                }
            }
        }
        if (!ok && lane == 0) {
            give_up();
        }
        __syncwarp();
    } else {
        // ================================ weights, mixing, output ========================================
        bool dead = false; // a thread whose wait ran out keeps walking, so that the named barriers see all of them
        auto wait = [&](uint32_t at, int parity) {
            if (!dead && !wait_or_abort(at, uint32_t(parity), s_abort)) {
                dead = true;
                give_up();
            }
            __syncwarp();
        };
        auto arrive = [&](int which) {
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(bar(which));
            }
        };
        const int quarter = warp & 3, part = warp >> 2, units = n_c / 8; // lanes of TMEM, and which of every four chunks or units
        const int key = quarter * 32 + lane;
        const uint32_t lanes = uint32_t(quarter * 32) << 16;
        const float to_exp = capped ? 2.f * kLog2e * p.scale / p.gates.softcap : -kLog2e * p.scale, cap2 = 2.f * kLog2e * p.gates.softcap;
        const Pair to_exp2 = pair(to_exp, to_exp), ones = pair(1.f, 1.f);
        const uint32_t w_s = base + uint32_t(lay.w);
        // a weight of column r: row r, 16-byte chunk (key / 8) ^ (r mod 8) of the row's 64-key half; this lane addresses the row of column
        // lane % 8 for keys 8 (lane / 8) .. of the warp's 32
        const uint32_t w_lane = w_s + uint32_t((quarter >> 1) * n_c * 128 + (lane & 7) * 128 + ((((quarter & 1) * 4 + (lane >> 3)) ^ (lane & 7)) << 4));

        // talk as mma operands, and the head whose row this lane addresses: byte offset of its kv head, place in the group
        uint32_t talk[MT][MT][4];
        int head_base[MT], head_at[MT];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
            for (int kt = 0; kt < MT; ++kt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float v[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const int h = mt * 16 + (lane >> 2) + (e & 1) * 8, g = kt * 16 + 2 * (lane & 3) + (e >> 1) * 8 + x;
                        v[x] = 0.f;
                        if (h < nh && g < nh) {
                            v[x] = p.gates.talk != nullptr ? to_f32(static_cast<const __nv_bfloat16 *>(p.gates.talk)[h * nh + g]) : float(h == g);
                        }
                    }
                    talk[mt][kt][e] = pack2<false>(v[0], v[1]);
                }
            }
            const int head = mt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
            head_base[mt] = head < nh ? head / share * n_c * kBk * 2 : -1;
            head_at[mt] = head % share;
        }

        auto load_q = [&](const Fragment &f) {
            for (int i = tid; i < n_columns * 16; i += kWorkers * 32) {
                const int col = i >> 4, cc = i & 15, c = small_div(col, inv_n_c), r = col - c * n_c, qi = small_div(r, inv_share), h = c * share + r - qi * share;
                uint4 v = make_uint4(0, 0, 0, 0);
                if (qi < f.block.n_q) {
                    v = *reinterpret_cast<const uint4 *>(p.q + ((f.row0 + qi) * nh + h) * kD + cc * 8);
                }
                *reinterpret_cast<uint4 *>(smem + lay.q + c * n_c * kD * 2 + (cc >> 3) * n_c * 128 + r * 128 + (((cc & 7) ^ (r & 7)) << 4)) = v;
            }
            fence_proxy_async_smem();
            arrive(kBarQ);
        };

        Fragment f, next;
        bool more = next_fragment(p, walk, f);
        if (more) {
            load_q(f);
        }
        int n = 0;
        while (more) {
            const Block &blk = f.block;
            for (int t = f.from; t < f.upto; ++t, ++n) {
                const int first = (blk.tile0 + t) * kBk;
                const bool edge = first + kBk > blk.pos0 + 1 || (p.batch.window > 0 && first + p.batch.window < blk.pos0 + blk.n_q);
                float ago[4]; // from this thread's keys to the block's first query
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    ago[k] = float(blk.pos0 - first - quarter * 32 - (lane >> 2) - 8 * k);
                }
                const int chunks = (n_c + kChunk - 1) / kChunk;
                for (int c = 0, k = 0; c < groups; ++c) {
                    for (int piece = 0; piece < chunks; ++piece, ++k) {
                        if ((k & 3) != part) {
                            continue;
                        }
                        const int col0 = c * n_c + piece * kChunk, n_units = min(kChunk, n_c - piece * kChunk) / 8;
                        wait(s_bar(n, c), (n >> 1) & 1);
                        tc_fence_after();
                        uint32_t weights[kChunk / 8][4]; // f16 pairs of four keys
#pragma unroll
                        for (int half = 0; half < 2; ++half) { // 16 keys at a time, two of them this thread's
                            uint32_t raw[16]; // (columns past the chunk are S or O columns all the same, and go unused)
                            tmem_ld_fragments(tmem + lanes + (uint32_t(16 * half) << 16) + uint32_t(col0), raw);
                            tmem_wait_ld();
                            if (half == 1) {
                                tc_fence_before();
                                arrive(kBarRead + c);
                            }
                            const Pair ago_a = pair(ago[2 * half], ago[2 * half]), ago_b = pair(ago[2 * half + 1], ago[2 * half + 1]);
#pragma unroll
                            for (int u = 0; u < kChunk / 8; ++u) {
                                if (u >= n_units) {
                                    break;
                                }
                                const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(columns + 2 * (col0 + u * 8) + 4 * (lane & 3));
                                Pair x = pair(__uint_as_float(raw[4 * u]), __uint_as_float(raw[4 * u + 1]));
                                Pair y = pair(__uint_as_float(raw[4 * u + 2]), __uint_as_float(raw[4 * u + 3]));
                                const Pair a = fma2(k2.x, ago_a, k2.y), b = fma2(k2.x, ago_b, k2.y);
                                if (capped) { // softcap tanh(y) = softcap - 2 softcap / (1 + e^(2 y))
                                    x = one_plus_ex2(mul2(x, to_exp2), ones);
                                    y = one_plus_ex2(mul2(y, to_exp2), ones);
                                    const Pair r = rcp4(x, y, cap2), first_key = fma2(r, y, a);
                                    y = fma2(r, x, b);
                                    x = first_key;
                                } else {
                                    x = fma2(x, to_exp2, a);
                                    y = fma2(y, to_exp2, b);
                                }
                                x = one_plus_ex2(x, ones);
                                y = one_plus_ex2(y, ones);
                                const Pair r = rcp4(x, y, kWeightUnit);
                                float w[4];
                                unpair(mul2(r, y), w[0], w[1]);
                                unpair(mul2(r, x), w[2], w[3]);
                                if (edge) {
                                    const float window = p.batch.window > 0 ? float(p.batch.window) : INFINITY;
                                    const int col = piece * kChunk + u * 8 + 2 * (lane & 3);
#pragma unroll
                                    for (int i = 0; i < 4; ++i) {
                                        const float far = ago[2 * half + i / 2] + float(small_div(col + i % 2, inv_share));
                                        w[i] = far >= 0.f && far < window ? w[i] : 0.f;
                                    }
                                }
                                weights[u][2 * half] = pack2<false>(w[0], w[1]);
                                weights[u][2 * half + 1] = pack2<false>(w[2], w[3]);
                            }
                        }
                        if (n > 0) {
                            wait(pv_bar(n - 1, c), ((n - 1) >> 1) & 1);
                        }
                        const uint32_t at = w_lane + uint32_t(c * n_c * kBk * 2 + piece * kChunk * 128);
#pragma unroll
                        for (int u = 0; u < kChunk / 8; ++u) {
                            if (u < n_units) {
                                stmatrix_x4_trans(at + uint32_t(u * 1024), weights[u][0], weights[u][1], weights[u][2], weights[u][3]);
                            }
                        }
                    }
                }
                named_barrier_sync(1, kWorkers * 32); // weights of all heads are in place
                constexpr int kAtOnce = MT == 1 ? 4 : 2;
                // a warp per query and half of the keys: 16 keys of all heads at a time, results in place of the operands
                for (int item = warp; item < blk.n_q * 2; item += kWorkers) {
                    const int half = (item & 1) * n_c * 128, q_row = (item >> 1) * share;
                    uint32_t row_at[MT];
#pragma unroll
                    for (int kt = 0; kt < MT; ++kt) {
                        const int row = q_row + head_at[kt];
                        row_at[kt] = w_s + uint32_t(head_base[kt] + half + row * 128 + (((lane >> 4) ^ (row & 7)) << 4));
                    }
#pragma unroll
                    for (int kb0 = 0; kb0 < 4; kb0 += kAtOnce) {
                        uint32_t in[kAtOnce][MT][4], at[kAtOnce][MT];
#pragma unroll
                        for (int b = 0; b < kAtOnce; ++b) {
#pragma unroll
                            for (int kt = 0; kt < MT; ++kt) {
                                at[b][kt] = head_base[kt] < 0 ? base + uint32_t(lay.misc) : row_at[kt] ^ uint32_t((kb0 + b) << 5);
                                ldmatrix_x4_trans(in[b][kt], at[b][kt]);
                            }
                        }
                        __syncwarp();
#pragma unroll
                        for (int mt = 0; mt < MT; ++mt) {
                            float y[kAtOnce][2][4] = {}; // [16 keys][8 of them]
#pragma unroll
                            for (int kt = 0; kt < MT; ++kt) {
#pragma unroll
                                for (int b = 0; b < kAtOnce; ++b) {
                                    mma_f16(y[b][0], talk[mt][kt], in[b][kt][0], in[b][kt][1]);
                                    mma_f16(y[b][1], talk[mt][kt], in[b][kt][2], in[b][kt][3]);
                                }
                            }
#pragma unroll
                            for (int b = 0; b < kAtOnce; ++b) { // (rows of padding heads: zeros, to where zeros lie)
                                stmatrix_x4(at[b][mt], pack2<true>(y[b][0][0], y[b][0][1]), pack2<true>(y[b][0][2], y[b][0][3]),
                                            pack2<true>(y[b][1][0], y[b][1][1]), pack2<true>(y[b][1][2], y[b][1][3]));
                            }
                        }
                    }
                }
                fence_proxy_async_smem();
                arrive(kBarP);
            }
            more = next_fragment(p, walk, next);
            if (more) {
                load_q(next); // every S of this fragment is done: its queries are free
            }
            // ---- the block's output, whole or in pieces ----
            wait(pv_bar(n - 1, groups - 1), ((n - 1) >> 1) & 1);
            tc_fence_after();
            const bool whole = f.from == 0 && f.upto == blk.n_tiles;
            const int64_t slot = int64_t(n_columns) * kD;
            auto slot_of = [&](int cta, bool begins) { return p.partials + (int64_t(cta) * 2 + (begins ? 1 : 0)) * slot; };
            auto each_unit = [&](auto &&body) {
                for (int g = part; g < groups * units; g += 4) {
                    body(g * 8);
                }
            };
            auto store = [&](int col, const float (&v)[8]) {
                const int c = small_div(col, inv_n_c), r = col - c * n_c;
                int qi = small_div(r, inv_share), hl = r - qi * share;
                __nv_bfloat16 *dst = p.out + (f.row0 + qi) * p.out_stride + int64_t(c * share + hl) * kD + key;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    if (qi < blk.n_q) {
                        *dst = __float2bfloat16_rn(v[i] * (1.f / kWeightUnit));
                    }
                    dst += kD;
                    if (++hl == share) { // the next query's first head of the group
                        hl = 0;
                        ++qi;
                        dst += p.out_stride - int64_t(share) * kD;
                    }
                }
            };
            if (whole) {
                each_unit([&](int col) {
                    float v[8];
                    tmem_ld8(tmem_o + lanes + uint32_t(col), v);
                    store(col, v);
                });
                tc_fence_before();
                arrive(kBarO);
            } else {
                float *own = slot_of(int(blockIdx.x), f.from == 0);
                each_unit([&](int col) {
                    float v[8];
                    tmem_ld8(tmem_o + lanes + uint32_t(col), v);
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        own[int64_t(col + i) * kD + key] = v[i];
                    }
                });
                tc_fence_before();
                arrive(kBarO);
                // CTAs that hold tiles of the block: share c holds unit u iff c is the largest with c * total < (u + 1) * ctas
                const int64_t unit0 = f.block_begin + kBlockCost;
                const int first_cta = int(((unit0 + 1) * ctas - 1) / total), last_cta = int(((unit0 + blk.n_tiles) * ctas - 1) / total);
                __threadfence();
                named_barrier_sync(1, kWorkers * 32);
                if (tid == 0) {
                    misc[6] = atomicAdd(p.counters + first_cta, 1) == last_cta - first_cta;
                    if (misc[6]) {
                        p.counters[first_cta] = 0;
                    }
                }
                named_barrier_sync(1, kWorkers * 32);
                const bool last = misc[6] != 0;
                if (last) {
                    __threadfence();
                    each_unit([&](int col) {
                        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                        for (int cta = first_cta; cta <= last_cta; ++cta) {
                            const float *from = slot_of(cta, cta == first_cta) + int64_t(col) * kD + key;
#pragma unroll
                            for (int i = 0; i < 8; ++i) {
                                v[i] += __ldcg(from + i * kD);
                            }
                        }
                        store(col, v);
                    });
                }
                named_barrier_sync(1, kWorkers * 32); // `last` has been read
            }
            f = next;
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == kIssuer) {
        tmem_dealloc(tmem, 512);
    }
}

int sm_count() {
    static int n = [] {
        int dev = 0, v = 0;
        LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
        LLAISYS_CUDA_CHECK(cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev));
        return v;
    }();
    return n;
}

template <int MT>
void launch(cudaStream_t s, const CUtensorMap &map_k, const CUtensorMap &map_v, const Params &p, size_t smem, int grid, bool overlap) {
    auto kernel = attention_gates_tc_kernel<MT>;
    LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit));
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
    LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, map_k, map_v, p));
}

} // namespace

void attention_gates_tc_scratch(size_t *floats, size_t *counters) {
    *floats = size_t(sm_count()) * 2 * kMaxColumns * kD;
    *counters = size_t(sm_count());
}

int attention_gates_tc(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                       const GateArgs &gates, const AttnOut &out, const AttnScratch &scratch) {
    if (dtype != LLAISYS_DTYPE_BF16 || kv.d != kD || kv.vDim() != kD || kv.page_size != 16 || kv.block_table == nullptr ||
        kv.tma_tile_desc == nullptr || batch.q_starts == nullptr || batch.kv_lens == nullptr || kv.nkvh <= 0 || kv.nkvh > kMaxGroups ||
        batch.nh > 32 || batch.nh % kv.nkvh != 0 || batch.n_seqs <= 0 || batch.n_seqs > 8192 || batch.max_q_len < 8 || batch.keep_first != 0 ||
        out.out == nullptr || out.part != nullptr || out.row_scale != nullptr || reinterpret_cast<uintptr_t>(q) % 16 != 0) {
        return -1;
    }
    Params p{};
    p.share = batch.nh / kv.nkvh;
    auto padded = [&](int bq) { return (bq * p.share + 15) / 16 * 16; };
    for (int bq = 1; bq <= std::min(batch.max_q_len, 64) && kv.nkvh * padded(bq) <= kMaxColumns; ++bq) {
        p.bq = bq;
    }
    if (p.bq < 4) {
        return -1;
    }
    p.groups = kv.nkvh;
    p.n_c = padded(p.bq);
    const int n_columns = p.groups * p.n_c;
    p.stages = kMaxStages;
    while (p.stages > 2 && Layout(p.stages, n_columns).total > kSmemLimit) {
        --p.stages;
    }
    const Layout lay(p.stages, n_columns);
    const int grid = sm_count();
    if (lay.total > kSmemLimit || scratch.partials == nullptr || scratch.counters == nullptr || scratch.error_flag == nullptr ||
        scratch.partials_floats < size_t(grid) * 2 * size_t(n_columns) * kD || scratch.counters_len < size_t(grid)) {
        return -1;
    }
    p.batch = batch;
    p.gates = gates;
    p.q = static_cast<const __nv_bfloat16 *>(q);
    p.out = static_cast<__nv_bfloat16 *>(out.out);
    p.out_stride = out.row_stride ? out.row_stride : int64_t(batch.nh) * kD;
    p.scale = scale;
    p.page0 = kv.tma_page0;
    p.block_table = kv.block_table;
    p.table_stride = kv.table_stride;
    p.num_pages = kv.num_pages;
    p.partials = scratch.partials;
    p.counters = scratch.counters;
    p.error_flag = scratch.error_flag;
    CUtensorMap map_k, map_v;
    std::memcpy(&map_k, kv.tma_tile_desc, sizeof(map_k));
    std::memcpy(&map_v, static_cast<const unsigned char *>(kv.tma_tile_desc) + sizeof(map_k), sizeof(map_v));
    auto s = static_cast<cudaStream_t>(stream);
    batch.nh <= 16 ? launch<1>(s, map_k, map_v, p, size_t(lay.total), grid, kv.overlap_launch)
                   : launch<2>(s, map_k, map_v, p, size_t(lay.total), grid, kv.overlap_launch);
    check_launch("attention_gates_tc");
    return 0;
}

} // namespace llaisys::kernels
