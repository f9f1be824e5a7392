// Attention over pages of latents (layers with one kv head whose V rows are the beginning of their K rows) on the 5th-generation tensor
// cores: decode, and chunks of few tokens. All heads read the SAME row per key, so a row is fetched once and serves as K and as V.
//
// Roofline: HBM while the queries are few: (rank + turned dims) * 2 bytes per cached token and sequence.
//
// Both products are transposed, so that keys and value dims fill the 128 rows of an MMA and the few (query, head) pairs are its N:
//     S^T [128 keys, N]  = K Q^T           A = K tile (K-major),  B = queries
//     O^T [128 dims, N] += V^T P           A = V tile (MN-major: the same bytes), B = weights
// A UNIT is (sequence, group of up to 32 heads, block of queries that fills the 32 columns); it visits its keys 128 at a time (a TILE, 8
// pages). The tiles of all units form one line that is cut into equal pieces, one per SM; a unit inside a piece is stored finished, one
// that is cut leaves (O, max, sum) per piece, and a second small launch merges those in the order of the pieces.
//
// Per CTA (one per SM; a tile of rank 512 takes 144 KiB):
//   warps 0-3   one key per thread: scale, mask, column maxima (transposing shuffles, then across the warps), weights to shared memory,
//               O rescaled in TMEM only when a column's maximum grew by more than 2^8; queries of the next unit; results
//   warp 4      issues the MMAs (an elected lane); waits for K pair by pair, frees V pair by pair
//   warps 5, 6  TMA of pages, 64 dims x 16 tokens per box, half of a tile's pages each, into a ring of PAIRS (128 dims x 128 keys, 32 KiB)
//               and one slot for the dims behind the last pair, which are no part of V
// Every wait is bounded; one that runs out sets the error word and the CTA winds down. No cluster launch, no multicast.
#include "kernels.hpp"
#include "launch_utils.cuh"
#include "matrix_map.cuh"
#include "tcgen05_utils.cuh"

#include <algorithm>
#include <mutex>

namespace llaisys::kernels {

namespace {

constexpr int kTile = 128, kPage = 16, kPagesPerTile = kTile / kPage;
constexpr int kChunkBytes = kTile * 128, kPairBytes = 2 * kChunkBytes; // 64 dims and 128 dims of a tile
constexpr int kMaxPairs = 4, kMaxRing = 6;
constexpr int kThreads = 224, kIssuer = 4, kProducer = 5;
constexpr int kUnitCost = 1; // what a unit costs besides its tiles, in tiles
constexpr int kMinPiece = 3;
constexpr int kErrTimeout = 8;
constexpr float kRescaleThreshold = 8.f; // log2 units
constexpr int kSmemLimit = 227 * 1024;

enum : int {
    kBarFull = 0,                    // [ring] producers -> issuer: a pair landed
    kBarFree = kBarFull + kMaxRing,  // [ring] issuer (commit) -> producers: a pair has been used as V
    kBarTail = kBarFree + kMaxRing,  // producers -> issuer: the dims behind the pairs landed
    kBarS,                           // issuer (commit) -> softmax: S is there; -> producers: the tail slot is free
    kBarP,                           // softmax (128) -> issuer: S read, weights stored, O rescaled
    kBarO,                           // issuer (commit) -> softmax: O stable, weights used
    kBarQ,                           // softmax (128) -> issuer: queries of the next unit stored
    kNumBars
};

struct Params {
    const int32_t *block_table;
    int32_t table_stride, num_pages;
    const int32_t *seq_ids, *kv_lens, *q_starts; // q_starts null: one query per sequence
    int32_t n_seqs, nh;
    int32_t group, n_groups, block; // heads of a group, groups, queries of a block
    int32_t dim, rank;              // elements of a row, of its V part
    int32_t chunks, pairs, ring;    // 64-dim pieces of a row; pairs of them that hold V; slots of the ring
    const void *q;
    void *out;
    long long out_stride;
    const float *row_scale;
    float scale_log2;
    float *partials;
    int32_t *error_flag;
};

struct SeqGeom {
    int q_start, q_len, kv_len, off, tiles, units, length; // length: on the line
};

__device__ __forceinline__ SeqGeom seq_geom(const Params &p, int a) {
    SeqGeom g;
    g.q_start = p.q_starts != nullptr ? p.q_starts[a] : a;
    g.q_len = p.q_starts != nullptr ? p.q_starts[a + 1] - g.q_start : 1;
    g.kv_len = min(max(p.kv_lens[a], g.q_len), p.table_stride * kPage);
    g.q_len = min(g.q_len, g.kv_len);
    g.off = g.kv_len - g.q_len; // query t sees keys j <= t + off
    g.tiles = (g.kv_len + kTile - 1) / kTile;
    g.units = (g.q_len + p.block - 1) / p.block * p.n_groups;
    g.length = g.units * (g.tiles + kUnitCost);
    return g;
}

// Length of the line, and (kFind) the sequence that holds position `at` with the position of its beginning; at < 0: the first position
// of piece -1 - at of n_pieces, found by the same pass where every thread has at most one sequence. For whole CTAs of whole warps;
// s_scan: 34 ints of shared memory.
__device__ __forceinline__ int piece_length(int line, int n_pieces) {
    const int even = (line + n_pieces - 1) / n_pieces;
    return even < kMinPiece ? kMinPiece : even;
}

template <bool kFind>
__device__ __forceinline__ int scan_line(const Params &p, int at, int n_pieces, int *s_scan, int &seq, int &seq_begin) {
    const int tid = int(threadIdx.x), lane = tid & 31, warp = tid >> 5, n_warps = int(blockDim.x) >> 5;
    int before = 0;
    for (int base = 0; base < p.n_seqs; base += int(blockDim.x)) {
        const int len = base + tid < p.n_seqs ? seq_geom(p, base + tid).length : 0;
        int incl = len;
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
            const int v = __shfl_up_sync(0xffffffffu, incl, o);
            incl += lane >= o ? v : 0;
        }
        __syncthreads();
        if (lane == 31) {
            s_scan[warp] = incl;
        }
        __syncthreads();
        int warps_before = 0, total = 0;
        for (int w = 0; w < n_warps; ++w) {
            warps_before += w < warp ? s_scan[w] : 0;
            total += s_scan[w];
        }
        const int begin = before + warps_before + incl - len;
        if (kFind && at < 0) { // (a single round: the total is known)
            at = (-1 - at) * piece_length(total, n_pieces);
        }
        if (kFind && len > 0 && begin <= at && at < begin + len) {
            s_scan[32] = base + tid;
            s_scan[33] = begin;
        }
        before += total;
    }
    if (kFind) {
        __syncthreads();
        seq = s_scan[32];
        seq_begin = s_scan[33];
    }
    return before;
}

struct Walker {
    int a, seq_begin;
    SeqGeom g;
};
struct Fragment {
    int unit, t0, t1; // tiles [t0, t1) of the unit
    int begin;        // of the unit on the line
};
// The fragment that starts at or after `pos` and before piece_end; `pos` moves on to its first tile.
__device__ __forceinline__ bool locate(const Params &p, Walker &w, int &pos, int piece_end, Fragment &f) {
    while (pos < piece_end) {
        while (pos >= w.seq_begin + w.g.length) {
            if (w.a + 1 >= p.n_seqs) {
                return false;
            }
            w.seq_begin += w.g.length;
            ++w.a;
            w.g = seq_geom(p, w.a);
        }
        const int per = w.g.tiles + kUnitCost, x = pos - w.seq_begin, unit = x / per, t = x - unit * per;
        if (t >= w.g.tiles) {
            pos += per - t;
            continue;
        }
        f.unit = unit;
        f.t0 = t;
        f.t1 = min(w.g.tiles, t + (piece_end - pos));
        f.begin = w.seq_begin + unit * per;
        return true;
    }
    return false;
}

// v[i] of 32 lanes, i < N -> in lane c the combination of every lane's v[c % N]
template <int N, typename Op>
__device__ __forceinline__ float reduce_columns(float (&v)[N], int lane, Op op) {
    if constexpr (N == 16) {
#pragma unroll
        for (int i = 0; i < N; ++i) {
            v[i] = op(v[i], __shfl_xor_sync(0xffffffffu, v[i], 16));
        }
    }
#pragma unroll
    for (int o = N / 2; o > 0; o /= 2) {
        const bool upper = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float keep = upper ? v[i + o] : v[i], send = upper ? v[i] : v[i + o];
            v[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, o));
        }
    }
    return v[0];
}

template <int N>
__device__ __forceinline__ void load_columns(uint32_t taddr, float (&v)[N]) {
    if constexpr (N == 32) {
        tmem_ld32(taddr, v);
    } else {
        tmem_ld16(taddr, v);
        tmem_wait_ld();
    }
}
template <int N>
__device__ __forceinline__ void store_columns(uint32_t taddr, const float (&v)[N]) {
    if constexpr (N == 32) {
        tmem_st32(taddr, v);
    } else {
        tmem_st16(taddr, v);
    }
}

constexpr int partial_floats(int n, int pairs) { return n * (pairs * 128) + 2 * n; }

template <bool kBf16, int N>
__global__ void __launch_bounds__(kThreads, 1) attention_latent_kernel(const __grid_constant__ CUtensorMap tmap, Params p) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    __shared__ uint64_t s_bars[kNumBars];
    __shared__ float s_max[2][4][N];
    __shared__ int s_scan[34];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort_word;
    volatile int *s_abort = &s_abort_word;
    const int tid = int(threadIdx.x), warp = tid >> 5, lane = tid & 31;
    const uint32_t raw = smem_u32(smem_raw), base = (raw + 1023u) & ~1023u;
    const uint32_t ring_u32 = base, tail_u32 = ring_u32 + uint32_t(p.ring) * kPairBytes;
    const bool has_tail = p.chunks > 2 * p.pairs;
    const uint32_t q_u32 = tail_u32 + (has_tail ? kChunkBytes : 0), p_u32 = q_u32 + uint32_t(p.chunks) * (N * 128);
    const uint32_t bars = smem_u32(s_bars);
    auto bar = [&](int which) { return bars + uint32_t(which) * 8; };

    // this CTA's piece (index arrays are older than the kernel before this one: see KVView::overlap_launch)
    Walker walker;
    int line;
    {
        const bool one_round = p.n_seqs <= kThreads;
        line = one_round ? scan_line<true>(p, -1 - int(blockIdx.x), int(gridDim.x), s_scan, walker.a, walker.seq_begin)
                         : scan_line<false>(p, 0, 0, s_scan, walker.a, walker.seq_begin);
        const int piece = piece_length(line, int(gridDim.x));
        if (int(blockIdx.x) * piece >= line) {
            grid_dependency_wait();
            grid_launch_dependents();
            return;
        }
        if (!one_round) {
            scan_line<true>(p, int(blockIdx.x) * piece, 0, s_scan, walker.a, walker.seq_begin);
        }
        walker.g = seq_geom(p, walker.a);
    }
    const int piece = piece_length(line, int(gridDim.x)), piece_begin = int(blockIdx.x) * piece, piece_end = min(line, piece_begin + piece);
    if (tid == 0) {
        for (int i = 0; i < kNumBars; ++i) {
            const int count = i == kBarP || i == kBarQ ? 128 : ((i >= kBarFull && i < kBarFree) || i == kBarTail ? 2 : 1);
            mbar_init(bar(i), uint32_t(count));
        }
        s_abort_word = 0;
        mbar_init_fence();
    }
    constexpr int kColO = 32;
    constexpr uint32_t kCols = N == 32 ? 256 : 128;
    static_assert(kColO + kMaxPairs * N <= int(kCols), "TMEM columns");
    if (warp == kIssuer) {
        tmem_alloc(smem_u32(&s_tmem), kCols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    grid_dependency_wait();
    grid_launch_dependents();
    auto give_up = [&]() {
        s_abort_word = 1;
        atomicOr(p.error_flag, kErrTimeout);
    };
    auto wait = [&](int which, int phase) { return __all_sync(0xffffffffu, wait_or_abort(bar(which), uint32_t(phase) & 1u, s_abort)); };

    if (warp >= kProducer) {
        const int half = warp - kProducer;
        bool ok = true;
        int slot = 0, round = 0, tile_no = 0;
        Fragment f;
        for (int pos = piece_begin; ok && locate(p, walker, pos, piece_end, f); pos += f.t1 - f.t0) {
            const int n_pages = (walker.g.kv_len + kPage - 1) / kPage;
            const int32_t *table = p.block_table + (long long)(p.seq_ids != nullptr ? p.seq_ids[walker.a] : walker.a) * p.table_stride;
            // (behind the last page: that page again -- its rows enter the products with weight zero and only have to be finite)
            auto entry = [&](int t) { return lane < 4 && t < f.t1 ? table[min(t * kPagesPerTile + half * 4 + lane, n_pages - 1)] : 0; };
            int pages = entry(f.t0);
            for (int t = f.t0; t < f.t1 && ok; ++t, ++tile_no) {
                if ((pages < 0 || pages >= p.num_pages)) {
                    atomicOr(p.error_flag, kErrBadPage);
                    pages = 0;
                }
                int row[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    row[i] = __shfl_sync(0xffffffffu, pages, i) * kPage;
                }
                const int next = entry(t + 1);
                for (int pair = 0; pair < p.pairs && ok; ++pair) {
                    if (round > 0) {
                        ok = wait(kBarFree + slot, round - 1);
                    }
                    const int n = min(p.chunks - 2 * pair, 2);
                    if (ok && elect_one()) {
                        const uint32_t dst = ring_u32 + uint32_t(slot) * kPairBytes + uint32_t(half) * (4 * 2048);
                        mbar_arrive_expect_tx(bar(kBarFull + slot), uint32_t(4 * n) * 2048u);
#pragma unroll
                        for (int c = 0; c < 2; ++c) {
#pragma unroll
                            for (int i = 0; i < 4; ++i) {
                                if (c < n) {
                                    tma_load_2d(dst + uint32_t(c * kChunkBytes + i * 2048), &tmap, (2 * pair + c) * 64, row[i], bar(kBarFull + slot));
                                }
                            }
                        }
                    }
                    __syncwarp();
                    if (++slot == p.ring) {
                        slot = 0;
                        ++round;
                    }
                }
                if (has_tail && ok) {
                    if (tile_no > 0) {
                        ok = wait(kBarS, tile_no - 1);
                    }
                    if (ok && elect_one()) {
                        mbar_arrive_expect_tx(bar(kBarTail), 4u * 2048u);
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            tma_load_2d(tail_u32 + uint32_t(half) * (4 * 2048) + uint32_t(i * 2048), &tmap, 2 * p.pairs * 64, row[i], bar(kBarTail));
                        }
                    }
                    __syncwarp();
                }
                pages = next;
            }
        }
        if (!ok && lane == 0) {
            give_up();
        }
    } else if (warp == kIssuer) {
        const uint32_t idesc_s = make_idesc(kBf16, false, kTile, N), idesc_o = idesc_s | (1u << 15); // (A MN-major)
        bool ok = true;
        int slot_s = 0, round_s = 0, slot_o = 0, tile_no = 0, n_fragments = 0;
        Fragment f;
        for (int pos = piece_begin; ok && locate(p, walker, pos, piece_end, f); pos += f.t1 - f.t0, ++n_fragments) {
            ok = wait(kBarQ, n_fragments);
            for (int t = f.t0; t < f.t1 && ok; ++t, ++tile_no) {
                for (int pair = 0; pair < p.pairs && ok; ++pair) {
                    ok = wait(kBarFull + slot_s, round_s);
                    tc_fence_after();
                    const int n = min(p.chunks - 2 * pair, 2);
                    const uint32_t k = ring_u32 + uint32_t(slot_s) * kPairBytes, q = q_u32 + uint32_t(2 * pair) * (N * 128);
                    if (ok && elect_one()) {
#pragma unroll
                        for (int c = 0; c < 2; ++c) {
                            if (c < n) {
#pragma unroll
                                for (int ks = 0; ks < 4; ++ks) {
                                    umma_f16(tmem, smem_desc_sw128(k + uint32_t(c * kChunkBytes + ks * 32), 0, 1024),
                                             smem_desc_sw128(q + uint32_t(c * (N * 128) + ks * 32), 0, 1024), idesc_s, pair + c + ks > 0 ? 1u : 0u);
                                }
                            }
                        }
                        if (pair == p.pairs - 1 && !has_tail) {
                            umma_commit(bar(kBarS));
                        }
                    }
                    __syncwarp();
                    if (++slot_s == p.ring) {
                        slot_s = 0;
                        ++round_s;
                    }
                }
                if (has_tail && ok) {
                    ok = wait(kBarTail, tile_no);
                    tc_fence_after();
                    if (ok && elect_one()) {
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks) {
                            umma_f16(tmem, smem_desc_sw128(tail_u32 + uint32_t(ks * 32), 0, 1024),
                                     smem_desc_sw128(q_u32 + uint32_t(2 * p.pairs * (N * 128) + ks * 32), 0, 1024), idesc_s, 1u);
                        }
                        umma_commit(bar(kBarS));
                    }
                    __syncwarp();
                }
                ok = ok && wait(kBarP, tile_no);
                tc_fence_after();
                for (int pair = 0; pair < p.pairs && ok; ++pair) {
                    const uint32_t v = ring_u32 + uint32_t(slot_o) * kPairBytes;
                    if (elect_one()) {
#pragma unroll
                        for (int kk = 0; kk < kTile / 16; ++kk) {
                            umma_f16(tmem + uint32_t(kColO + pair * N), smem_desc_sw128(v + uint32_t(kk * 2048), kChunkBytes, 1024),
                                     smem_desc_sw128(p_u32 + uint32_t((kk >> 2) * (N * 128) + (kk & 3) * 32), 0, 1024), idesc_o,
                                     t > f.t0 || kk > 0 ? 1u : 0u);
                        }
                        umma_commit(bar(kBarFree + slot_o));
                        if (pair == p.pairs - 1) {
                            umma_commit(bar(kBarO));
                        }
                    }
                    __syncwarp();
                    slot_o = slot_o + 1 == p.ring ? 0 : slot_o + 1;
                }
            }
        }
        if (!ok && lane == 0) {
            give_up();
        }
    } else {
        const uint32_t lane_base = tmem + (uint32_t(warp * 32) << 16);
        const int col = lane % N; // the column whose maximum and sum this lane keeps
        auto unit_at = [&](const SeqGeom &g, const Fragment &f, int &h0, int &heads, int &first) {
            const int block = f.unit / p.n_groups, group = f.unit - block * p.n_groups;
            h0 = group * p.group;
            heads = min(p.group, p.nh - h0);
            first = block * p.block; // query of the chunk
        };
        // kLanes neighbouring threads per row; a row's pieces in two batches, every load of a batch in flight
        constexpr int kLanes = 128 / N, kBatch = (2 * kMaxPairs + 1) * 8 / kLanes / 2 + 1;
        auto load_q = [&](const SeqGeom &g, const Fragment &f) {
            int h0, heads, first;
            unit_at(g, f, h0, heads, first);
            const int c = tid / kLanes, e0 = tid % kLanes, t = c / p.group, h = c - t * p.group, pieces = p.chunks * 8;
            const bool holds = t < p.block && h < heads && first + t < g.q_len;
            const uint4 *src = reinterpret_cast<const uint4 *>(static_cast<const unsigned char *>(p.q) +
                                                               ((long long)(g.q_start + first + t) * p.nh + h0 + h) * p.dim * 2);
            const int n = holds ? p.dim / 8 : 0;
            for (int b = e0; b < pieces; b += kBatch * kLanes) {
                uint4 vals[kBatch];
#pragma unroll
                for (int i = 0; i < kBatch; ++i) {
                    const int e = b + i * kLanes;
                    vals[i] = e < n ? src[e] : make_uint4(0u, 0u, 0u, 0u);
                }
#pragma unroll
                for (int i = 0; i < kBatch; ++i) {
                    const int e = b + i * kLanes;
                    if (e < pieces) {
                        const uint32_t dst = q_u32 + uint32_t((e >> 3) * (N * 128) + c * 128 + (((e & 7) ^ (c & 7)) << 4));
                        asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};\n" ::"r"(dst), "r"(vals[i].x), "r"(vals[i].y), "r"(vals[i].z), "r"(vals[i].w)
                                     : "memory");
                    }
                }
            }
            fence_proxy_async_smem();
            mbar_arrive(bar(kBarQ));
        };
        bool dead = false;
        int tile_no = 0;
        Fragment f;
        int pos = piece_begin;
        bool any_left = locate(p, walker, pos, piece_end, f);
        if (any_left) {
            load_q(walker.g, f);
        }
        while (any_left) {
            const SeqGeom g = walker.g;
            int h0, heads, first;
            unit_at(g, f, h0, heads, first);
            float m_used = -INFINITY, l[N];
#pragma unroll
            for (int c = 0; c < N; ++c) {
                l[c] = 0.f;
            }
            for (int t = f.t0; t < f.t1; ++t, ++tile_no) {
                dead = dead || !wait(kBarS, tile_no);
                float x[N], top[N];
                if (!dead) {
                    tc_fence_after();
                    load_columns<N>(lane_base, x);
                    const int key = t * kTile + tid;
#pragma unroll
                    for (int c = 0; c < N; ++c) {
                        x[c] *= p.scale_log2;
                    }
                    if (t * kTile + kTile - 1 > g.off + first) { // (the same for every thread)
                        int limit = min(g.off + first, g.kv_len - 1), left = p.group;
#pragma unroll
                        for (int c = 0; c < N; ++c) {
                            if (left == 0) { // the next query's columns
                                limit = min(limit + 1, g.kv_len - 1);
                                left = p.group;
                            }
                            --left;
                            x[c] = key <= limit ? x[c] : -INFINITY;
                        }
                    }
#pragma unroll
                    for (int c = 0; c < N; ++c) {
                        top[c] = x[c];
                    }
                    const float mine = reduce_columns<N>(top, lane, [](float a, float b) { return fmaxf(a, b); });
                    if (lane < N) {
                        s_max[tile_no & 1][warp][lane] = mine;
                    }
                }
                asm volatile("bar.sync 1, 128;\n" ::: "memory");
                if (dead) {
                    continue;
                }
                const float (*tops)[N] = s_max[tile_no & 1];
                const float mx = fmaxf(fmaxf(tops[0][col], tops[1][col]), fmaxf(tops[2][col], tops[3][col]));
                float alpha = 1.f;
                const bool grow = mx > m_used + kRescaleThreshold;
                if (grow) {
                    alpha = fast_exp2(m_used - mx); // 0 on the fragment's first visible tile
                    m_used = mx;
                }
                const bool any_grow = __any_sync(0xffffffffu, grow); // (the same in all warps)
                const float ref = m_used == -INFINITY ? 0.f : m_used;
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    x[c] = fast_exp2(x[c] - __shfl_sync(0xffffffffu, ref, c));
                }
                if (any_grow) {
#pragma unroll
                    for (int c = 0; c < N; ++c) {
                        l[c] *= __shfl_sync(0xffffffffu, alpha, c);
                    }
                }
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    l[c] += x[c];
                }
                if (tile_no > 0) {
                    dead = !wait(kBarO, tile_no - 1);
                    if (dead) {
                        continue;
                    }
                    tc_fence_after();
                    if (any_grow && t > f.t0) {
                        for (int pair = 0; pair < p.pairs; ++pair) {
                            float o[N];
                            load_columns<N>(lane_base + uint32_t(kColO + pair * N), o);
#pragma unroll
                            for (int c = 0; c < N; ++c) {
                                o[c] *= __shfl_sync(0xffffffffu, alpha, c);
                            }
                            store_columns<N>(lane_base + uint32_t(kColO + pair * N), o);
                        }
                        tmem_wait_st();
                    }
                }
                // weights: row = column of the product, 128 keys in two halves of 128 bytes
                const uint32_t at = p_u32 + uint32_t((tid >> 6) * (N * 128)) + uint32_t(tid & 7) * 2, piece16 = uint32_t(tid & 63) >> 3;
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    const uint16_t w = kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(x[c])) : __half_as_ushort(__float2half_rn(x[c]));
                    asm volatile("st.shared.u16 [%0], %1;\n" ::"r"(at + uint32_t(c * 128) + ((piece16 ^ uint32_t(c & 7)) << 4)), "h"(w) : "memory");
                }
                fence_proxy_async_smem();
                tc_fence_before();
                mbar_arrive(bar(kBarP));
            }
            // queries of the next unit: every score of this one has been read
            const Fragment cur = f;
            pos += f.t1 - f.t0;
            any_left = locate(p, walker, pos, piece_end, f);
            if (any_left && !dead) {
                load_q(walker.g, f);
            }
            // ---- results ----
            const float sum_w = reduce_columns<N>(l, lane, [](float a, float b) { return a + b; });
            dead = dead || !wait(kBarO, tile_no - 1);
            tc_fence_after();
            asm volatile("bar.sync 1, 128;\n" ::: "memory"); // (maxima of the last tile have been read)
            if (lane < N) {
                s_max[0][warp][lane] = sum_w;
            }
            asm volatile("bar.sync 1, 128;\n" ::: "memory");
            const float sum = (s_max[0][0][col] + s_max[0][1][col]) + (s_max[0][2][col] + s_max[0][3][col]);
            asm volatile("bar.sync 1, 128;\n" ::: "memory");
            if (dead) {
                continue;
            }
            if (cur.t0 == 0 && cur.t1 == g.tiles) {
                const int t_col = col / p.group, h_col = col - t_col * p.group, row_col = g.q_start + first + t_col;
                const bool holds = t_col < p.block && h_col < heads && first + t_col < g.q_len;
                const unsigned columns = __ballot_sync(0xffffffffu, holds);
                float factor = sum > 0.f ? 1.f / sum : 0.f;
                if (p.row_scale != nullptr && holds) {
                    factor *= p.row_scale[(long long)row_col * p.nh + h0 + h_col];
                }
                float factors[N];
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    factors[c] = __shfl_sync(0xffffffffu, factor, c);
                }
                uint16_t *out = static_cast<uint16_t *>(p.out) + (long long)(g.q_start + first) * p.out_stride + (long long)h0 * p.rank + tid;
                const long long next_query = p.out_stride - (long long)(p.group - 1) * p.rank;
                for (int pair = 0; pair < p.pairs; ++pair, out += 128) {
                    float o[N];
                    load_columns<N>(lane_base + uint32_t(kColO + pair * N), o);
                    uint16_t *at = out;
                    int left = p.group;
#pragma unroll
                    for (int c = 0; c < N; ++c) {
                        if ((columns >> c & 1u) != 0 && pair * 128 + tid < p.rank) {
                            const float v = o[c] * factors[c];
                            *at = kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(v)) : __half_as_ushort(__float2half_rn(v));
                        }
                        --left;
                        at += left != 0 ? (long long)p.rank : next_query;
                        left = left != 0 ? left : p.group;
                    }
                }
            } else {
                float *part = p.partials + (long long)(int(blockIdx.x) * 2 + (cur.t0 == 0 ? 1 : 0)) * partial_floats(N, p.pairs);
                for (int pair = 0; pair < p.pairs; ++pair) {
                    float o[N];
                    load_columns<N>(lane_base + uint32_t(kColO + pair * N), o);
#pragma unroll
                    for (int c = 0; c < N; ++c) {
                        part[c * (p.pairs * 128) + pair * 128 + tid] = o[c];
                    }
                }
                if (tid < N) {
                    part[N * p.pairs * 128 + tid] = m_used;
                    part[N * p.pairs * 128 + N + tid] = sum;
                }
            }
            tc_fence_before(); // the reads of O come before the next unit's weights arrive
        }
        if (dead && lane == 0) {
            give_up();
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == kIssuer) {
        tc_fence_after();
        tmem_dealloc(tmem, kCols);
    }
}

// Results of units that were cut: one warp per (row, head).
template <bool kBf16, int N>
__global__ void __launch_bounds__(256) latent_merge_kernel(Params p, int n_pieces) {
    __shared__ int s_scan[34];
    grid_dependency_wait();
    grid_launch_dependents();
    const int row = int(blockIdx.x), lane = int(threadIdx.x) & 31, h = int(blockIdx.y) * 8 + (int(threadIdx.x) >> 5);
    // the row's sequence, and where that begins on the line
    int a = row;
    if (p.q_starts != nullptr) {
        int lo = 0, hi = p.n_seqs - 1;
        const int at = p.q_starts[0] + row;
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (p.q_starts[mid] <= at) {
                lo = mid;
            } else {
                hi = mid - 1;
            }
        }
        a = lo;
    }
    int seq_begin = 0;
    {
        int mine = 0;
        for (int i = int(threadIdx.x); i < a; i += int(blockDim.x)) {
            mine += seq_geom(p, i).length;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            mine += __shfl_xor_sync(0xffffffffu, mine, o);
        }
        if (lane == 0) {
            s_scan[threadIdx.x >> 5] = mine;
        }
        __syncthreads();
        for (int w = 0; w < 8; ++w) {
            seq_begin += s_scan[w];
        }
        __syncthreads();
    }
    int dummy_seq, dummy_begin;
    const int line = scan_line<false>(p, 0, 0, s_scan, dummy_seq, dummy_begin), piece = piece_length(line, n_pieces);
    if (h >= p.nh) {
        return;
    }
    const SeqGeom g = seq_geom(p, a);
    const int t = p.q_starts != nullptr ? p.q_starts[0] + row - g.q_start : 0;
    if (t >= g.q_len) {
        return;
    }
    const int group = h / p.group, block = t / p.block, col = (t - block * p.block) * p.group + h - group * p.group;
    const int begin = seq_begin + (block * p.n_groups + group) * (g.tiles + kUnitCost);
    const int first = begin / piece, last = (begin + g.tiles - 1) / piece;
    if (first == last) {
        return;
    }
    const int width = p.pairs * 128;
    auto part = [&](int s) { return p.partials + (long long)(s * 2 + (s * piece <= begin ? 1 : 0)) * partial_floats(N, p.pairs); };
    float m = -INFINITY;
    for (int s = first; s <= last; ++s) {
        m = fmaxf(m, part(s)[N * width + col]);
    }
    float sum = 0.f;
    float4 acc[kMaxPairs];
#pragma unroll
    for (int i = 0; i < kMaxPairs; ++i) {
        acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int s = first; s <= last; ++s) {
        const float *from = part(s);
        const float ms = from[N * width + col], w = ms == -INFINITY ? 0.f : fast_exp2(ms - m);
        sum = fmaf(from[N * width + N + col], w, sum);
#pragma unroll
        for (int i = 0; i < kMaxPairs; ++i) {
            if (i < p.pairs) {
                const float4 o = *reinterpret_cast<const float4 *>(from + col * width + i * 128 + lane * 4);
                acc[i].x = fmaf(o.x, w, acc[i].x);
                acc[i].y = fmaf(o.y, w, acc[i].y);
                acc[i].z = fmaf(o.z, w, acc[i].z);
                acc[i].w = fmaf(o.w, w, acc[i].w);
            }
        }
    }
    const long long out_row = g.q_start + t;
    float factor = sum > 0.f ? 1.f / sum : 0.f;
    if (p.row_scale != nullptr) {
        factor *= p.row_scale[out_row * p.nh + h];
    }
#pragma unroll
    for (int i = 0; i < kMaxPairs; ++i) {
        const int dim = i * 128 + lane * 4;
        if (i < p.pairs && dim < p.rank) { // (rank: whole 16-byte pieces)
            uint2 w = make_uint2(pack2<kBf16>(acc[i].x * factor, acc[i].y * factor), pack2<kBf16>(acc[i].z * factor, acc[i].w * factor));
            *reinterpret_cast<uint2 *>(static_cast<unsigned char *>(p.out) + (out_row * p.out_stride + (long long)h * p.rank + dim) * 2) = w;
        }
    }
}

int sm_count() {
    static int counts[64] = {};
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    int &n = counts[dev & 63];
    if (n == 0) {
        LLAISYS_CUDA_CHECK(cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev));
        n = n > 0 ? n : 1;
    }
    return n;
}

size_t fixed_smem(const Params &p, int n) {
    return 1024 + size_t(p.chunks > 2 * p.pairs ? kChunkBytes : 0) + size_t(p.chunks) * n * 128 + size_t(2) * n * 128;
}

template <bool kBf16, int N>
void launch(cudaStream_t s, const CUtensorMap &tmap, Params p, int rows) {
    const size_t fixed = fixed_smem(p, N);
    p.ring = int(std::min<size_t>(kMaxRing, (size_t(kSmemLimit) - 4096 - fixed) / kPairBytes)); // (4 KiB: static shared memory)
    const size_t smem = fixed + size_t(p.ring) * kPairBytes;
    static std::once_flag once[64];
    int dev = 0;
    LLAISYS_CUDA_CHECK(cudaGetDevice(&dev));
    std::call_once(once[dev & 63], [] {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(attention_latent_kernel<kBf16, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - 4096));
    });
    const int grid = sm_count();
    launch_programmatic_smem(attention_latent_kernel<kBf16, N>, dim3(unsigned(grid)), kThreads, smem, s, tmap, p);
    launch_programmatic(latent_merge_kernel<kBf16, N>, dim3(unsigned(rows), unsigned((p.nh + 7) / 8)), 256u, s, p, grid);
}

} // namespace

bool attention_latent_covers(llaisysDataType_t dtype, size_t nh, size_t rank, size_t dim) {
    return (dtype == LLAISYS_DTYPE_BF16 || dtype == LLAISYS_DTYPE_F16) && nh != 0 && rank != 0 && rank <= 128 * kMaxPairs && rank % 8 == 0 &&
           dim >= rank && dim % 8 == 0 && (dim + 63) / 64 <= 2 * ((rank + 127) / 128) + 1;
}

size_t attention_latent_scratch(size_t rank) { return size_t(2) * sm_count() * partial_floats(32, int((rank + 127) / 128)); }

int attention_latent_tc(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                        const AttnOut &out, const AttnScratch &scratch) {
    if (!attention_latent_covers(dtype, size_t(batch.nh), size_t(kv.vDim()), size_t(kv.d)) || kv.v_base != kv.k_base || kv.nkvh != 1 ||
        kv.page_size != kPage || kv.block_table == nullptr || kv.token_stride != kv.d || kv.page_stride != int64_t(kPage) * kv.d ||
        batch.kv_lens == nullptr || batch.n_seqs <= 0 || batch.window > 0 || batch.fade_a != nullptr || out.out == nullptr || out.part != nullptr ||
        out.peers != nullptr || scratch.error_flag == nullptr || scratch.partials == nullptr ||
        scratch.partials_floats < attention_latent_scratch(size_t(kv.vDim())) || !aligned16(q) || !aligned16(out.out) || out.row_stride % 4 != 0 ||
        !aligned16(kv.k_base) || (batch.q_starts == nullptr && batch.const_q_len != 1)) {
        return -1;
    }
    const bool bf16 = dtype == LLAISYS_DTYPE_BF16;
    Params p{};
    p.block_table = kv.block_table;
    p.table_stride = kv.table_stride;
    p.num_pages = kv.num_pages;
    p.seq_ids = batch.seq_ids;
    p.kv_lens = batch.kv_lens;
    p.q_starts = batch.q_starts;
    p.n_seqs = batch.n_seqs;
    p.nh = batch.nh;
    const bool narrow = batch.nh <= 16 && batch.max_q_len <= 1; // (16 columns are enough)
    const int n = narrow ? 16 : 32;
    p.n_groups = (batch.nh + n - 1) / n;
    p.group = (batch.nh + p.n_groups - 1) / p.n_groups;
    p.block = n / p.group;
    p.dim = kv.d;
    p.rank = kv.vDim();
    p.chunks = (p.dim + 63) / 64;
    p.pairs = (p.rank + 127) / 128;
    p.q = q;
    p.out = out.out;
    p.out_stride = out.row_stride != 0 ? out.row_stride : (long long)batch.nh * p.rank;
    p.row_scale = out.row_scale;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.partials = scratch.partials;
    p.error_flag = scratch.error_flag;
    CUtensorMap tmap;
    if (!matrix_map(&tmap, kv.k_base, uint64_t(kv.num_pages) * kPage, uint64_t(kv.d), kPage, bf16)) {
        return -1;
    }
    auto s = static_cast<cudaStream_t>(stream);
    if (narrow) {
        bf16 ? launch<true, 16>(s, tmap, p, batch.total_q) : launch<false, 16>(s, tmap, p, batch.total_q);
    } else {
        bf16 ? launch<true, 32>(s, tmap, p, batch.total_q) : launch<false, 32>(s, tmap, p, batch.total_q);
    }
    check_launch("attention_latent_tc");
    return 0;
}

} // namespace llaisys::kernels
