// K1 paged append and K5 paged gather: bit-exact row movement between [rows, nkvh, d] tensors and the page
// pool, 16 bytes per thread.
//
// Work decomposition: one thread per 16-byte piece of one (row, K-or-V, kv-head) head-row. A head-row is
// d*elem_size bytes (256 B for bf16, d 128) and is contiguous on both sides, so a quarter-warp moves a full
// head-row with coalesced 128-bit loads and stores. The slot lookup (two int32 loads per row, then one table
// entry) hits in L1 for the other threads of the row.
//
// Roofline: HBM. Algorithmic bytes per row = 2 * (2 * nkvh * d * elem_size) (read the new K and V row, write
// them) + 8 (sequence id and position) + 4 (table entry).
#include "launch_utils.cuh"

#include <algorithm>

namespace llaisys::kernels {

namespace {

struct CopyGeom {
    int64_t page_stride_b, head_stride_b, token_stride_b; // in bytes
    int32_t vecs_per_head_row;                            // d * elem_size / 16
    int32_t nkvh, page_size, num_pages, table_stride;
};

// Resolves (table row, position) to a physical page and slot; returns false (and flags) if out of range.
__device__ __forceinline__ bool resolve_slot(const int32_t *__restrict__ table, const CopyGeom &g, int32_t seq_row,
                                             int32_t pos, int32_t max_blocks, int32_t *error_flag, int32_t &page,
                                             int32_t &slot) {
    const int32_t blk = pos / g.page_size;
    if (pos < 0 || blk >= max_blocks || seq_row < 0) {
        atomicOr(error_flag, kErrBadPosition);
        return false;
    }
    page = table ? table[int64_t(seq_row) * g.table_stride + blk] : blk;
    slot = pos - blk * g.page_size;
    if (page < 0 || page >= g.num_pages) {
        atomicOr(error_flag, kErrBadPage);
        return false;
    }
    return true;
}

// One warp per new row, kRows rows per warp and pass. A row is moved by lane l as 16-byte piece l (+ 32, ...) of the K
// row and of the V row: with 2 kv-heads of 128 16-bit dims a row of K is 512 B, one coalesced warp-wide read, written as
// two 256 B head-rows. What bounds the kernel is latency, not bytes: a row's slot takes three dependent loads (sequence
// id and position, then the table entry), and with one row per warp in flight that chain -- not the 2 KiB moved -- set
// the pace (63 % of the copy rate). So a pass first issues the index loads AND the data loads of all its rows, which do
// not depend on the slots, then resolves the slots, then stores: kRows KiB of reads in flight per warp while the index
// chain runs underneath.
template <int kRows, int kIters>
__global__ void __launch_bounds__(256)
    paged_append_kernel(uint4 *__restrict__ k_pool, uint4 *__restrict__ v_pool, const uint4 *__restrict__ k_rows,
                        const uint4 *__restrict__ v_rows, const int32_t *__restrict__ table,
                        const int32_t *__restrict__ seq_ids, const int32_t *__restrict__ positions, CopyGeom g,
                        int32_t n_rows, int32_t max_blocks, int32_t *error_flag, const uint4 *__restrict__ side_src,
                        uint4 *__restrict__ side_dst, int32_t side_vecs) {
    // Under a programmatic launch this grid may start early: let the next kernel do the same, then wait for the
    // previous one (it may still be reading the pages this grid writes).
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    const int32_t vecs_per_row = g.vecs_per_head_row * g.nkvh; // per K (or V) row; at most 32 * kIters
    const int lane = threadIdx.x & 31;
    const int32_t warps = int32_t((gridDim.x * blockDim.x) >> 5);
    const int32_t warp_id = int32_t((blockIdx.x * blockDim.x + threadIdx.x) >> 5);
    for (int32_t row0 = warp_id; row0 < n_rows; row0 += kRows * warps) {
        int32_t seq[kRows], pos[kRows];
        uint4 kd[kRows][kIters], vd[kRows][kIters];
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            const int32_t row = row0 + u * warps;
            seq[u] = row < n_rows ? seq_ids[row] : -1;
            pos[u] = row < n_rows ? positions[row] : 0;
        }
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            const int32_t row = row0 + u * warps;
#pragma unroll
            for (int it = 0; it < kIters; ++it) {
                const int32_t in_row = lane + 32 * it;
                if (row < n_rows && in_row < vecs_per_row) {
                    const int64_t src = int64_t(row) * vecs_per_row + in_row;
                    kd[u][it] = __ldcs(k_rows + src); // read once: do not keep in cache
                    vd[u][it] = __ldcs(v_rows + src);
                }
            }
        }
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            const int32_t row = row0 + u * warps;
            int32_t page, slot;
            if (row >= n_rows || !resolve_slot(table, g, seq[u], pos[u], max_blocks, error_flag, page, slot)) {
                continue;
            }
            const int64_t slot_vec = (int64_t(page) * g.page_stride_b + int64_t(slot) * g.token_stride_b) / 16;
#pragma unroll
            for (int it = 0; it < kIters; ++it) {
                const int32_t in_row = lane + 32 * it;
                if (in_row < vecs_per_row) {
                    const int32_t kvh = in_row / g.vecs_per_head_row;
                    const int32_t vec = in_row - kvh * g.vecs_per_head_row;
                    const int64_t dst = slot_vec + int64_t(kvh) * (g.head_stride_b / 16) + vec;
                    k_pool[dst] = kd[u][it];
                    v_pool[dst] = vd[u][it];
                }
            }
        }
    }
    // An unrelated plain copy riding on this launch (the host step's q rows, read from mapped host memory): four
    // vectors per thread in flight.
    const int32_t threads = int32_t(gridDim.x * blockDim.x), me = int32_t(blockIdx.x * blockDim.x + threadIdx.x);
    for (int32_t i = me; i < side_vecs; i += 4 * threads) {
        uint4 val[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if (i + u * threads < side_vecs) {
                val[u] = side_src[i + u * threads];
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if (i + u * threads < side_vecs) {
                side_dst[i + u * threads] = val[u];
            }
        }
    }
}

// Plain copies of up to three small blocks (multiples of 16 bytes) in one launch: the host step's index arrays and q
// rows, read from mapped host memory -- a kernel's loads start sooner than a copy-engine transfer is set up.
struct CopyList {
    const uint4 *src[3];
    uint4 *dst[3];
    int32_t vecs[3];
};
__global__ void small_copies_kernel(CopyList l) {
    // lets a kernel launched behind this one with programmatic stream serialisation begin at once (it waits for these
    // copies where it needs them); no effect on an ordinary successor
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int32_t threads = int32_t(gridDim.x * blockDim.x), me = int32_t(blockIdx.x * blockDim.x + threadIdx.x);
#pragma unroll
    for (int b = 0; b < 3; ++b) {
        for (int32_t i = me; i < l.vecs[b]; i += threads) {
            l.dst[b][i] = l.src[b][i];
        }
    }
}

__global__ void paged_gather_kernel(const uint4 *__restrict__ k_pool, const uint4 *__restrict__ v_pool,
                                    uint4 *__restrict__ k_out, uint4 *__restrict__ v_out,
                                    const int32_t *__restrict__ table, CopyGeom g, int32_t seq_row, int32_t n_tokens,
                                    int32_t max_blocks, int32_t *error_flag) {
    const int32_t vecs_per_row = g.vecs_per_head_row * g.nkvh;
    const int64_t total = int64_t(n_tokens) * 2 * vecs_per_row;
    const int64_t stride = int64_t(gridDim.x) * blockDim.x;
    for (int64_t i = int64_t(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
        const int32_t tok = int32_t(i / (2 * vecs_per_row));
        const int32_t r = int32_t(i - int64_t(tok) * 2 * vecs_per_row);
        const int32_t is_v = r / vecs_per_row;
        const int32_t in_row = r - is_v * vecs_per_row;
        const int32_t kvh = in_row / g.vecs_per_head_row;
        const int32_t vec = in_row - kvh * g.vecs_per_head_row;
        int32_t page, slot;
        if (!resolve_slot(table, g, seq_row, tok, max_blocks, error_flag, page, slot)) {
            continue;
        }
        const int64_t off_b = int64_t(page) * g.page_stride_b + int64_t(kvh) * g.head_stride_b +
                              int64_t(slot) * g.token_stride_b;
        const uint4 val = (is_v ? v_pool : k_pool)[off_b / 16 + vec];
        (is_v ? v_out : k_out)[int64_t(tok) * vecs_per_row + in_row] = val;
    }
}

CopyGeom make_geom(const KVView &kv, size_t elem_size) {
    CHECK_ARGUMENT((size_t(kv.d) * elem_size) % 16 == 0, "paged copy: head rows must be a multiple of 16 bytes");
    CHECK_ARGUMENT((size_t(kv.token_stride) * elem_size) % 16 == 0 && (size_t(kv.head_stride) * elem_size) % 16 == 0 &&
                       (size_t(kv.page_stride) * elem_size) % 16 == 0,
                   "paged copy: strides must be multiples of 16 bytes");
    CopyGeom g;
    g.page_stride_b = kv.page_stride * int64_t(elem_size);
    g.head_stride_b = kv.head_stride * int64_t(elem_size);
    g.token_stride_b = kv.token_stride * int64_t(elem_size);
    g.vecs_per_head_row = int32_t(size_t(kv.d) * elem_size / 16);
    g.nkvh = kv.nkvh;
    g.page_size = kv.page_size;
    g.num_pages = kv.num_pages;
    g.table_stride = kv.table_stride;
    return g;
}

int grid_for(int64_t threads, int block) {
    const int64_t want = (threads + block - 1) / block;
    const int64_t cap = 148 * 8;
    return int(want < cap ? (want ? want : 1) : cap);
}

// K1b: the step just before attention, fused. Input is the packed projection output qkv [rows, (nh + 2 nkvh) * d] (plus
// an optional bias row); q and k heads get the half-split rotary embedding (angle = pos / theta^(2j/d) in f32, as the
// rope operator), q goes to a contiguous [rows, nh, d] tensor, k and v go straight into their page slots. One thread
// handles VEC elements of the lower half of a head row and the matching VEC of the upper half (VEC = 16 bytes of T, or
// 1 when d is not a multiple of 2 VEC): f32 arithmetic, one rounding.
template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) Pack {
    T v[VEC];
};

template <typename T, int VEC, bool kPerHead>
__global__ void paged_rope_append_kernel(unsigned char *__restrict__ k_pool, unsigned char *__restrict__ v_pool,
                                         T *__restrict__ q_out, const T *__restrict__ qkv, const T *__restrict__ bias,
                                         const int32_t *__restrict__ table, const int32_t *__restrict__ seq_ids,
                                         const int32_t *__restrict__ positions, CopyGeom g, int32_t n_rows, int32_t nh,
                                         int32_t d, float theta, int32_t max_blocks, int32_t *error_flag) {
    using P = Pack<T, VEC>;
    // Under a programmatic launch: let the next kernel (the decode attention) start its set-up, then wait for the
    // projection that produced qkv.
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    // theta^(2j/d) for the d/2 pair indices, once per CTA instead of one powf per element (before the wait: it depends
    // on nothing the previous kernel writes)
    extern __shared__ float s_divisor[];
    const int32_t half = d / 2;
    for (int32_t j = threadIdx.x; j < half; j += blockDim.x) {
        s_divisor[j] = powf(theta, 2.f * float(j) / float(d));
    }
    __syncthreads();
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    // A thread owns VEC pair indices of one row and every head_groups-th head: the sines and cosines depend on
    // (position, pair index) only, so they are computed once and reused for the thread's heads. Large calls (prefill)
    // use few groups -- less transcendental work per byte; small ones (a decode step) one group per head -- the
    // shortest dependent chain per thread.
    const int32_t vec_per_head = half / VEC;
    const int32_t heads = nh + 2 * g.nkvh;
    const int32_t head_groups = kPerHead ? heads : 4; // kPerHead: one head per thread (small calls)
    const int64_t total = int64_t(n_rows) * head_groups * vec_per_head;
    const int64_t stride = int64_t(gridDim.x) * blockDim.x;
    const int64_t row_elems = int64_t(heads) * d;
    for (int64_t i = int64_t(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += stride) {
        const int32_t row = int32_t(i / (head_groups * vec_per_head));
        const int32_t r = int32_t(i - int64_t(row) * head_groups * vec_per_head);
        const int32_t first_head = r / vec_per_head;
        const int32_t j0 = (r - first_head * vec_per_head) * VEC;
        const int32_t pos = positions[row];
        float sn[VEC], cs[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            sincosf(float(pos) / s_divisor[j0 + e], &sn[e], &cs[e]);
        }
        int32_t page = 0, slot = 0;
        // The slot lookup (three dependent loads) is needed only by threads that reach a K or V head: a one-head thread
        // of a small call does it on demand; a many-head thread of a large call starts it up front, under its other loads.
        bool resolved = false, slot_ok = false;
        if (head_groups < heads) {
            slot_ok = resolve_slot(table, g, seq_ids[row], pos, max_blocks, error_flag, page, slot);
            resolved = true;
        }
        for (int32_t head = first_head; head < heads; head += head_groups) {
            const int64_t in_off = int64_t(row) * row_elems + int64_t(head) * d + j0;
            P lo = *reinterpret_cast<const P *>(qkv + in_off);
            P hi = *reinterpret_cast<const P *>(qkv + in_off + half);
            float a[VEC], b[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                a[e] = to_f32(lo.v[e]);
                b[e] = to_f32(hi.v[e]);
            }
            if (bias != nullptr) {
                const P blo = *reinterpret_cast<const P *>(bias + int64_t(head) * d + j0);
                const P bhi = *reinterpret_cast<const P *>(bias + int64_t(head) * d + j0 + half);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    a[e] += to_f32(blo.v[e]);
                    b[e] += to_f32(bhi.v[e]);
                }
            }
            const bool is_v = head >= nh + g.nkvh;
            if (!is_v) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    const float x = a[e], y = b[e];
                    a[e] = x * cs[e] - y * sn[e];
                    b[e] = y * cs[e] + x * sn[e];
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                lo.v[e] = from_f32<T>(a[e]);
                hi.v[e] = from_f32<T>(b[e]);
            }
            if (head < nh) {
                T *dst = q_out + (int64_t(row) * nh + head) * d + j0;
                *reinterpret_cast<P *>(dst) = lo;
                *reinterpret_cast<P *>(dst + half) = hi;
                continue;
            }
            if (!resolved) {
                slot_ok = resolve_slot(table, g, seq_ids[row], pos, max_blocks, error_flag, page, slot);
                resolved = true;
            }
            if (!slot_ok) {
                continue;
            }
            const int32_t kvh = is_v ? head - nh - g.nkvh : head - nh;
            const int64_t off_b = int64_t(page) * g.page_stride_b + int64_t(kvh) * g.head_stride_b +
                                  int64_t(slot) * g.token_stride_b + int64_t(j0) * int64_t(sizeof(T));
            unsigned char *dst = (is_v ? v_pool : k_pool) + off_b;
            *reinterpret_cast<P *>(dst) = lo;
            *reinterpret_cast<P *>(dst + int64_t(half) * int64_t(sizeof(T))) = hi;
        }
    }
}

// Elements [at, at + VEC) of a q or k head row after norm (inv, w; w null: none), rotation and a factor: the partners across the rotated
// range are read from the row itself. VEC divides rot_dims / 2, so a piece lies in one half.
template <typename T, int VEC>
__device__ __forceinline__ Pack<T, VEC> norm_rotate(Pack<T, VEC> x, const T *src, int32_t at, float inv, const T *w,
                                                    const NormAppendArgs &a, int64_t row, float factor) {
    using P = Pack<T, VEC>;
    const int32_t half = a.rot_dims / 2;
    const bool turns = at < a.rot_dims;
    if (w == nullptr && !turns && factor == 1.f) {
        return x;
    }
    float f[VEC];
    auto normed = [&](const P &v, int32_t from, float (&y)[VEC]) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            y[e] = to_f32(v.v[e]);
        }
        if (w != nullptr) {
            const P ww = *reinterpret_cast<const P *>(w + from);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                y[e] = y[e] * inv * to_f32(ww.v[e]);
            }
        }
    };
    normed(x, at, f);
    if (turns) {
        const bool first = at < half;
        const int32_t other = first ? at + half : at - half, angle = first ? at : other;
        float g[VEC];
        normed(*reinterpret_cast<const P *>(src + other), other, g);
        const float2 *cs = reinterpret_cast<const float2 *>(a.rot_table) + row * half + angle;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float2 t = cs[e];
            f[e] = first ? f[e] * t.x - g[e] * t.y : f[e] * t.x + g[e] * t.y;
        }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        x.v[e] = from_f32<T>(f[e] * factor);
    }
    return x;
}

// K1c: one warp per (row, head) over the nh query, nkvh key and nkvh value heads of a projection row. Query and key heads
// are divided by their root mean square and weighted; the warp of a query head also turns that head's gate into the factor
// the attention kernel applies. f32 arithmetic, one rounding.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
    paged_norm_append_kernel(unsigned char *__restrict__ k_pool, unsigned char *__restrict__ v_pool, NormAppendArgs a,
                             const int32_t *__restrict__ table, CopyGeom g, int32_t d, int32_t dv, int64_t v_head_stride_b,
                             int64_t v_token_stride_b, int32_t max_blocks, int32_t *error_flag) {
    using P = Pack<T, VEC>;
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int32_t heads = a.nh + 2 * g.nkvh;
    const int64_t item = (int64_t(blockIdx.x) * blockDim.x + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (item >= int64_t(a.n_rows) * heads) {
        return;
    }
    const int64_t row = item / heads;
    const int32_t head = int32_t(item - row * heads);
    const bool is_q = head < a.nh, is_v = head >= a.nh + g.nkvh;
    const T *proj = static_cast<const T *>(a.proj) + row * a.row_stride;
    const int32_t kvh = is_v ? head - a.nh - g.nkvh : head - a.nh;
    const T *src = proj + (is_q ? a.q_at + int64_t(head) * d : (is_v ? a.v_at + int64_t(kvh) * dv : a.k_at + int64_t(kvh) * d));
    const int32_t n = is_v ? dv : d;
    const T *w = static_cast<const T *>(is_q ? a.q_norm : a.k_norm);
    float inv = 1.f;
    if (is_v) {
        w = nullptr;
    } else if (w != nullptr) {
        float ss = 0.f;
        for (int32_t i = lane * VEC; i < n; i += 32 * VEC) {
            const P x = *reinterpret_cast<const P *>(src + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                ss = fmaf(to_f32(x.v[e]), to_f32(x.v[e]), ss);
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            ss += __shfl_xor_sync(0xffffffffu, ss, o);
        }
        inv = rsqrtf(ss / float(n) + a.eps);
    }
    T *dst;
    if (is_q) {
        dst = static_cast<T *>(a.q_out) + (row * a.nh + head) * d;
        if (lane == 0 && a.row_scale != nullptr) {
            a.row_scale[row * a.nh + head] =
                a.gate_at < 0 ? a.gate_scale : a.gate_scale / (1.f + expf(-to_f32(proj[a.gate_at + head])));
        }
    } else {
        int32_t page, slot;
        if (!resolve_slot(table, g, a.seq_ids[row], a.positions[row], max_blocks, error_flag, page, slot)) {
            return;
        }
        const int64_t off = int64_t(page) * g.page_stride_b +
                            (is_v ? int64_t(kvh) * v_head_stride_b + int64_t(slot) * v_token_stride_b
                                  : int64_t(kvh) * g.head_stride_b + int64_t(slot) * g.token_stride_b);
        dst = reinterpret_cast<T *>((is_v ? v_pool : k_pool) + off);
    }
    for (int32_t i = lane * VEC; i < n; i += 32 * VEC) {
        P x = *reinterpret_cast<const P *>(src + i);
        if (!is_v) {
            x = norm_rotate<T, VEC>(x, src, i, inv, w, a, row, is_q && a.head_scale != nullptr ? a.head_scale[head] : 1.f);
        }
        *reinterpret_cast<P *>(dst + i) = x;
    }
}

// The same for head rows of at most 32 16-byte pieces: `lanes` (a power of two) neighbouring lanes share a head row, one
// piece each, which stays in registers between the norm and the store; a thread keeps kItems rows in flight.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
    paged_norm_append_pieces_kernel(unsigned char *__restrict__ k_pool, unsigned char *__restrict__ v_pool, NormAppendArgs a,
                                    const int32_t *__restrict__ table, CopyGeom g, int32_t d, int32_t dv, int64_t v_head_stride_b,
                                    int64_t v_token_stride_b, int32_t lanes, int32_t max_blocks, int32_t *error_flag) {
    using P = Pack<T, VEC>;
    constexpr int kItems = 2;
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int32_t heads = a.nh + 2 * g.nkvh, total = int32_t(a.n_rows) * heads;
    const int32_t per_block = int32_t(blockDim.x) / lanes;
    const int32_t item0 = int32_t(blockIdx.x) * per_block * kItems + int32_t(threadIdx.x) / lanes;
    const int32_t piece = int32_t(threadIdx.x) % lanes, at = piece * VEC;
    P x[kItems];
    int32_t row[kItems], head[kItems];
    bool holds[kItems];
    float ss[kItems];
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
        const int32_t item = item0 + u * per_block;
        row[u] = item / heads;
        head[u] = item - row[u] * heads;
        const bool is_q = head[u] < a.nh, is_v = head[u] >= a.nh + g.nkvh;
        holds[u] = item < total && at < (is_v ? dv : d);
        if (holds[u]) {
            const int64_t part = is_q ? a.q_at + int64_t(head[u]) * d
                                      : (is_v ? a.v_at + int64_t(head[u] - a.nh - g.nkvh) * dv : a.k_at + int64_t(head[u] - a.nh) * d);
            x[u] = *reinterpret_cast<const P *>(static_cast<const T *>(a.proj) + int64_t(row[u]) * a.row_stride + part + at);
        }
    }
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
        ss[u] = 0.f;
        if (holds[u]) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                ss[u] = fmaf(to_f32(x[u].v[e]), to_f32(x[u].v[e]), ss[u]);
            }
        }
        for (int o = lanes / 2; o > 0; o >>= 1) {
            ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o);
        }
    }
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
        if (!holds[u]) {
            continue;
        }
        const bool is_q = head[u] < a.nh, is_v = head[u] >= a.nh + g.nkvh;
        if (!is_v) {
            const T *src = static_cast<const T *>(a.proj) + int64_t(row[u]) * a.row_stride +
                           (is_q ? a.q_at + int64_t(head[u]) * d : a.k_at + int64_t(head[u] - a.nh) * d);
            x[u] = norm_rotate<T, VEC>(x[u], src, at, rsqrtf(ss[u] / float(d) + a.eps), static_cast<const T *>(is_q ? a.q_norm : a.k_norm), a,
                                       row[u], is_q && a.head_scale != nullptr ? a.head_scale[head[u]] : 1.f);
        }
        if (is_q) {
            *reinterpret_cast<P *>(static_cast<T *>(a.q_out) + (int64_t(row[u]) * a.nh + head[u]) * d + at) = x[u];
            if (piece == 0 && a.row_scale != nullptr) {
                const T *proj = static_cast<const T *>(a.proj) + int64_t(row[u]) * a.row_stride;
                a.row_scale[int64_t(row[u]) * a.nh + head[u]] =
                    a.gate_at < 0 ? a.gate_scale : a.gate_scale / (1.f + expf(-to_f32(proj[a.gate_at + head[u]])));
            }
            continue;
        }
        int32_t page, slot;
        if (!resolve_slot(table, g, a.seq_ids[row[u]], a.positions[row[u]], max_blocks, error_flag, page, slot)) {
            continue;
        }
        const int32_t kvh = is_v ? head[u] - a.nh - g.nkvh : head[u] - a.nh;
        const int64_t off = int64_t(page) * g.page_stride_b +
                            (is_v ? int64_t(kvh) * v_head_stride_b + int64_t(slot) * v_token_stride_b
                                  : int64_t(kvh) * g.head_stride_b + int64_t(slot) * g.token_stride_b);
        *reinterpret_cast<P *>((is_v ? v_pool : k_pool) + off + int64_t(at) * int64_t(sizeof(T))) = x[u];
    }
}

// The row form of NormAppendArgs: one CTA per row, because q and k are normed over all their heads at once. A row's pieces of
// VEC elements lie in q, then k, then v; the first PER_THREAD of a thread stay in registers between the sums and the stores.
template <typename T, int VEC, int PER_THREAD>
__global__ void paged_row_norm_append_kernel(unsigned char *__restrict__ k_pool, unsigned char *__restrict__ v_pool, NormAppendArgs a,
                                             const int32_t *__restrict__ table, CopyGeom g, int32_t d, int32_t dv,
                                             int64_t v_head_stride_b, int64_t v_token_stride_b, int32_t max_blocks, int32_t *error_flag) {
    using P = Pack<T, VEC>;
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int64_t row = blockIdx.x;
    const int32_t nq = a.nh * d / VEC, nk = g.nkvh * d / VEC, n = nq + nk + g.nkvh * dv / VEC;
    const T *proj = static_cast<const T *>(a.proj) + row * a.row_stride, *bias = static_cast<const T *>(a.bias);
    struct Piece {
        float v[VEC];
    };
    auto load = [&](int32_t i) {
        const int64_t at = i < nq ? a.q_at + int64_t(i) * VEC : (i < nq + nk ? a.k_at + int64_t(i - nq) * VEC : a.v_at + int64_t(i - nq - nk) * VEC);
        const P x = *reinterpret_cast<const P *>(proj + at);
        Piece f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            f.v[e] = to_f32(x.v[e]);
        }
        if (bias != nullptr) {
            const P b = *reinterpret_cast<const P *>(bias + at);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                f.v[e] += to_f32(b.v[e]);
            }
        }
        return f;
    };
    float sq = 0.f, sk = 0.f;
    auto square = [&](int32_t i, const Piece &f) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            s = fmaf(f.v[e], f.v[e], s);
        }
        sq += i < nq ? s : 0.f;
        sk += i >= nq && i < nq + nk ? s : 0.f;
    };
    Piece held[PER_THREAD];
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * int32_t(blockDim.x);
        if (i < n) {
            held[r] = load(i);
            square(i, held[r]);
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * int32_t(blockDim.x); i < nq + nk; i += int32_t(blockDim.x)) {
        square(i, load(i));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    __shared__ float part_q[32], part_k[32];
    if ((threadIdx.x & 31) == 0) {
        part_q[threadIdx.x >> 5] = sq;
        part_k[threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int i = 0; i < int(blockDim.x >> 5); ++i) { // every thread sums the few partials in the same order
        sq += part_q[i];
        sk += part_k[i];
    }
    const int32_t pos = a.positions[row];
    float inv_q = a.q_norm != nullptr ? rsqrtf(sq / float(a.nh * d) + a.eps) : 1.f;
    const float inv_k = a.k_norm != nullptr ? rsqrtf(sk / float(g.nkvh * d) + a.eps) : 1.f;
    if (a.temp_coef != 0.f) {
        inv_q *= fmaf(a.temp_coef, logf(floorf(__fdiv_rn(float(pos + 1), a.temp_every)) + 1.f), 1.f);
    }
    int32_t page = 0, slot = 0;
    const bool stores = resolve_slot(table, g, a.seq_ids[row], pos, max_blocks, error_flag, page, slot);
    auto store = [&](int32_t i, const Piece &f) {
        const bool is_q = i < nq, is_k = !is_q && i < nq + nk;
        const int32_t at = (is_q ? i : (is_k ? i - nq : i - nq - nk)) * VEC;
        const T *w = static_cast<const T *>(is_q ? a.q_norm : (is_k ? a.k_norm : nullptr));
        const float inv = is_q ? inv_q : (is_k ? inv_k : 1.f);
        P o;
        if (w != nullptr) {
            const P ww = *reinterpret_cast<const P *>(w + at);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                o.v[e] = from_f32<T>(f.v[e] * inv * to_f32(ww.v[e]));
            }
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                o.v[e] = from_f32<T>(f.v[e] * inv);
            }
        }
        if (is_q) {
            *reinterpret_cast<P *>(static_cast<T *>(a.q_out) + row * a.nh * d + at) = o;
            return;
        }
        if (!stores) {
            return;
        }
        const int32_t len = is_k ? d : dv, head = at / len;
        const int64_t off = int64_t(page) * g.page_stride_b + (at - head * len) * int64_t(sizeof(T)) +
                            (is_k ? int64_t(head) * g.head_stride_b + int64_t(slot) * g.token_stride_b
                                  : int64_t(head) * v_head_stride_b + int64_t(slot) * v_token_stride_b);
        *reinterpret_cast<P *>((is_k ? k_pool : v_pool) + off) = o;
    };
#pragma unroll
    for (int r = 0; r < PER_THREAD; ++r) {
        const int32_t i = int32_t(threadIdx.x) + r * int32_t(blockDim.x);
        if (i < n) {
            store(i, held[r]);
        }
    }
    for (int32_t i = int32_t(threadIdx.x) + PER_THREAD * int32_t(blockDim.x); i < n; i += int32_t(blockDim.x)) {
        store(i, load(i));
    }
}

// K1d: one CTA per row (see LatentAppendArgs). Pieces of VEC elements; the first kHeld of a thread of either latent stay in registers
// between the sums and the stores, and the token's slot is looked up under the sums.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_append_kernel(T *__restrict__ k_pool, LatentAppendArgs a, const int32_t *__restrict__ table,
                                                            CopyGeom g, int32_t max_blocks, int32_t *error_flag) {
    using P = Pack<T, VEC>;
    constexpr int kHeld = 2;
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int64_t row = blockIdx.x;
    const int32_t tid = int32_t(threadIdx.x), step = int32_t(blockDim.x), nq = a.q_rank / VEC, nk = a.rank / VEC;
    const T *proj = static_cast<const T *>(a.proj) + row * a.row_stride;
    const P *q = reinterpret_cast<const P *>(proj + a.q_at), *kv = reinterpret_cast<const P *>(proj + a.kv_at);
    const int32_t seq = a.seq_ids[row], pos = a.positions[row];
    P hq[kHeld], hk[kHeld];
    float sq = 0.f, sk = 0.f;
    auto square = [](const P &x, float &s) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            s = fmaf(to_f32(x.v[e]), to_f32(x.v[e]), s);
        }
    };
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
        if (tid + u * step < nq) {
            hq[u] = q[tid + u * step];
        }
        if (tid + u * step < nk) {
            hk[u] = kv[tid + u * step];
        }
    }
    const float2 *turn = reinterpret_cast<const float2 *>(a.rot_table) + row * (a.rot_dims / 2);
    float2 t0 = make_float2(1.f, 0.f);
    float u0 = 0.f, v0 = 0.f; // this thread's first pair to turn
    const T *z = proj + a.kv_at + a.rank;
    if (tid < a.rot_dims / 2) {
        t0 = turn[tid];
        u0 = to_f32(z[2 * tid]);
        v0 = to_f32(z[2 * tid + 1]);
    }
    int32_t page, slot;
    const bool stores = resolve_slot(table, g, seq, pos, max_blocks, error_flag, page, slot);
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
        if (tid + u * step < nq) {
            square(hq[u], sq);
        }
        if (tid + u * step < nk) {
            square(hk[u], sk);
        }
    }
    for (int32_t i = tid + kHeld * step; i < nq; i += step) {
        square(q[i], sq);
    }
    for (int32_t i = tid + kHeld * step; i < nk; i += step) {
        square(kv[i], sk);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    __shared__ float part_q[8], part_k[8];
    if ((tid & 31) == 0) {
        part_q[tid >> 5] = sq;
        part_k[tid >> 5] = sk;
    }
    if (a.row_scale != nullptr) {
        for (int32_t h = tid; h < a.nh; h += step) {
            a.row_scale[row * a.nh + h] = a.gate_at < 0 ? 1.f : 1.f / (1.f + expf(-to_f32(proj[a.gate_at + h])));
        }
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int32_t i = 0; i < step >> 5; ++i) { // every thread sums the few partials in the same order
        sq += part_q[i];
        sk += part_k[i];
    }
    const float inv_q = rsqrtf(sq / float(a.q_rank) + a.eps), inv_k = rsqrtf(sk / float(a.rank) + a.eps);
    auto normed = [](const P &x, const P &w, float inv) {
        P y;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            y.v[e] = from_f32<T>(to_f32(x.v[e]) * inv * to_f32(w.v[e]));
        }
        return y;
    };
    const P *q_norm = static_cast<const P *>(a.q_norm), *kv_norm = static_cast<const P *>(a.kv_norm);
    P *q_out = reinterpret_cast<P *>(static_cast<T *>(a.q_latent) + row * a.q_latent_stride);
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
        if (tid + u * step < nq) {
            q_out[tid + u * step] = normed(hq[u], q_norm[tid + u * step], inv_q);
        }
    }
    for (int32_t i = tid + kHeld * step; i < nq; i += step) {
        q_out[i] = normed(q[i], q_norm[i], inv_q);
    }
    if (!stores) {
        return;
    }
    T *dst = k_pool + int64_t(page) * (g.page_stride_b / int64_t(sizeof(T))) + int64_t(slot) * (g.token_stride_b / int64_t(sizeof(T)));
#pragma unroll
    for (int u = 0; u < kHeld; ++u) {
        if (tid + u * step < nk) {
            reinterpret_cast<P *>(dst)[tid + u * step] = normed(hk[u], kv_norm[tid + u * step], inv_k);
        }
    }
    for (int32_t i = tid + kHeld * step; i < nk; i += step) {
        reinterpret_cast<P *>(dst)[i] = normed(kv[i], kv_norm[i], inv_k);
    }
    for (int32_t i = tid; i < a.rot_dims / 2; i += step) {
        const float u = i == tid ? u0 : to_f32(z[2 * i]), v = i == tid ? v0 : to_f32(z[2 * i + 1]);
        const float2 t = i == tid ? t0 : turn[i];
        dst[a.rank + 2 * i] = from_f32<T>(u * t.x - v * t.y);
        dst[a.rank + 2 * i + 1] = from_f32<T>(v * t.x + u * t.y);
    }
}

template <typename T>
void launch_latent_append(cudaStream_t s, const KVView &kv, const LatentAppendArgs &a, int32_t max_blocks, int32_t *error_flag) {
    CopyGeom g{};
    g.page_stride_b = kv.page_stride * int64_t(sizeof(T));
    g.token_stride_b = kv.token_stride * int64_t(sizeof(T));
    g.nkvh = 1;
    g.page_size = kv.page_size;
    g.num_pages = kv.num_pages;
    g.table_stride = kv.table_stride;
    constexpr int kVec = 16 / int(sizeof(T));
    const bool wide = a.q_rank % kVec == 0 && a.rank % kVec == 0 && a.row_stride % kVec == 0 && a.q_at % kVec == 0 && a.kv_at % kVec == 0 &&
                      a.q_latent_stride % kVec == 0 && kv.token_stride % kVec == 0 && aligned16(a.proj) && aligned16(a.q_norm) &&
                      aligned16(a.kv_norm) && aligned16(a.q_latent) && aligned16(kv.k_base);
    const int32_t pieces = std::max(a.q_rank, a.rank) / (wide ? kVec : 1);
    auto kernel = wide ? latent_append_kernel<T, kVec> : latent_append_kernel<T, 1>;
    launch_programmatic(kernel, dim3(unsigned(a.n_rows)), pieces <= 128 ? 64u : (pieces <= 512 ? 128u : 256u), s, static_cast<T *>(kv.k_base), a,
                        kv.block_table, g, max_blocks, error_flag);
}

// One CTA per (page, sequence); P: the widest piece that divides a row.
template <typename P>
__global__ void __launch_bounds__(128) latent_gather_kernel(const unsigned char *__restrict__ pool, const int32_t *__restrict__ table, CopyGeom g,
                                                            P *__restrict__ out, int64_t out_pieces, int32_t row_pieces,
                                                            const int32_t *__restrict__ seq_ids, const int32_t *__restrict__ page_starts,
                                                            const int32_t *__restrict__ kv_lens, int32_t *error_flag) {
    asm volatile("griddepcontrol.wait;\n" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory");
    const int32_t i = int32_t(blockIdx.y), blk = int32_t(blockIdx.x), len = kv_lens[i], start = page_starts[i];
    if (start < 0 || blk * g.page_size >= len) {
        return;
    }
    int32_t page, slot;
    if (!resolve_slot(table, g, seq_ids[i], blk * g.page_size, g.table_stride, error_flag, page, slot)) {
        return;
    }
    const unsigned char *src = pool + int64_t(page) * g.page_stride_b;
    P *dst = out + int64_t(start + blk) * g.page_size * out_pieces;
    for (int32_t u = int32_t(threadIdx.x); u < g.page_size * row_pieces; u += 128) {
        const int32_t t = u / row_pieces, c = u - t * row_pieces;
        P v{};
        if (blk * g.page_size + t < len) {
            v = reinterpret_cast<const P *>(src + int64_t(t) * g.token_stride_b)[c];
        }
        dst[int64_t(t) * out_pieces + c] = v;
    }
}

template <typename T>
void launch_norm_append(cudaStream_t s, const KVView &kv, const NormAppendArgs &a, int32_t max_blocks, int32_t *error_flag) {
    CopyGeom g{};
    g.page_stride_b = kv.page_stride * int64_t(sizeof(T));
    g.head_stride_b = kv.head_stride * int64_t(sizeof(T));
    g.token_stride_b = kv.token_stride * int64_t(sizeof(T));
    g.nkvh = kv.nkvh;
    g.page_size = kv.page_size;
    g.num_pages = kv.num_pages;
    g.table_stride = kv.table_stride;
    constexpr int kVec = 4;
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const int32_t d = kv.d, dv = kv.vDim();
    cudaLaunchConfig_t cfg{};
    cfg.stream = s;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    if (a.row_norm != 0) {
        CHECK_ARGUMENT(a.rot_dims == 0 && a.gate_at < 0 && a.row_scale == nullptr && a.head_scale == nullptr && a.temp_every > 0.f,
                       "norm append: the row form takes neither a rotation, a gate nor factors per head");
        constexpr int kRow = 16 / int(sizeof(T));
        const bool pieces = d % kRow == 0 && dv % kRow == 0 && a.row_stride % kRow == 0 && a.q_at % kRow == 0 && a.k_at % kRow == 0 &&
                            a.v_at % kRow == 0 && aligned(a.proj) && aligned(a.bias) && aligned(a.q_norm) && aligned(a.k_norm) && aligned(a.q_out);
        const int64_t n = (int64_t(a.nh) * d + int64_t(kv.nkvh) * (d + dv)) / (pieces ? kRow : 1);
        CHECK_ARGUMENT(n < (int64_t(1) << 30), "norm append: row too long");
        const int64_t threads = (n + 2) / 3 + 31;
        cfg.gridDim = dim3(unsigned(a.n_rows));
        cfg.blockDim = dim3(unsigned(threads < 64 ? 64 : (threads > 512 ? 512 : threads / 32 * 32)));
        auto row_kernel = pieces ? paged_row_norm_append_kernel<T, kRow, 3> : paged_row_norm_append_kernel<T, 1, 3>;
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, row_kernel, static_cast<unsigned char *>(kv.k_base), static_cast<unsigned char *>(kv.v_base),
                                              NormAppendArgs(a), kv.block_table, g, d, dv, kv.vHeadStride() * int64_t(sizeof(T)),
                                              kv.vTokenStride() * int64_t(sizeof(T)), max_blocks, error_flag));
        return;
    }
    const bool wide = d % kVec == 0 && dv % kVec == 0 && a.row_stride % kVec == 0 && a.q_at % kVec == 0 && a.k_at % kVec == 0 &&
                      a.v_at % kVec == 0 && aligned(a.proj) && aligned(a.q_norm) && aligned(a.k_norm) && aligned(a.q_out) &&
                      a.rot_dims / 2 % kVec == 0;
    const int64_t warps = int64_t(a.n_rows) * (a.nh + 2 * kv.nkvh);
    cfg.gridDim = dim3(unsigned((warps + 7) / 8));
    cfg.blockDim = dim3(256);
    constexpr int kPiece = 16 / int(sizeof(T));
    const int32_t longest = d > dv ? d : dv;
    // (small calls are latency-bound: there the kernel with a warp per head row has the shorter chain)
    if (a.n_rows > 1024 && d % kPiece == 0 && dv % kPiece == 0 && longest <= 32 * kPiece && a.row_stride % kPiece == 0 && a.q_at % kPiece == 0 &&
        a.k_at % kPiece == 0 && a.v_at % kPiece == 0 && a.rot_dims / 2 % kPiece == 0 && wide && int64_t(a.n_rows) * (a.nh + 2 * kv.nkvh) < (int64_t(1) << 31)) {
        int32_t lanes = 1;
        while (lanes * kPiece < longest) {
            lanes *= 2;
        }
        const int64_t per_block = 2 * (256 / lanes);
        cfg.gridDim = dim3(unsigned((warps + per_block - 1) / per_block)); // (`warps` = head rows)
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, paged_norm_append_pieces_kernel<T, kPiece>, static_cast<unsigned char *>(kv.k_base),
                                              static_cast<unsigned char *>(kv.v_base), NormAppendArgs(a), kv.block_table, g, d, dv,
                                              kv.vHeadStride() * int64_t(sizeof(T)), kv.vTokenStride() * int64_t(sizeof(T)), lanes,
                                              max_blocks, error_flag));
        return;
    }
    auto kernel = wide ? paged_norm_append_kernel<T, kVec> : paged_norm_append_kernel<T, 1>;
    LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, static_cast<unsigned char *>(kv.k_base),
                                          static_cast<unsigned char *>(kv.v_base), NormAppendArgs(a), kv.block_table, g, d, dv,
                                          kv.vHeadStride() * int64_t(sizeof(T)), kv.vTokenStride() * int64_t(sizeof(T)),
                                          max_blocks, error_flag));
}

template <typename T>
void launch_rope_append(cudaStream_t s, const KVView &kv, void *q_out, const void *qkv, const void *bias,
                        const int32_t *seq_ids, const int32_t *positions, int32_t n_rows, int32_t nh, float theta,
                        int32_t max_blocks, int32_t *error_flag) {
    constexpr int kVec = 16 / int(sizeof(T));
    const CopyGeom g = make_geom(kv, sizeof(T));
    const int32_t d = kv.d;
    auto aligned = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool wide = d % (2 * kVec) == 0 && aligned(q_out) && aligned(qkv) && aligned(bias) && aligned(kv.k_base) &&
                      aligned(kv.v_base);
    const bool per_head = n_rows <= 1024;
    const int32_t head_groups = per_head ? nh + 2 * kv.nkvh : 4;
    const int64_t threads = int64_t(n_rows) * head_groups * (d / 2 / (wide ? kVec : 1));
    const int block = 256, grid = grid_for(threads, block);
    auto *kp = static_cast<unsigned char *>(kv.k_base);
    auto *vp = static_cast<unsigned char *>(kv.v_base);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned(grid));
    cfg.blockDim = dim3(unsigned(block));
    cfg.dynamicSmemBytes = size_t(d / 2) * sizeof(float);
    cfg.stream = s;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = kv.overlap_launch ? 1 : 0;
    T *qo = static_cast<T *>(q_out);
    const T *qi = static_cast<const T *>(qkv), *bi = static_cast<const T *>(bias);
    const int32_t *table = kv.block_table;
    auto go = [&](auto kernel) {
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, kp, vp, qo, qi, bi, table, seq_ids, positions, g, n_rows, nh, d,
                                              theta, max_blocks, error_flag));
    };
    if (wide) {
        per_head ? go(paged_rope_append_kernel<T, kVec, true>) : go(paged_rope_append_kernel<T, kVec, false>);
    } else {
        per_head ? go(paged_rope_append_kernel<T, 1, true>) : go(paged_rope_append_kernel<T, 1, false>);
    }
}

} // namespace

void paged_append(stream_t stream, size_t elem_size, const KVView &kv, const void *k_rows, const void *v_rows,
                  const int32_t *seq_ids, const int32_t *positions, int32_t n_rows, int32_t max_blocks,
                  int32_t *error_flag, const void *side_src, void *side_dst, size_t side_bytes) {
    if (n_rows <= 0) {
        return;
    }
    CHECK_ARGUMENT(side_bytes % 16 == 0 && side_bytes / 16 < size_t(INT32_MAX), "paged append: side copy size");
    const CopyGeom g = make_geom(kv, elem_size);
    const int32_t vecs_per_row = g.vecs_per_head_row * g.nkvh;
    CHECK_ARGUMENT(vecs_per_row <= 256, "paged append: a K row of more than 4 KiB is not supported");
    const int block = 256;
    // a warp per row while that fills the GPU; from there on 2, then 4 rows per warp and pass
    const int64_t full = int64_t(148) * 8 * (block / 32);
    const int rows_per_warp = n_rows >= 4 * full ? 4 : (n_rows >= 2 * full ? 2 : 1);
    const int grid = grid_for(std::max<int64_t>(int64_t(n_rows + rows_per_warp - 1) / rows_per_warp * 32, int64_t(side_bytes / 64)), block);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(unsigned(grid));
    cfg.blockDim = dim3(unsigned(block));
    cfg.stream = static_cast<cudaStream_t>(stream);
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = kv.overlap_launch ? 1 : 0;
    auto go = [&](auto kernel) {
        LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, static_cast<uint4 *>(kv.k_base), static_cast<uint4 *>(kv.v_base),
                                              static_cast<const uint4 *>(k_rows), static_cast<const uint4 *>(v_rows),
                                              kv.block_table, seq_ids, positions, g, n_rows, max_blocks, error_flag,
                                              static_cast<const uint4 *>(side_src), static_cast<uint4 *>(side_dst),
                                              int32_t(side_bytes / 16)));
    };
    if (vecs_per_row <= 32) {
        rows_per_warp == 4 ? go(paged_append_kernel<4, 1>) : rows_per_warp == 2 ? go(paged_append_kernel<2, 1>)
                                                                               : go(paged_append_kernel<1, 1>);
    } else if (vecs_per_row <= 64) {
        rows_per_warp >= 2 ? go(paged_append_kernel<2, 2>) : go(paged_append_kernel<1, 2>);
    } else {
        go(paged_append_kernel<1, 8>);
    }
    check_launch("paged_append");
}

void small_copies(stream_t stream, const void *const *src, void *const *dst, const size_t *bytes, int n) {
    CHECK_ARGUMENT(n >= 0 && n <= 3, "small_copies: at most three blocks");
    CopyList l{};
    size_t most = 0;
    for (int i = 0; i < n; ++i) {
        CHECK_ARGUMENT(bytes[i] % 16 == 0 && bytes[i] / 16 < size_t(INT32_MAX) &&
                           reinterpret_cast<uintptr_t>(src[i]) % 16 == 0 && reinterpret_cast<uintptr_t>(dst[i]) % 16 == 0,
                       "small_copies: blocks must be 16-byte aligned multiples of 16 bytes");
        l.src[i] = static_cast<const uint4 *>(src[i]);
        l.dst[i] = static_cast<uint4 *>(dst[i]);
        l.vecs[i] = int32_t(bytes[i] / 16);
        most = std::max(most, bytes[i] / 16);
    }
    if (most == 0) {
        return;
    }
    const int block = 256;
    small_copies_kernel<<<grid_for(int64_t(most), block), block, 0, static_cast<cudaStream_t>(stream)>>>(l);
    check_launch("small_copies");
}

void paged_gather(stream_t stream, size_t elem_size, const KVView &kv, int32_t seq_row, int32_t n_tokens,
                  void *k_out, void *v_out, int32_t *error_flag) {
    if (n_tokens <= 0) {
        return;
    }
    const CopyGeom g = make_geom(kv, elem_size);
    const int block = 256;
    const int grid = grid_for(int64_t(n_tokens) * 2 * g.vecs_per_head_row * g.nkvh, block);
    paged_gather_kernel<<<grid, block, 0, static_cast<cudaStream_t>(stream)>>>(
        static_cast<const uint4 *>(kv.k_base), static_cast<const uint4 *>(kv.v_base), static_cast<uint4 *>(k_out),
        static_cast<uint4 *>(v_out), kv.block_table, g, seq_row, n_tokens,
        kv.block_table ? kv.table_stride : INT32_MAX, error_flag);
    check_launch("paged_gather");
}

void paged_rope_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, void *q_out, const void *qkv,
                       const void *bias, const int32_t *seq_ids, const int32_t *positions, int32_t n_rows, int32_t nh,
                       float theta, int32_t max_blocks, int32_t *error_flag) {
    if (n_rows <= 0) {
        return;
    }
    CHECK_ARGUMENT(kv.d % 2 == 0, "rope append: head_dim must be even");
    auto s = static_cast<cudaStream_t>(stream);
    switch (dtype) {
    case LLAISYS_DTYPE_F32:
        launch_rope_append<float>(s, kv, q_out, qkv, bias, seq_ids, positions, n_rows, nh, theta, max_blocks, error_flag);
        break;
    case LLAISYS_DTYPE_F16:
        launch_rope_append<__half>(s, kv, q_out, qkv, bias, seq_ids, positions, n_rows, nh, theta, max_blocks, error_flag);
        break;
    case LLAISYS_DTYPE_BF16:
        launch_rope_append<__nv_bfloat16>(s, kv, q_out, qkv, bias, seq_ids, positions, n_rows, nh, theta, max_blocks,
                                          error_flag);
        break;
    default:
        EXCEPTION_UNSUPPORTED_DATATYPE(dtype);
    }
    check_launch("paged_rope_append");
}

void paged_norm_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const NormAppendArgs &args,
                       int32_t max_blocks, int32_t *error_flag) {
    if (args.n_rows == 0) {
        return;
    }
    auto s = static_cast<cudaStream_t>(stream);
    switch (dtype) {
    case LLAISYS_DTYPE_F32:
        launch_norm_append<float>(s, kv, args, max_blocks, error_flag);
        break;
    case LLAISYS_DTYPE_F16:
        launch_norm_append<__half>(s, kv, args, max_blocks, error_flag);
        break;
    case LLAISYS_DTYPE_BF16:
        launch_norm_append<__nv_bfloat16>(s, kv, args, max_blocks, error_flag);
        break;
    default:
        EXCEPTION_UNSUPPORTED_DATATYPE(dtype);
    }
    check_launch("paged_norm_append");
}

void latent_gather(stream_t stream, size_t elem_size, const KVView &kv, void *out, int64_t out_stride, const int32_t *seq_ids,
                   const int32_t *page_starts, const int32_t *kv_lens, int32_t n_seqs, int32_t max_kv_len, int32_t *error_flag) {
    if (n_seqs == 0 || max_kv_len == 0) {
        return;
    }
    const size_t row = size_t(kv.d) * elem_size, step = size_t(out_stride) * elem_size;
    CHECK_ARGUMENT(row % 16 == 0 && step % 16 == 0 && aligned16(out) && n_seqs <= 65535, "latent gather: rows of whole 16-byte pieces");
    CopyGeom g{};
    g.page_stride_b = kv.page_stride * int64_t(elem_size);
    g.token_stride_b = kv.token_stride * int64_t(elem_size);
    g.nkvh = 1;
    g.page_size = kv.page_size;
    g.num_pages = kv.num_pages;
    g.table_stride = kv.table_stride;
    launch_programmatic(latent_gather_kernel<uint4>, dim3(unsigned((max_kv_len + kv.page_size - 1) / kv.page_size), unsigned(n_seqs)), 128u,
                        static_cast<cudaStream_t>(stream), static_cast<const unsigned char *>(kv.k_base), kv.block_table, g,
                        static_cast<uint4 *>(out), int64_t(step / 16), int32_t(row / 16), seq_ids, page_starts, kv_lens, error_flag);
    check_launch("latent_gather");
}

void latent_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const LatentAppendArgs &args, int32_t max_blocks,
                   int32_t *error_flag) {
    if (args.n_rows == 0) {
        return;
    }
    CHECK_ARGUMENT(args.q_rank > 0 && args.rank > 0 && args.rot_dims % 2 == 0 && kv.nkvh == 1, "latent append: bad sizes");
    dispatch(dtype, [&](auto tag) { launch_latent_append<decltype(tag)>(static_cast<cudaStream_t>(stream), kv, args, max_blocks, error_flag); });
    check_launch("latent_append");
}

} // namespace llaisys::kernels
