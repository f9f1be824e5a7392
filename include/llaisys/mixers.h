/*
 * llaisys C ABI -- token mixers beyond plain causal attention, on device buffers and an explicit stream: caches whose
 * layers differ in shape, attention with a sliding window and an output factor per head, the position-free norm + append
 * in front of it, and gated linear attention with recurrent state. NVIDIA devices. No counterpart in the reference.
 * Status codes as in paged_kv.h; as for every ...Dev call there: no host validation of index arrays, no staging copy.
 */
#ifndef LLAISYS_MIXERS_H
#define LLAISYS_MIXERS_H

#include "paged_kv.h"

#ifdef __cplusplus
extern "C" {
#endif

/* As llaisysPagedKVCreate, with one shape per layer: nkvh[l] kv-heads, K rows of k_dim[l] and V rows of v_dim[l] elements
 * (any length: rows are padded to 16 bytes in the pool). Append, gather and rope append need equal, unpadded rows. */
LLAISYS_API int llaisysPagedKVCreateLayers(llaisysPagedKV_t *kv_out, llaisysDeviceType_t device_type, int device_id,
                                           llaisysDataType_t dtype, size_t nlayer, const size_t *nkvh, const size_t *k_dim,
                                           const size_t *v_dim, size_t num_pages, size_t page_size, size_t max_seqs,
                                           size_t max_pages_per_seq);

/* One projection row per token, [n_rows, row_stride] of the cache's dtype, holding q [nh, k_dim] at element q_at, k
 * [nkvh, k_dim] at k_at, v [nkvh, v_dim] at v_at and (gate_at >= 0) one gate number per query head. q and k heads are
 * divided by their root mean square (eps inside the root) and weighted with q_norm / k_norm [k_dim] (NULL: left as they
 * are); q goes to q_out [n_rows, nh, k_dim], k and v to token positions[i] of sequence seq_ids[i], and row_scale
 * [n_rows, nh] (NULL: none) becomes gate_scale * sigmoid(gate) -- gate_scale alone without a gate. */
struct LlaisysNormAppend {
    const void *proj;
    int64_t row_stride, q_at, k_at, v_at, gate_at;
    const void *q_norm, *k_norm;
    float eps, gate_scale;
    void *q_out;
    float *row_scale;
    const int32_t *seq_ids_dev, *positions_dev;
    size_t n_rows, nh;
};
LLAISYS_API int llaisysPagedKVNormAppendDev(llaisysPagedKV_t kv, size_t layer, const struct LlaisysNormAppend *args,
                                            llaisysStream_t stream);

/* Attention over the pages with options. q_starts_dev NULL: one query per sequence (total_q = n_seqs); else ragged chunks as
 * in llaisysPagedAttentionPrefillDev. window > 0: the query at position i sees keys j with 0 <= i - j < window.
 * row_scale [total_q, nh] (device, may be NULL) multiplies every head's output; row r of out starts at r * row_stride
 * elements (0: packed rows of nh * v_dim). */
LLAISYS_API int llaisysPagedAttentionOptDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q,
                                            const int32_t *seq_ids_dev, const int32_t *q_starts_dev, const int32_t *kv_lens_dev,
                                            size_t n_seqs, size_t total_q, size_t max_q_len, size_t max_kv_len, size_t nh,
                                            float scale, size_t window, const float *row_scale, size_t row_stride,
                                            llaisysStream_t stream);

/* Gated linear attention. Per head, with state S [dk, dv] in f32 (row-major, slot s of the sequence in seq_ids at
 * state + s * slot_stride + head * dk * dv):
 *     a_t = sigmoid(decay_w z_t + decay_b)^(1 / tau),   S_t = diag(a_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T (q_scale q_t)
 *     out_t = out_scale * o_t / sqrt(mean(o_t^2) + eps) * norm_w * silu(g_t)
 * proj [n_rows, row_stride] holds q, k (heads x dk), v, g (heads x dv) and z (rank numbers) at the given elements; decay_w
 * [heads * dk, rank], decay_b [heads * dk], norm_w [dv], out (row r, head h at r * out_stride + h * dv), all of `dtype`.
 * Sequence i owns rows [q_starts[i], q_starts[i + 1]) and has kv_lens[i] tokens after the call; one whose tokens are all in
 * this call starts from a zero state whatever its slot holds. scratch_raw [n_rows, heads * dv] and scratch_decay
 * [n_rows, heads * dk] f32: needed by chunks of more than one token (decode = 0), and scratch_segments (see
 * llaisysGatedLinearSegmentFloats) where long runs are to be cut into segments that run in parallel (NULL: they are not).
 * decode = 1: every sequence has exactly one row (q_starts unused). */
struct LlaisysGatedLinear {
    const void *proj;
    int64_t row_stride, q_at, k_at, v_at, g_at, z_at;
    const void *decay_w, *decay_b, *norm_w;
    float tau, q_scale, eps, out_scale;
    size_t heads, dk, dv, rank;
    float *state;
    int64_t slot_stride;
    const int32_t *seq_ids_dev, *q_starts_dev, *kv_lens_dev;
    size_t n_seqs, n_rows, max_q_len;
    void *out;
    int64_t out_stride;
    float *scratch_raw, *scratch_decay, *scratch_segments;
    size_t scratch_segment_floats;
};
LLAISYS_API int llaisysGatedLinearDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype,
                                      const struct LlaisysGatedLinear *args, int decode, llaisysStream_t stream);
/* Floats of scratch_segments that serve every call of these sizes (0: such calls are never cut). */
LLAISYS_API size_t llaisysGatedLinearSegmentFloats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MIXERS_H */
