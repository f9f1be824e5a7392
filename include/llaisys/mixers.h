/*
 * llaisys C ABI -- token mixers beyond plain causal attention, on device buffers and an explicit stream: caches whose
 * layers differ in shape, attention with a sliding window (that can keep a sequence's first tokens) and an output factor per
 * head or a penalty on distance, attention over latents, attention without a softmax whose weights are mixed over the heads, the norm /
 * rotation + append in front of them, gated linear attention, the gated delta rule, minGRU and the Mamba-2 state space with recurrent
 * state, and mixtures of experts.
 * NVIDIA devices. No counterpart in the reference.
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
 * are); then, with rot_dims > 0, dims i and i + rot_dims / 2 (i < rot_dims / 2) of each turn by the angle whose cosine and
 * sine are rot_table[row][i] (llaisysRotaryTableDev); q goes to q_out [n_rows, nh, k_dim], k and v to token positions[i] of sequence seq_ids[i], and row_scale
 * [n_rows, nh] (NULL: none) becomes gate_scale * sigmoid(gate) -- gate_scale alone without a gate. */
struct LlaisysNormAppend {
    const void *proj;
    int64_t row_stride, q_at, k_at, v_at, gate_at;
    const void *q_norm, *k_norm;
    float eps, gate_scale;
    void *q_out;
    float *row_scale;
    const int32_t *seq_ids_dev, *positions_dev;
    size_t n_rows, nh, rot_dims;
    const float *rot_table; /* [n_rows, rot_dims / 2, 2] */
    /* The row form (row_norm != 0; no rotation, no gate): bias, element by element of a row (NULL: none), is added to q, k and v;
     * q_norm [nh, k_dim] and k_norm [nkvh, k_dim] follow ONE root mean square over the whole of q and of k; q is multiplied by
     * 1 + temp_coef ln(floor((position + 1) / temp_every) + 1). */
    int row_norm;
    const void *bias;
    float temp_coef, temp_every;
    const float *head_scale; /* [nh] f32, not the row form: factor on every query head after norm and rotation (NULL: none) */
};
/* table[row, i] = (cos, sin)(positions[row] * freq[i]), i < half, all on the device */
LLAISYS_API int llaisysRotaryTableDev(llaisysDeviceType_t device_type, int device_id, float *table, const int32_t *positions_dev,
                                      const float *freq_dev, size_t n_rows, size_t half, llaisysStream_t stream);
/* the same with angles formed and reduced in f64 */
LLAISYS_API int llaisysRotaryTableWideDev(llaisysDeviceType_t device_type, int device_id, float *table, const int32_t *positions_dev,
                                          const double *freq_dev, size_t n_rows, size_t half, llaisysStream_t stream);
LLAISYS_API int llaisysPagedKVNormAppendDev(llaisysPagedKV_t kv, size_t layer, const struct LlaisysNormAppend *args,
                                            llaisysStream_t stream);

/* Attention over the pages with options. q_starts_dev NULL: one query per sequence (total_q = n_seqs); else ragged chunks as
 * in llaisysPagedAttentionPrefillDev. window > 0: the query at position i sees keys j <= i with i - j < window or
 * j < keep_first. row_scale [total_q, nh] (device, may be NULL) multiplies every head's output; row r of out starts at r * row_stride
 * elements (0: packed rows of nh * v_dim). */
LLAISYS_API int llaisysPagedAttentionOptDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q,
                                            const int32_t *seq_ids_dev, const int32_t *q_starts_dev, const int32_t *kv_lens_dev,
                                            size_t n_seqs, size_t total_q, size_t max_q_len, size_t max_kv_len, size_t nh,
                                            float scale, size_t window, size_t keep_first, const float *row_scale,
                                            size_t row_stride, llaisysStream_t stream);

/* The same without kept tokens and factors, with a penalty on distance: fade_a[h] ln(1 + fade_b[h] (i - j)) is taken off head h's score of
 * key j for the query at position i, after the scale. fade_a, fade_b [nh] f32 on the device, fade_b >= 0. */
LLAISYS_API int llaisysPagedAttentionFadeDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q, const int32_t *seq_ids_dev,
                                             const int32_t *q_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t total_q,
                                             size_t max_q_len, size_t max_kv_len, size_t nh, float scale, size_t window,
                                             const float *fade_a, const float *fade_b, size_t row_stride, llaisysStream_t stream);

/* ---- latents ----
 * A cache whose layers hold ONE row of rank[l] + rot_dim[l] elements per token: keys are whole rows, values their first rank elements, for
 * all heads. llaisysPagedAttentionOptDev runs over it with queries [rows, nh, rank + rot_dim] and outputs [rows, nh, rank]. */
LLAISYS_API int llaisysPagedKVCreateLatents(llaisysPagedKV_t *kv_out, llaisysDeviceType_t device_type, int device_id,
                                            llaisysDataType_t dtype, size_t nlayer, const size_t *rank, const size_t *rot_dim,
                                            size_t num_pages, size_t page_size, size_t max_seqs, size_t max_pages_per_seq);

/* Of a projection row: the q_rank elements at q_at, divided by their root mean square (eps inside the root) and weighted with q_norm, go to
 * q_latent (rows q_latent_stride apart); the rank elements at kv_at, treated alike with kv_norm, and behind them the next rot_dims
 * elements, dims 2 i and 2 i + 1 turned by the angle whose cosine and sine are rot_table[row][i], go to token positions[i] of sequence
 * seq_ids[i]; row_scale [n_rows, nh] (NULL: none) becomes the sigmoid of the nh elements at gate_at (< 0: 1). */
struct LlaisysLatentAppend {
    const void *proj;
    int64_t row_stride, q_at, kv_at, gate_at;
    size_t q_rank, rank, rot_dims, nh;
    const void *q_norm, *kv_norm;
    float eps;
    const float *rot_table;
    void *q_latent;
    int64_t q_latent_stride;
    float *row_scale;
    const int32_t *seq_ids_dev, *positions_dev;
    size_t n_rows;
};
LLAISYS_API int llaisysPagedKVLatentAppendDev(llaisysPagedKV_t kv, size_t layer, const struct LlaisysLatentAppend *args,
                                              llaisysStream_t stream);
/* out[r, h, out_at ..] = the rot_dims elements of q [n_rows, nh, dim + rot_dims] behind the first dim, turned as above; out rows of heads
 * out_dim apart; out may be q (out_dim = dim + rot_dims, out_at = dim) */
LLAISYS_API int llaisysRotatePairsDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, void *out, size_t out_dim,
                                      size_t out_at, const void *q, size_t dim, size_t rot_dims, const float *rot_table, size_t n_rows,
                                      size_t nh, llaisysStream_t stream);
/* Rows of the sequences with page_starts[i] >= 0, side by side: token t of sequence i -> row 16 page_starts[i] + t of out (rows out_stride
 * elements apart), zero rows up to the next multiple of 16. max_kv_len: of those sequences. */
LLAISYS_API int llaisysPagedKVLatentGatherDev(llaisysPagedKV_t kv, size_t layer, void *out, int64_t out_stride,
                                              const int32_t *seq_ids_dev, const int32_t *page_starts_dev, const int32_t *kv_lens_dev,
                                              size_t n_seqs, size_t max_kv_len, llaisysStream_t stream);
/* Causal attention of ragged chunks over plain keys and values, 16-bit, on tcgen05: a head's key is its own `dim` elements of k [tokens,
 * nh, dim] and rot_dim elements that all heads share (row t at k_shared + t * shared_stride); v [tokens, nh, vdim], vdim 64 or 128. Sequence
 * i's keys begin at row 16 page_starts[i] (< 0: left out); key blocks of 64 may read past a sequence's end, so rows up to the next multiple of
 * 64 must exist and be finite. out: row r, head h at r * out_stride + h * vdim, times row_scale[r, h] (NULL: 1). Uses kv's workspace. */
struct LlaisysExpandedAttention {
    const void *q, *k, *k_shared, *v;
    int64_t shared_stride;
    size_t tokens, nh, dim, rot_dim, vdim;
    const int32_t *page_starts_dev, *q_starts_dev, *kv_lens_dev;
    size_t n_seqs;
    float scale;
    void *out;
    int64_t out_stride;
    const float *row_scale;
};
LLAISYS_API int llaisysPagedAttentionExpandedDev(llaisysPagedKV_t kv, const struct LlaisysExpandedAttention *args, llaisysStream_t stream);

/* Attention without a softmax over the pages: head h gives key j <= i (with i - j < window, if window > 0) the weight
 *     a_hij = sigmoid(s - slopes[h] * (i - j) + bias[h]),   s = softcap * tanh(scale <q, k> / softcap)   (softcap <= 0: scale <q, k>)
 * and weighs the values of its own kv head with sum_g talk[h, g] a_gij. slopes [nh] f32, bias [nh] and talk [nh, nh] of the cache's
 * dtype, all on the device; NULL: no distance term, no bias, no mixing. Other arguments as llaisysPagedAttentionOptDev. */
struct LlaisysGates {
    float softcap;
    const float *slopes;
    const void *bias, *talk;
};
LLAISYS_API int llaisysPagedAttentionGatesDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q, const int32_t *seq_ids_dev,
                                              const int32_t *q_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t total_q,
                                              size_t max_q_len, size_t max_kv_len, size_t nh, float scale, size_t window,
                                              const struct LlaisysGates *gates, size_t row_stride, llaisysStream_t stream);

/* minGRU, element by element over `width` channels: with z_t = sigmoid(z + bias_z) and u_t = x + bias_x,
 *     S_t = (1 - z_t) S_{t-1} + z_t g(u_t),   g(u) = u + 1/2 for u >= 0, sigmoid(u) below;   out_t = S_t silu(g)
 * z, x and g are `width` elements each at z_at, x_at and g_at of a projection row; biases [width] of `dtype`; the state [width] f32
 * of slot s at state + s * slot_stride. Sequences, rows, slots and `decode` as for LlaisysGatedLinear. Runs of more than 128 tokens
 * need the scratch (llaisysMinGruScratchFloats floats). */
struct LlaisysMinGru {
    const void *proj;
    int64_t row_stride, z_at, x_at, g_at;
    const void *bias_z, *bias_x;
    size_t width;
    float *state;
    int64_t slot_stride;
    const int32_t *seq_ids_dev, *q_starts_dev, *kv_lens_dev;
    size_t n_seqs, n_rows, max_q_len;
    void *out;
    int64_t out_stride;
    float *scratch;
    size_t scratch_floats;
};
LLAISYS_API size_t llaisysMinGruScratchFloats(size_t n_rows, size_t width);
LLAISYS_API int llaisysMinGruDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const struct LlaisysMinGru *args,
                                 int decode, llaisysStream_t stream);

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

/* Gated delta rule. q, k (kv_heads x dk) and v (heads x dv) of a projection row pass a causal convolution over time of `taps`
 * taps per channel (conv_q, conv_k, conv_v [channels, taps], the last tap is the current token's, zeros before a sequence's
 * start), then silu; q and k of a head become x / sqrt(sum(x^2) + unit_eps), q also times q_scale. Head h reads q/k head
 * h / (heads / kv_heads). Per head, with state S [dk, dv] in f32:
 *     S' = diag(g_t) S_{t-1},  u_t = beta_t (v_t - S'^T k_t),  S_t = S' + k_t u_t^T,  o_t = S_t^T q_t
 *     beta_t = sigmoid(b_t),   g_t = exp(-exp(a_log_h) * softplus(x_t + dt_bias))
 *     out_t = o_t / sqrt(mean(o_t^2) + eps) * norm_w * (gate_silu ? silu : sigmoid)(gate_t)
 * x_t: with decay_w NULL one number per head, at element a_at of the row (dt_bias [heads]); else one per head and key channel,
 * decay_w z_t with decay_w [heads * dk, rank] (rows decay_ld apart) and z_t the `rank` numbers at a_at (dt_bias [heads * dk]).
 * b_t: heads numbers at b_at. gate: heads x dv at gate + r * gate_stride. All but state and scratch are of `dtype`.
 * state: slot s of a sequence holds [heads][dk][dv], then the convolutions' inputs [taps][2 kv_heads dk + heads dv] (position p
 * at p mod taps); llaisysGatedDeltaSizes gives its floats. Sequences, rows and `decode` as for LlaisysGatedLinear. scratch
 * (16-byte aligned) is needed by chunks (decode = 0); with scratch_segments long runs are cut into segments that run in
 * parallel. */
struct LlaisysGatedDelta {
    const void *proj;
    int64_t row_stride, q_at, k_at, v_at, b_at, a_at;
    const void *conv_q, *conv_k, *conv_v;
    const void *decay_w;
    int64_t decay_ld;
    const void *a_log, *dt_bias, *norm_w, *gate;
    int64_t gate_stride;
    int gate_silu;
    float q_scale, eps, unit_eps;
    size_t taps, heads, kv_heads, dk, dv, rank;
    float *state;
    int64_t slot_stride;
    const int32_t *seq_ids_dev, *q_starts_dev, *kv_lens_dev;
    size_t n_seqs, n_rows, max_q_len;
    void *out;
    int64_t out_stride;
    float *scratch;
    size_t scratch_floats;
    float *scratch_segments;
    size_t scratch_segment_floats;
};
LLAISYS_API int llaisysGatedDeltaDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype,
                                     const struct LlaisysGatedDelta *args, int decode, llaisysStream_t stream);
/* Floats of a sequence's state, of `scratch` for n_rows rows and of `scratch_segments` (any pointer may be NULL). */
LLAISYS_API void llaisysGatedDeltaSizes(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t kv_heads, size_t dk, size_t dv,
                                        size_t taps, size_t *state_floats, size_t *scratch_floats, size_t *segment_floats);

/* Mamba-2 state space. x (heads x dv), B and C (groups x dk each) follow one another at x_at of a projection row; each channel passes a
 * causal convolution over time of `taps` taps (conv_w [channels, taps], the last tap is the current token's, zeros before a sequence's
 * start; conv_b [channels]) and silu. Per head, with state S [dk, dv] in f32 (head h uses group h / (heads / groups)):
 *     dt = softplus(dt_t + dt_bias_h),  S_t = exp(-exp(a_log_h) dt) S_{t-1} + dt B_t x_t^T,  y_t = S_t^T C_t + d_skip_h x_t
 * out = norm_w * u / sqrt(mean(u^2) + eps), u = y * silu(z), the mean over each of norm_groups equal parts of the heads x dv outputs. dt_t:
 * heads numbers at dt_at; z: heads x dv at z_at. a_log, dt_bias, d_skip [heads] f32; all else of `dtype` but state and scratch. state: slot s of
 * a sequence holds [heads][dk][dv], then the convolutions' inputs [taps][channels] (position p at p mod taps). Sequences, rows and
 * `decode` as for LlaisysGatedLinear. scratch is 16-byte aligned; with scratch_segments long runs are cut into segments that start in parallel. */
struct LlaisysStateSpace {
    const void *proj;
    int64_t row_stride, z_at, x_at, dt_at;
    const void *conv_w, *conv_b, *norm_w;
    const float *a_log, *dt_bias, *d_skip;
    size_t taps, heads, groups, dk, dv, norm_groups;
    float eps;
    float *state;
    int64_t slot_stride;
    const int32_t *seq_ids_dev, *q_starts_dev, *kv_lens_dev;
    size_t n_seqs, n_rows, max_q_len;
    void *out;
    int64_t out_stride;
    float *scratch;
    size_t scratch_floats;
    float *scratch_segments;
    size_t scratch_segment_floats;
};
LLAISYS_API int llaisysStateSpaceDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype,
                                     const struct LlaisysStateSpace *args, int decode, llaisysStream_t stream);
/* Floats of a sequence's state, of `scratch` for n_rows rows and of `scratch_segments` (any pointer may be NULL). */
LLAISYS_API void llaisysStateSpaceSizes(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t groups, size_t dk, size_t dv, size_t taps,
                                        size_t *state_floats, size_t *scratch_floats, size_t *segment_floats);

/* Mixture of experts over rows h [n_rows, width]. Scores s = softmax(logits) over experts + identity outputs; the `top` largest of
 * s + correction are chosen, among the best `keep` of `groups` equal groups of neighbours (a group counts as much as its best); weight of a
 * chosen one: scale * s / (sum of the chosen s + 1e-20). Expert e: down_e (silu(gate_e h) * up_e h), gate_up [experts][gate rows, up rows][width]
 * with ff rows each, down [experts][width][ff]; outputs from `experts` on are h itself. x [n_rows, width] f32 += the weighted sum;
 * next (NULL: none) = x / sqrt(mean(x^2) + eps) * *gain of the new x, and may be h. chosen and weights [n_rows, top] are results too.
 * place, line [n_rows, top], rows and out [n_rows, top, width], act [n_rows, top, ff]: scratch; counts [experts] zero before the first
 * call (left zero). */
struct LlaisysExperts {
    size_t experts, identity, top, groups, keep, width, ff, n_rows;
    float scale, eps;
    const void *gate_up, *down;
    const float *correction, *logits, *gain;
    const void *h;
    int32_t *chosen;
    float *weights;
    int32_t *place, *counts, *line;
    void *rows, *act, *out;
    float *x;
    void *next;
};
LLAISYS_API int llaisysExpertsDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const struct LlaisysExperts *args,
                                  llaisysStream_t stream);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MIXERS_H */
