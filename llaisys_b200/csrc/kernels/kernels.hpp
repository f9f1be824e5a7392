// Host-callable launchers of every CUDA kernel in the library. Each launcher queues work on `stream` and
// returns; none allocates, synchronises or touches host copies of the data. Launchers that return int give
// 0 when work was queued and a negative value when they have no kernel for the shape (the caller then picks
// another launcher); launch failures throw.
#pragma once

#include "args.hpp"

namespace llaisys::kernels {

// Queues a memset of `bytes` zero bytes.
void fill_zero(stream_t stream, void *ptr, size_t bytes);
// The address under which kernels of the current device can read a host buffer directly: non-null only for page-locked
// host memory that is mapped into the device's address space (what cudaHostAlloc / cudaMallocHost and torch's pinned
// tensors give); null for pageable memory, for device memory and on any error.
// All `bytes` bytes from host_ptr on must lie inside one such allocation.
const void *mapped_host_alias(const void *host_ptr, size_t bytes);
// Up to three plain copies (each a 16-byte aligned multiple of 16 bytes) done by ONE kernel launch: for small blocks in
// mapped host memory, where a kernel's loads start sooner than a copy-engine transfer is set up.
void small_copies(stream_t stream, const void *const *src, void *const *dst, const size_t *bytes, int n);

// c = a + b over n contiguous elements of F32 / F16 / BF16 (arithmetic in f32).
void add(stream_t stream, llaisysDataType_t dtype, void *c, const void *a, const void *b, size_t n);

// Strided copy dst[idx] = src[idx] for every index of `shape` (ndim <= 8), elements of elem_size bytes.
void rearrange(stream_t stream, size_t elem_size, size_t ndim, const size_t *shape, const ptrdiff_t *dst_strides,
               const ptrdiff_t *src_strides, void *dst, const void *src);

// The operators around the attention path (specs: reference README.md:157-302). HBM-bound single-pass kernels; linear is
// a cuBLAS GEMM (f32 accumulation) followed by the bias add.
void argmax_rows(stream_t stream, llaisysDataType_t dtype, int64_t *idx_out, void *val_out, const void *vals, size_t rows,
                 size_t n);
void embedding(stream_t stream, size_t elem_size, void *out, const int64_t *index, const void *weight, size_t n, size_t d,
               size_t vocab);
// accumulate: out += in . W^T (the residual add of a decoder block folded into the projection; one rounding of the sum).
// in_stride, out_stride: elements between rows of `in` and `out` (0: packed rows of k and n)
void linear(stream_t stream, llaisysDataType_t dtype, void *out, const void *in, const void *weight, const void *bias,
            size_t m, size_t n, size_t k, bool accumulate = false, size_t in_stride = 0, size_t out_stride = 0);
// K6: the tcgen05 weight-streaming kernel behind linear() for at most 128 rows of 16-bit activations (K a multiple of 64,
// N a multiple of 64, not vocabulary-sized). False = shape not covered, nothing launched. overlap: programmatic launch
// (the weight stream starts under the previous kernel's tail). linear_tc_status synchronises the stream and returns (and
// clears) the kernel's error word: 0, or 16 when a bounded wait ran out.
// 0 = the streaming kernel where it measured faster (default), 1 = wherever it applies, 2 = never. False: unknown value.
bool set_linear_policy(int policy);
bool linear_tc(stream_t stream, llaisysDataType_t dtype, void *out, const void *in, const void *weight, size_t m, size_t n,
               size_t k, bool accumulate, bool overlap);
int linear_tc_status(stream_t stream);
// out[r, i] = up * silu(gate) with gate = gu[r, i], up = gu[r, di + i]: the activation on a packed gate|up projection.
void swiglu_packed(stream_t stream, llaisysDataType_t dtype, void *out, const void *gate_up, size_t rows, size_t di);
// out[r, i] = up * max(gate, 0), packed alike
void relu_glu_packed(stream_t stream, llaisysDataType_t dtype, void *out, const void *gate_up, size_t rows, size_t di);
// Row-wise argmax with every row split over several CTAs (a vocabulary-sized row on one CTA leaves the GPU idle).
// scratch: 12 * rows bytes, zero before the first call; the kernel leaves it zero again.
void argmax_rows_split(stream_t stream, llaisysDataType_t dtype, int64_t *idx_out, const void *vals, size_t rows, size_t n,
                       void *scratch);
void bias_add(stream_t stream, llaisysDataType_t dtype, void *out, const void *bias, size_t rows, size_t n);
void rms_norm(stream_t stream, llaisysDataType_t dtype, void *out, const void *in, const void *weight, float eps, size_t rows,
              size_t d);
void rope(stream_t stream, llaisysDataType_t dtype, void *out, const void *in, const int64_t *pos, float theta, size_t seq,
          size_t heads, size_t d);
void swiglu(stream_t stream, llaisysDataType_t dtype, void *out, const void *gate, const void *up, size_t n);

// Device-resident decode loop support: state hand-over between steps, CUDA graph capture / replay, event timing.
void advance_decode_state(stream_t stream, int64_t *tokens, int64_t *prev, const int64_t *next, int64_t *pos64, int32_t *pos32,
                          int32_t *kv_lens, int64_t *log, int32_t *step_counter, int n);
void graph_capture_begin(stream_t stream);
void *graph_capture_end(stream_t stream); // instantiated executable graph
void graph_launch(void *exec, stream_t stream);
void graph_destroy(void *exec);
void *event_create();
void event_record(void *event, stream_t stream);
float event_elapsed_ms(void *start, void *stop); // synchronises on `stop`
void event_destroy(void *event);

// K1: row i of k_rows / v_rows [n_rows, nkvh, d] -> token positions[i] of the sequence in table row seq_ids[i].
// 16-byte vector copies; a row whose block or page is out of range is skipped and flagged. side_src / side_dst: an
// optional plain copy of side_bytes (a multiple of 16) done by the same launch.
void paged_append(stream_t stream, size_t elem_size, const KVView &kv, const void *k_rows, const void *v_rows,
                  const int32_t *seq_ids, const int32_t *positions, int32_t n_rows, int32_t max_blocks,
                  int32_t *error_flag, const void *side_src = nullptr, void *side_dst = nullptr, size_t side_bytes = 0);

// K1b: bias + rotary embedding + append in one pass over the packed projection qkv [n_rows, (nh + 2 nkvh) * d]: rotated q
// -> q_out [n_rows, nh, d]; rotated k and plain v -> their page slots (same addressing and flags as K1).
void paged_rope_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, void *q_out, const void *qkv,
                       const void *bias, const int32_t *seq_ids, const int32_t *positions, int32_t n_rows, int32_t nh,
                       float theta, int32_t max_blocks, int32_t *error_flag);

// K1c (see NormAppendArgs); same addressing and flags as K1.
void paged_norm_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const NormAppendArgs &args,
                       int32_t max_blocks, int32_t *error_flag);

// K1d (see LatentAppendArgs); same addressing and flags as K1.
void latent_append(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const LatentAppendArgs &args, int32_t max_blocks,
                   int32_t *error_flag);
// The dims behind the first `dim` of every head of q [n_rows, nh, dim + rot_dims] turn by the row's position (dims 2 i and 2 i + 1 by
// rot_table[row][i]) -> the same elements of out rows of out_dim behind the first out_at: out [n_rows, nh, out_dim]. out may be q.
void rotate_pairs(stream_t stream, llaisysDataType_t dtype, void *out, size_t out_dim, size_t out_at, const void *q, size_t dim, size_t rot_dims,
                  const float *rot_table, size_t n_rows, size_t nh);
// nh products side by side: out[r, h, :n] = in[r, h, :k] . W_h^T, W_h [n, k] at weight + h * n * k (transposed = false) or W_h^T stored
// [k, n] there (transposed = true). Strides in elements: between rows and between heads of `in` and `out`. f32 accumulation.
void linear_heads(stream_t stream, llaisysDataType_t dtype, void *out, const void *in, const void *weight, size_t rows, size_t nh, size_t n,
                  size_t k, bool transposed, size_t in_row, size_t in_head, size_t out_row, size_t out_head);

// Mamba-2 (see StateSpaceArgs). decode: one token per sequence. chunk: ragged runs of tokens.
void state_space_decode(stream_t stream, llaisysDataType_t dtype, const StateSpaceArgs &args);
void state_space_chunk(stream_t stream, llaisysDataType_t dtype, const StateSpaceArgs &args);
// Floats of one sequence's state, of StateSpaceArgs::scratch for n_rows rows and of StateSpaceArgs::segments (0: never cut).
size_t state_space_state_floats(size_t heads, size_t groups, size_t dk, size_t dv, size_t taps);
size_t state_space_scratch_floats(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t groups, size_t dk, size_t dv);
size_t state_space_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv);

// Mixture of experts (see ExpertArgs). route: scores, choice, weights, every choice's place among its expert's rows. apply: the
// chosen experts' outputs, a row each, in args.out. combine: x[r, :] += the weighted sum of row r's choices; next (may be null): what
// becomes dtype(rms_norm(x) * *gain) of the new x (args.h is a good place: rows are read before they are written).
void experts_route(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &args);
void experts_apply(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &args);
void experts_combine(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &args, float *x, void *next, const float *gain, float eps);
// The tcgen05 form behind experts_apply: 16-bit, width and ff in whole 16-byte pieces.
bool experts_tc_covers(llaisysDataType_t dtype, const ExpertArgs &args);
void experts_tc(stream_t stream, llaisysDataType_t dtype, const ExpertArgs &args); // after experts_route and the placing of rows

// Gated delta rule (see GatedDeltaArgs). decode: one token per sequence, everything in one launch. chunk: ragged runs of
// tokens.
void gated_delta_decode(stream_t stream, llaisysDataType_t dtype, const GatedDeltaArgs &args);
void gated_delta_chunk(stream_t stream, llaisysDataType_t dtype, const GatedDeltaArgs &args);
// Floats of one sequence's state: the matrices of all heads, then the newest `taps` inputs of the short convolutions.
size_t gated_delta_state_floats(size_t heads, size_t kv_heads, size_t dk, size_t dv, size_t taps);
// Floats of GatedDeltaArgs::scratch for n_rows rows, and of GatedDeltaArgs::segments (0: chunk calls are never cut).
size_t gated_delta_scratch_floats(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t kv_heads, size_t dk, size_t dv);
size_t gated_delta_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv);

// minGRU (see MinGruArgs). decode: one token per sequence. chunk: ragged runs of tokens.
void min_gru_decode(stream_t stream, llaisysDataType_t dtype, const MinGruArgs &args);
void min_gru_chunk(stream_t stream, llaisysDataType_t dtype, const MinGruArgs &args);
size_t min_gru_scratch_floats(size_t n_rows, size_t width); // of MinGruArgs::scratch

// Gated linear attention (see GatedLinearArgs). decode: one token per sequence, everything in one launch. chunk: ragged
// runs of tokens.
void gated_linear_decode(stream_t stream, llaisysDataType_t dtype, const GatedLinearArgs &args);
void gated_linear_chunk(stream_t stream, llaisysDataType_t dtype, const GatedLinearArgs &args);
// Floats of GatedLinearArgs::segments that serve every chunk call of these sizes; 0 = such calls are never cut.
size_t gated_linear_segment_floats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv);

// ---- operators of a residual stream kept in f32 (x float [rows, d]) around dtype activations ----
// x[r, :] = scale * w[tokens[r], :]; copy (may be null): the same rounded to dtype, row r at copy + r * copy_stride
void embed_scaled(stream_t stream, llaisysDataType_t dtype, float *x, void *copy, int64_t copy_stride, const int64_t *tokens,
                  const void *w, float scale, size_t rows, size_t d, size_t vocab);
// x[r, :] = w[tokens[r], :] + pairs[b, :] with b = (prev[r] * mul_prev + tokens[r] * mul_cur) mod buckets, or b = buckets where
// prev[r] < 0 (no token before this one); pairs has buckets + 1 rows
void embed_pairs(stream_t stream, llaisysDataType_t dtype, float *x, const int64_t *tokens, const int64_t *prev, const void *w,
                 const void *pairs, int64_t mul_prev, int64_t mul_cur, int64_t buckets, size_t rows, size_t d, size_t vocab);
// x[r, :] = w[tokens[r], :] + (sin, cos, sin, cos, ..)(positions[r] * freq[i]) for columns 2 i and 2 i + 1; freq [(d + 1) / 2] f64
void embed_positions(stream_t stream, llaisysDataType_t dtype, float *x, const int64_t *tokens, const int32_t *positions,
                     const double *freq, const void *w, size_t rows, size_t d, size_t vocab);
// out[r, :] = dtype(x[r, :]), row r at out + r * out_stride
void stream_cast(stream_t stream, llaisysDataType_t dtype, void *out, int64_t out_stride, const float *x, size_t rows, size_t d);
// out[i, :] = rms_norm(x[r, :]) * (offset + w) with r = row_index[i] (null: r = i), f32 arithmetic, one rounding. offset 1: a
// weight stored around zero
void stream_rms_norm(stream_t stream, llaisysDataType_t dtype, void *out, const float *x, const int64_t *row_index,
                     const void *w, float eps, size_t rows, size_t d, float offset = 0.f);
// the same with one number (f32, on the device) for all columns: out[i, :] = rms_norm(x[r, :]) * *gain
void stream_rms_norm_gain(stream_t stream, llaisysDataType_t dtype, void *out, const float *x, const int64_t *row_index,
                          const float *gain, float eps, size_t rows, size_t d);
// out (f32) = alpha * in . W^T (+ out when accumulate): a projection into the stream, or logits
void linear_f32(stream_t stream, llaisysDataType_t dtype, float *out, const void *in, const void *weight, size_t m, size_t n,
                size_t k, bool accumulate, float alpha = 1.f, size_t in_stride = 0);
// v = max(v, 0)^2 in place
void relu_squared(stream_t stream, llaisysDataType_t dtype, void *v, size_t n);
// out = gelu(in), tanh form, [rows, n] each with its own row stride (elements)
void gelu_tanh(stream_t stream, llaisysDataType_t dtype, void *out, int64_t out_stride, const void *in, int64_t in_stride,
               size_t rows, size_t n);
// x += scale * (rms_norm(a) * (branch_offset + wa) + rms_norm(b) * (branch_offset + wb)), a and b f32 [rows, d] like x (b may be
// null: one branch); h (may be null) = dtype(rms_norm(x) * (offset + w)) of the new x, the norm that comes next
void stream_add_normed(stream_t stream, llaisysDataType_t dtype, float *x, const float *a, const void *wa, const float *b,
                       const void *wb, float scale, float eps, void *h, const void *w, float offset, size_t rows, size_t d,
                       float branch_offset = 0.f);
// table[r, i] = (cos, sin)(positions[r] * freq[i]), i < half
void rotary_table(stream_t stream, float *table, const int32_t *positions, const float *freq, size_t rows, size_t half);
// the same with angles in f64, reduced to a turn before they are rounded
void rotary_table(stream_t stream, float *table, const int32_t *positions, const double *freq, size_t rows, size_t half);
// logits = cap * tanh(logits / cap) in place (cap <= 0: unchanged) and the row-wise argmax of the result, one launch;
// scratch as argmax_rows_split
void softcap_argmax(stream_t stream, float *logits, float cap, int64_t *idx_out, size_t rows, size_t n, void *scratch);

// K5: tokens [0, n_tokens) of table row seq_row -> k_out, v_out [n_tokens, nkvh, d].
void paged_gather(stream_t stream, size_t elem_size, const KVView &kv, int32_t seq_row, int32_t n_tokens,
                  void *k_out, void *v_out, int32_t *error_flag);

// Any dtype, V rows of up to 1024, any GQA ratio, any page size, windows, kept tokens, distance penalties: one CTA per (query row, query head), online
// softmax in f32. The correctness baseline for the specialised kernels and the kernel behind the legacy
// operator for shapes they do not cover.
void attention_generic(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch,
                       const void *q, float scale, const AttnOut &out, int32_t *error_flag);

// Attention without a softmax whose weights are mixed over the heads (see GateArgs). Any dtype and sizes, windows but no kept
// tokens, neither partial results nor output factors. The kernel behind shapes that attention_gates_tiles does not cover.
void attention_gates(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                     const GateArgs &gates, const AttnOut &out, int32_t *error_flag);

// The same on the tensor cores: bf16, rows of at most 128 in whole 16-element steps, 16-token pages, at most 64 heads. Returns -1 if
// the view or shape is not covered, or the scratch is smaller than attention_gates_tiles_scratch asks for.
int attention_gates_tiles(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                          const GateArgs &gates, const AttnOut &out, const AttnScratch &scratch);
void attention_gates_tiles_scratch(size_t longest_v_row, size_t *floats, size_t *counters);

// The same on tcgen05 for chunks over page pools that carry the half-tile tensor map (KVView::tma_tile_desc): bf16, K and V rows of 128,
// at most 32 heads and 16 kv heads, chunks of 8 tokens or more among them. Returns -1 if the view or shape is not covered, or the
// scratch (as above) is smaller than attention_gates_tc_scratch asks for.
int attention_gates_tc(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                       const GateArgs &gates, const AttnOut &out, const AttnScratch &scratch);
void attention_gates_tc_scratch(size_t *floats, size_t *counters);

// K2 (+ fused K3): split-KV flash decoding for 16-bit K/V, head_dim 128, page size 16, GQA group <= 8,
// one query per sequence. Returns -1 if the shape is not covered.
int attention_decode_split(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch,
                           const void *q, float scale, const AttnOut &out, const AttnScratch &scratch);
// Scratch the split-KV decode needs for a batch of n_seqs sequences of at most max_kv_len tokens.
void attention_decode_split_scratch(int32_t n_seqs, int32_t nh, int32_t nkvh, int32_t d, int32_t max_kv_len,
                                    size_t *partials_floats, size_t *counters_len);

// Number of persistent CTAs the split-KV decode kernels launch for a batch (two per SM, fewer for tiny batches).
int decode_grid_size(int32_t n_seqs, int32_t nkvh, int32_t max_kv_len);

// TMA edition of K2 + K3 for page pools that carry a tensor map (KVView::tma_desc). Same contract and scratch
// as attention_decode_split. k_new / v_new (both or neither; [n_seqs, nkvh, 128], 16-byte aligned): fused step -- row i
// is also appended as token kv_lens[i] - 1 of sequence i by the same launch. Returns -1 and sets *why (a static string)
// if the view or shape is not covered; nothing is queued then.
int attention_decode_tma(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch,
                         const void *q, float scale, const AttnOut &out, const AttnScratch &scratch,
                         const void *k_new = nullptr, const void *v_new = nullptr, const char **why = nullptr);
// Encodes the tensor map over a 16-bit page pool (head_dim 128, page 16) starting at pool_base into out_128_bytes
// (host memory): total_rows rows of 128 elements, nkvh of them per (page, K|V) block of 16 slots each. Returns -1
// when the driver cannot provide one (the cp.async kernel is used then).
int make_kv_tensor_map(void *out_128_bytes, void *pool_base, uint64_t total_rows, uint32_t nkvh, llaisysDataType_t dtype);

// K4: chunked-prefill attention on tcgen05 for page pools that carry the half-tile tensor map
// (KVView::tma_tile_desc): 16-bit K/V, head_dim 128, page 16, ragged causal chunks (batch.q_starts). Returns -1 if
// the view or shape is not covered, or the scratch is smaller than attention_prefill_tc_scratch asks for (partial
// results of tiles that are split over CTAs, and their arrival counters, which must be zero between launches).
int attention_prefill_tc(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch,
                         const void *q, float scale, const AttnOut &out, const AttnScratch &scratch);
void attention_prefill_tc_scratch(size_t *floats, size_t *counters);
// Two maps, 128 bytes each: the half-tile map (K) and the whole-tile-as-two-halves map (V).
int make_kv_tile_tensor_map(void *out_256_bytes, void *pool_base, uint64_t total_rows, uint32_t nkvh,
                            llaisysDataType_t dtype);

// Decode and short chunks over pages of latents (views whose V rows lie in their K rows) on tcgen05: 16-bit, 16-token pages, V parts of up
// to 512 elements, rows of whole 16-byte pieces of which at most one 64-element piece lies behind the V part's last 128. batch.q_starts may
// begin anywhere in q and out (rows are absolute; total_q: rows of this call). Returns -1 if the view or shape is not covered, or the
// scratch (attention_latent_scratch floats) is too small.
bool attention_latent_covers(llaisysDataType_t dtype, size_t nh, size_t rank, size_t dim);
size_t attention_latent_scratch(size_t rank);
int attention_latent_tc(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                        const AttnOut &out, const AttnScratch &scratch);

// K4 over plain tensors with keys in two parts (see ExpandedArgs): 16-bit, own parts of up to 128 dims and shared ones of up to 64 in steps
// of 8, V rows of 64 or 128. Returns -1 if the sizes or the scratch (as attention_prefill_tc) do not fit.
bool attention_expanded_covers(llaisysDataType_t dtype, size_t dim, size_t rot_dim, size_t vdim);
int attention_expanded_tc(stream_t stream, llaisysDataType_t dtype, const ExpandedArgs &args, const AttnScratch &scratch);

// Rows [0, kv_lens[i]) of the sequences with page_starts[i] >= 0 (layers whose V rows lie in their K rows) -> out rows 16 page_starts[i] ..,
// kv.d elements each, out_stride apart, zeros up to the next multiple of 16 rows. max_kv_len: of those sequences.
void latent_gather(stream_t stream, size_t elem_size, const KVView &kv, void *out, int64_t out_stride, const int32_t *seq_ids,
                   const int32_t *page_starts, const int32_t *kv_lens, int32_t n_seqs, int32_t max_kv_len, int32_t *error_flag);

// K3: out[r, :] = sum_p w_p o_p[r, :] / sum_p w_p, w_p = l_p exp(m_p - max_p m_p), over n_parts partials laid out
// float [n_parts][n_rows][d + 2].
void lse_merge(stream_t stream, llaisysDataType_t dtype, void *out, const float *parts, int32_t n_parts,
               int32_t n_rows, int32_t d);

} // namespace llaisys::kernels
