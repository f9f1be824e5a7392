// Plain-data argument blocks shared by the CPU loops and the CUDA kernels of the attention path.
// Everything here is host-compilable (no CUDA types) so the operator layer can stay ordinary C++.
#pragma once

#include "llaisys.h"

#include <cstddef>
#include <cstdint>

#ifdef __CUDACC__
#define LLAISYS_ARGS_FN __host__ __device__
#else
#define LLAISYS_ARGS_FN
#endif

namespace llaisys::kernels {

// Where the K and V rows of a sequence live. One description covers both layouts on the path:
//   paged pool   pool[page][K|V][kvh][slot][d]  -> page_stride = 2*nkvh*ps*d, head_stride = ps*d, token_stride = d,
//                v_base = k_base + nkvh*ps*d, block_table maps (sequence row, block) -> physical page;
//   contiguous   k[total, nkvh, d] as the legacy operator receives it
//                -> page_stride = ps*nkvh*d, head_stride = d, token_stride = nkvh*d, block_table = nullptr
//                (block b IS page b).
struct KVView {
    void *k_base = nullptr; // element (page 0, kv-head 0, slot 0, dim 0) of K (written only by append)
    void *v_base = nullptr; // same for V
    int64_t page_stride = 0;      // all strides in elements
    int64_t head_stride = 0;
    int64_t token_stride = 0;
    const int32_t *block_table = nullptr; // [rows][table_stride] on the executing device, or nullptr
    int32_t table_stride = 0;
    int32_t page_size = 16;
    int32_t num_pages = 0; // physical pages addressable through this view (bounds check)
    int32_t nkvh = 0;
    int32_t d = 0; // elements of a K row (and of a V row unless v_d says otherwise)
    // V rows of another shape than K rows (0 = the same): used by the generic attention and the norm + append kernel; every
    // other kernel needs equal shapes.
    int32_t v_d = 0;
    int64_t v_head_stride = 0, v_token_stride = 0;
    LLAISYS_ARGS_FN int32_t vDim() const { return v_d ? v_d : d; }
    LLAISYS_ARGS_FN int64_t vHeadStride() const { return v_d ? v_head_stride : head_stride; }
    LLAISYS_ARGS_FN int64_t vTokenStride() const { return v_d ? v_token_stride : token_stride; }
    // Optional TMA view of the same memory (page pools only): a 128-byte tensor-map blob in HOST memory over the
    // whole multi-layer pool, and the index of this layer's page 0 in it (layer * num_pages).
    // Launch append / decode with programmatic stream serialisation: the kernel's set-up and its first K/V copies may
    // overlap the tail of the previous kernel on the stream. Contract for the caller: index arrays and block tables were
    // written before that previous kernel started (K/V rows, q and outputs are only touched after it completed).
    bool overlap_launch = false;
    const void *tma_desc = nullptr;      // box = K and V of a page, 64 dims (decode)
    const void *tma_tile_desc = nullptr; // prefill, two maps of 128 bytes: box = one half-tile, 16 slots x 64 dims (K); box = a
                                         // tile as its two halves, 16 slots x 64 dims x 2 (V)
    int64_t tma_page0 = 0;
};

// Which queries attend to which sequences. Arrays live on the executing device; a null array selects the
// scalar that follows it (the legacy single-sequence operator has no arrays to pass).
struct AttnBatch {
    const int32_t *seq_ids = nullptr;  // [n_seqs] row of block_table per sequence; null: row i for sequence i
    const int32_t *kv_lens = nullptr;  // [n_seqs]; null: every sequence has const_kv_len tokens
    const int32_t *q_starts = nullptr; // [n_seqs + 1] first query row of each sequence; null: const_q_len each
    // The same seq_ids / kv_lens in HOST memory, for a caller that has them there anyway: the TMA decode kernel then takes
    // them by value with the launch (batches of at most 256 sequences) and the device arrays above may be null.
    const int32_t *host_seq_ids = nullptr;
    const int32_t *host_kv_lens = nullptr;
    int32_t const_kv_len = 0;
    int32_t const_q_len = 1;
    int32_t n_seqs = 0;
    int32_t total_q = 0; // rows of q / out
    int32_t max_q_len = 1;
    int32_t max_kv_len = 0;
    int32_t nh = 0;
    int32_t window = 0; // > 0: a query at position i sees keys j with 0 <= i - j < window; 0: all earlier keys
    int32_t keep_first = 0; // with a window: keys j < keep_first stay visible behind it (j <= i)
    // Distance penalty of the softmax kernels: fade_a[h] ln(1 + fade_b[h] (i - j)) is taken off head h's score (after the scale).
    // f32 [nh] on the executing device; null: none. fade_b >= 0.
    const float *fade_a = nullptr, *fade_b = nullptr;
};

// Output selection: `out` [total_q, nh, d] in the KV dtype, or `part` float [total_q, nh, d + 2] holding the
// locally normalised output followed by m (max scaled score, natural-log units) and l (sum of exp(score - m)).
struct AttnOut {
    void *out = nullptr;
    float *part = nullptr;
    // out only: every (row, head) of the normalised output is multiplied by row_scale[row * nh + h] (an output gate), and
    // row r starts at out + r * row_stride elements (0 = packed rows of nh * d)
    const float *row_scale = nullptr;
    int64_t row_stride = 0;
    const struct PeerSink *peers = nullptr; // decode over a page pool only: partial rows go to exchange slots instead
};

// Attention without a softmax: the weight of a visible key j for head h and the query at position i is
//   a_hij = sigmoid(score - slopes_h (i - j) + bias_h),  score = softcap tanh(scale <q, k> / softcap), or scale <q, k> without a cap,
// and head h weighs the values of its kv head with sum_g talk[h, g] a_gij. Nothing is normalised over the keys.
struct GateArgs {
    float softcap = 0.f;           // <= 0: none
    const float *slopes = nullptr; // [nh] on the device; null: no distance term
    const void *bias = nullptr;    // [nh], cache dtype; null: none
    const void *talk = nullptr;    // [nh, nh], cache dtype; null: every head keeps its own weights
};

// Exchange buffers of a KV-range split across the GPUs of a node, as rank `rank` sees them: table[r] (an array in
// device memory) is rank r's buffer, peer memory for r != rank, and `own` is table[rank]. A buffer holds 2 (step
// parity) x world slots of slot_floats 8-byte words -- slot s of parity p is written by rank s; a word is a float and,
// beside it, the number of the step it belongs to, so that a reader can tell a current value from a stale one without
// any flag or fence -- then, at epoch_offset bytes, the step counter (merges completed). `rows` is local memory for
// this rank's rows [n_rows][d + 2] on their way out: the kernel completes a row there and copies it to every rank.
struct PeerSink {
    unsigned char *const *table = nullptr;
    unsigned char *own = nullptr;
    float *rows = nullptr;
    int32_t world = 0, rank = 0;
    size_t slot_floats = 0, epoch_offset = 0;
};

// Device-side scratch a launch may use (split-KV partials and arrival counters); owned by the caller.
struct AttnScratch {
    float *partials = nullptr;    // float [capacity]
    size_t partials_floats = 0;
    int32_t *counters = nullptr;  // int32 [counters_len], all zero between launches
    size_t counters_len = 0;
    int32_t *error_flag = nullptr; // set non-zero when a kernel skipped an out-of-range page / position
};

// K1c: what enters attention, fused: from a packed projection row [.. q | k | v .. gate ..] the per-head RMS norm of q and k
// (one weight of `d` for all heads), the rotation of their first rot_dims dimensions, k and v into their page slots, q to a
// packed tensor, and the output gate of every head turned into a factor for the attention kernel's epilogue. Norm, rotation
// and gate are optional.
struct NormAppendArgs {
    const void *proj = nullptr; // [n_rows, row_stride] elements of the cache's dtype
    int64_t row_stride = 0;
    int64_t q_at = 0, k_at = 0, v_at = 0, gate_at = 0; // first element of each part in a row; gate_at < 0: no gate
    const void *q_norm = nullptr, *k_norm = nullptr;   // [d], cache dtype; null = no norm
    float eps = 0.f;
    // dims i and i + rot_dims / 2 (i < rot_dims / 2) turn by the angle whose (cos, sin) is rot_table[row][i] (rotary_table)
    int32_t rot_dims = 0;
    const float *rot_table = nullptr; // [n_rows, rot_dims / 2, 2]
    void *q_out = nullptr;      // [n_rows, nh, d]
    float *row_scale = nullptr; // [n_rows, nh] = gate_scale * sigmoid(gate)
    float gate_scale = 1.f;
    const int32_t *seq_ids = nullptr, *positions = nullptr; // per row, on the device
    size_t n_rows = 0;
    int32_t nh = 0;
    // The row form (row_norm != 0; no rotation, no gate): `bias` (element e belongs to element e of a row; null: none) is added
    // to q, k and v; q_norm [nh * d] and k_norm [nkvh * d] go with ONE root mean square over the whole of q and of k; q is then
    // multiplied by 1 + temp_coef ln(floor((position + 1) / temp_every) + 1)
    int32_t row_norm = 0;
    const void *bias = nullptr;
    float temp_coef = 0.f, temp_every = 1.f;
    const float *head_scale = nullptr; // [nh] f32, not the row form: factor on every query head after norm and rotation; null: none
};

// K1d: what enters attention over latents. Of a packed projection row [.. query latent | key latent, key part to turn | gates ..]: the
// query latent normed -> q_latent; the key latent normed and, behind it, the other key dims turned by their position -> the
// token's row of the cache (KVView of one kv head, K rows of rank + rot_dims); a gate per head -> factor of the attention's epilogue.
struct LatentAppendArgs {
    const void *proj = nullptr; // [n_rows, row_stride], cache dtype
    int64_t row_stride = 0;
    int64_t q_at = 0, kv_at = 0, gate_at = 0; // gate_at < 0: no gate
    int32_t q_rank = 0, rank = 0, rot_dims = 0, nh = 0;
    const void *q_norm = nullptr, *kv_norm = nullptr; // [q_rank], [rank]
    float eps = 0.f;
    const float *rot_table = nullptr; // [n_rows, rot_dims / 2, 2] (rotary_table): dims 2 i and 2 i + 1 turn
    void *q_latent = nullptr;         // [n_rows, q_latent_stride]
    int64_t q_latent_stride = 0;
    float *row_scale = nullptr;       // [n_rows, nh] = sigmoid(gate)
    const int32_t *seq_ids = nullptr, *positions = nullptr;
    size_t n_rows = 0;
};

// Causal attention of ragged chunks over plain K and V tensors of a whole batch, the keys of a head being `dim` dims of their own and
// rot_dim dims that all heads share. Sequence i's keys are rows 16 page_starts[i] .. + kv_lens[i] (page_starts[i] < 0: left out); rows up
// to the next multiple of 64 may be read and must be finite.
struct ExpandedArgs {
    const void *q = nullptr;        // [rows, nh, dim + rot_dim]
    const void *k = nullptr;        // [tokens, nh, dim]
    const void *k_shared = nullptr; // row t at k_shared + t * shared_stride, [rot_dim]
    int64_t shared_stride = 0;
    const void *v = nullptr;        // [tokens, nh, vdim]
    int64_t tokens = 0;
    int32_t nh = 0, dim = 0, rot_dim = 0, vdim = 0;
    const int32_t *page_starts = nullptr, *q_starts = nullptr, *kv_lens = nullptr; // [n_seqs], [n_seqs + 1], [n_seqs] on the device
    int32_t n_seqs = 0;
    float scale = 1.f;
    void *out = nullptr; // row r, head h: out + r * out_stride + h * vdim, times row_scale[r * nh + h] (null: 1)
    int64_t out_stride = 0;
    const float *row_scale = nullptr;
};

// Mamba-2 over one packed projection row [.. z | .. x, B, C .. | dt ..]: x (heads x dv), B and C (groups x dk each) follow one another at
// x_at, pass a causal convolution of `taps` taps per channel with a bias, and silu. Per head a state S [dk, dv]; head h uses group
// h / (heads / groups):
//   dt = softplus(dt_t + dt_bias_h),  S_t = exp(-exp(a_log_h) dt) S_{t-1} + dt B_t x_t^T,  y_t = S_t^T C_t + d_skip_h x_t
// out = norm_w * rms_norm(y * silu(z)), the norm in norm_groups equal parts of the heads' concatenated outputs.
struct StateSpaceArgs {
    const void *proj = nullptr; // [n_rows, row_stride], model dtype
    int64_t row_stride = 0;
    int64_t z_at = 0, x_at = 0, dt_at = 0;
    const void *conv_w = nullptr, *conv_b = nullptr; // [channels, taps] (the last tap is the current token's), [channels]
    const void *norm_w = nullptr;                    // [heads * dv]
    const float *a_log = nullptr, *dt_bias = nullptr, *d_skip = nullptr; // [heads]
    int32_t taps = 0, heads = 0, groups = 0, dk = 0, dv = 0, norm_groups = 1;
    float eps = 0.f;
    // slot s: the heads' matrices [heads][dk][dv], then convolution inputs [taps][channels]: position p at p mod taps
    float *state = nullptr;
    int64_t slot_stride = 0;
    // the batch: sequence i owns rows [q_starts[i], q_starts[i + 1]) and state slot seq_ids[i]; kv_lens[i] tokens after the
    // step (a sequence whose first token is in the step starts from zero)
    const int32_t *seq_ids = nullptr, *q_starts = nullptr, *kv_lens = nullptr;
    int32_t n_seqs = 0, n_rows = 0, max_q_len = 0;
    void *out = nullptr; // row r: out + r * out_stride, [heads * dv], model dtype
    int64_t out_stride = 0;
    float *scratch = nullptr; // state_space_scratch_floats, 16-byte aligned
    size_t scratch_floats = 0;
    float *segments = nullptr; // state_space_segment_floats; null: runs are never cut
    size_t segment_floats = 0;
    LLAISYS_ARGS_FN int32_t inner() const { return heads * dv; }
    LLAISYS_ARGS_FN int32_t channels() const { return heads * dv + 2 * groups * dk; }
};

// Mixture of experts over rows h [n_rows, width]. The router's logits become scores s = softmax over experts + identity outputs;
// `top` of them are chosen by s + correction, among the best `keep` of `groups` equal groups (a group counts as much as its best
// choice score); weight of a chosen one: scale * s / (sum of the chosen s + 1e-20). Expert e: down_e (silu(gate_e h) * up_e h);
// outputs from `experts` on are identity experts: h itself.
struct ExpertArgs {
    int32_t experts = 0, identity = 0, top = 0, groups = 1, keep = 1;
    float scale = 1.f;
    int32_t width = 0, ff = 0;        // ff: padded rows per expert of `gate_up` halves, columns of `down`
    const void *gate_up = nullptr;    // [experts][2 ff][width]: gate rows, then up rows
    const void *down = nullptr;       // [experts][width][ff]
    const float *correction = nullptr; // [experts + identity]
    const float *logits = nullptr;    // [n_rows, experts + identity]
    const void *h = nullptr;          // [n_rows, width], model dtype
    int32_t n_rows = 0;
    // routing (written by experts_route): per row `top` choices; rows of every expert in one line, expert after expert
    int32_t *chosen = nullptr;  // [n_rows, top] expert
    float *weights = nullptr;   // [n_rows, top]
    int32_t *place = nullptr;   // [n_rows, top] row in the line (after experts_place); -1 for an identity expert
    int32_t *counts = nullptr;  // [experts] rows of every expert, zero before experts_route
    int32_t *line = nullptr;    // [n_rows * top] source row of every row in the line
    void *rows = nullptr;       // [n_rows * top, width] the line's inputs (tensor-core form)
    void *act = nullptr;        // [n_rows * top, ff]
    void *out = nullptr;        // [n_rows * top, width]
};

// Gated linear attention over one packed projection (per head a state S [dk, dv], decayed per key channel):
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T (q_scale q_t),  a_t = exp(log_sigmoid(W_a2 z_t + b) / tau)
//   out_t = out_scale * rms_norm(o_t, norm) * silu(g_t)
// q, k: heads x dk; v, g, out: heads x dv; z: the low-rank half of the decay projection, `rank` numbers shared by all heads.
struct GatedLinearArgs {
    const void *proj = nullptr; // [n_rows, row_stride], model dtype
    int64_t row_stride = 0;
    int64_t q_at = 0, k_at = 0, v_at = 0, g_at = 0, z_at = 0;
    const void *decay_w = nullptr; // [heads * dk, rank], model dtype
    const void *decay_b = nullptr; // [heads * dk]
    const void *norm_w = nullptr;  // [dv]
    float tau = 1.f, q_scale = 1.f, eps = 0.f, out_scale = 1.f;
    int32_t heads = 0, dk = 0, dv = 0, rank = 0;
    float *state = nullptr; // slot s, head h: state + s * slot_stride + h * dk * dv, row-major [dk, dv]
    int64_t slot_stride = 0;
    // the batch: sequence i owns rows [q_starts[i], q_starts[i + 1]) and state slot seq_ids[i]; kv_lens[i] tokens after the
    // step (a sequence whose first token is in the step starts from zero)
    const int32_t *seq_ids = nullptr, *q_starts = nullptr, *kv_lens = nullptr;
    int32_t n_seqs = 0, n_rows = 0, max_q_len = 0;
    void *out = nullptr; // row r, head h: out + r * out_stride + h * dv, model dtype
    int64_t out_stride = 0;
    float *raw = nullptr;   // scratch [n_rows, heads * dv]
    float *decay = nullptr; // scratch [n_rows, heads * dk]
    // scratch for cutting long runs into segments that run in parallel (gated_linear_segment_floats); null: never cut
    float *segments = nullptr;
    size_t segment_floats = 0;
};

// Gated delta rule over one packed projection. q, k (kv_heads x dk) and v (heads x dv) pass a causal convolution of `taps` taps
// per channel and silu; q and k become unit vectors x / sqrt(sum x^2 + unit_eps), q times q_scale; head h reads q/k head
// h / (heads / kv_heads). Per head a state S [dk, dv]:
//   S' = diag(g_t) S_{t-1},  u_t = beta_t (v_t - S'^T k_t),  S_t = S' + k_t u_t^T,  o_t = S_t^T q_t
//   beta_t = sigmoid(b_t),  log g_t = -exp(A_log_h) softplus(x_t + dt_bias)
// x_t: one number per head (decay_w null: at a_at of the row), or per head and key channel, decay_w z_t with the `rank` numbers
// z_t at a_at. out_t = rms_norm(o_t, norm) * gate(y_t), y_t heads x dv at `gate`.
struct GatedDeltaArgs {
    const void *proj = nullptr; // [n_rows, row_stride], model dtype
    int64_t row_stride = 0;
    int64_t q_at = 0, k_at = 0, v_at = 0, b_at = 0, a_at = 0;
    const void *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr; // [channels, taps]; the last tap is the current token's
    int32_t taps = 0;
    const void *decay_w = nullptr; // [heads * dk, rank], rows decay_ld apart; null: one decay per head
    int64_t decay_ld = 0;
    const void *a_log = nullptr;   // [heads]
    const void *dt_bias = nullptr; // [heads] or [heads * dk]
    const void *norm_w = nullptr;  // [dv]
    const void *gate = nullptr;    // row r, head h: gate + r * gate_stride + h * dv
    int64_t gate_stride = 0;
    int32_t gate_silu = 0;         // 1: silu(y), 0: sigmoid(y)
    float q_scale = 1.f, eps = 0.f, unit_eps = 1e-6f;
    int32_t heads = 0, kv_heads = 0, dk = 0, dv = 0, rank = 0;
    // slot s: the heads' matrices [heads][dk][dv], then convolution inputs [taps][2 kv_heads dk + heads dv]: position p at
    // p mod taps
    float *state = nullptr;
    int64_t slot_stride = 0;
    // the batch, as in GatedLinearArgs
    const int32_t *seq_ids = nullptr, *q_starts = nullptr, *kv_lens = nullptr;
    int32_t n_seqs = 0, n_rows = 0, max_q_len = 0;
    void *out = nullptr; // row r, head h: out + r * out_stride + h * dv, model dtype
    int64_t out_stride = 0;
    float *scratch = nullptr; // chunk only, 16-byte aligned (gated_delta_scratch_floats)
    size_t scratch_floats = 0;
    float *segments = nullptr; // see gated_delta_segment_floats; null: never cut
    size_t segment_floats = 0;
    LLAISYS_ARGS_FN int32_t channels() const { return 2 * kv_heads * dk + heads * dv; }
};

// minGRU over one packed projection, element by element: with z = sigmoid(z_at .. + bias_z) and u = x_at .. + bias_x,
//   S_t = (1 - z_t) S_{t-1} + z_t g(u_t),  g(u) = u + 1/2 for u >= 0, sigmoid(u) for u < 0;   out_t = S_t silu(g_at ..)
struct MinGruArgs {
    const void *proj = nullptr; // [n_rows, row_stride], model dtype
    int64_t row_stride = 0;
    int64_t z_at = 0, x_at = 0, g_at = 0;
    const void *bias_z = nullptr, *bias_x = nullptr; // [width]
    int32_t width = 0;
    float *state = nullptr; // slot s: state + s * slot_stride, [width]
    int64_t slot_stride = 0;
    // the batch, as in GatedLinearArgs
    const int32_t *seq_ids = nullptr, *q_starts = nullptr, *kv_lens = nullptr;
    int32_t n_seqs = 0, n_rows = 0, max_q_len = 0;
    void *out = nullptr; // row r: out + r * out_stride, model dtype
    int64_t out_stride = 0;
    float *scratch = nullptr; // min_gru_scratch_floats, for runs of more than 128 tokens
    size_t scratch_floats = 0;
};

using stream_t = void *;

} // namespace llaisys::kernels
