/*
 * llaisys C ABI -- what every decoder-only model of the library can do, whatever its network: batched sequences over a
 * paged cache (and recurrent state, where the network has it), mixed prefill / decode steps, a device-resident decode
 * loop, logits. No counterpart in the reference, which declares one model family (reference:
 * include/llaisys/models/qwen2.h:7-40).
 *
 * A family's create function returns its handle; a struct LlaisysQwen2Model * may be passed, cast, wherever a
 * struct LlaisysModel * is expected (the functions of models/qwen2.h named alike do the same thing). Status codes as in
 * paged_kv.h.
 */
#ifndef LLAISYS_MODELS_MODEL_H
#define LLAISYS_MODELS_MODEL_H

#include "../tensor.h"

#ifdef __cplusplus
extern "C" {
#endif

struct LlaisysModel;

LLAISYS_API void llaisysModelDestroy(struct LlaisysModel *model);
LLAISYS_API size_t llaisysModelVocab(struct LlaisysModel *model);
/* Copies one checkpoint tensor (host memory, LLAISYS_DTYPE_BF16 or F32, row-major) into the weight of that name.
 * *known_out = 0 when the model has no weight of that name (nothing is copied). For families whose weights are named;
 * LLAISYS_E_UNSUPPORTED where they are loaded through handles (Qwen2). */
LLAISYS_API int llaisysModelLoadTensor(struct LlaisysModel *model, const char *name, llaisysDataType_t dtype,
                                       const size_t *shape, size_t ndim, const void *data, int *known_out);
/* Weights still to be loaded: returns how many, and the first one's name in name_out (at most cap bytes with the end). */
LLAISYS_API size_t llaisysModelMissingTensors(struct LlaisysModel *model, char *name_out, size_t cap);
/* Sizes the cache: at most max_seqs live sequences of at most max_tokens tokens each. pool_tokens: tokens all live
 * sequences together can hold, in whole pages of 16; 0 = max_seqs * max_tokens. */
LLAISYS_API int llaisysModelConfigureCache(struct LlaisysModel *model, size_t max_seqs, size_t max_tokens, size_t pool_tokens);
LLAISYS_API int llaisysModelSeqAdd(struct LlaisysModel *model, int32_t *seq_out);
/* See llaisysQwen2ModelSeqAddWithPrefix. A model with recurrent state never matches a prefix (*matched_out = 0). */
LLAISYS_API int llaisysModelSeqAddWithPrefix(struct LlaisysModel *model, const int64_t *tokens, size_t n, int32_t *seq_out,
                                             size_t *matched_out);
LLAISYS_API int llaisysModelSeqFree(struct LlaisysModel *model, int32_t seq);
LLAISYS_API size_t llaisysModelFreePages(struct LlaisysModel *model);
/* One implicit sequence: appends the tokens and writes the greedy next token; Reset forgets the sequence. */
LLAISYS_API int llaisysModelInfer(struct LlaisysModel *model, const int64_t *tokens, size_t n, int64_t *next_out);
LLAISYS_API int llaisysModelReset(struct LlaisysModel *model);
/* Appends n_tokens[i] new tokens (packed back to back, host int64) to sequence seq_ids[i]; next_out[n_seqs] = the greedy
 * next token of every sequence. Any mix of chunk lengths >= 1. */
LLAISYS_API int llaisysModelStep(struct LlaisysModel *model, const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs,
                                 const int64_t *tokens, int64_t *next_out);
/* The same step with logits and greedy tokens at chosen rows of the packed tokens (rows[n_rows], any order; none = the
 * vocabulary projection is skipped) instead of at every sequence's last token: next_out[n_rows],
 * llaisysModelLastLogits gives [n_rows][vocab]. */
LLAISYS_API int llaisysModelStepRows(struct LlaisysModel *model, const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs,
                                     const int64_t *tokens, const int32_t *rows, size_t n_rows, int64_t *next_out);
/* See llaisysQwen2ModelDecodeLoop, ...LastLogits, ...LastLoopMs. */
LLAISYS_API int llaisysModelDecodeLoop(struct LlaisysModel *model, const int32_t *seq_ids, size_t n_seqs,
                                       const int64_t *first_tokens, size_t n_steps, int64_t *tokens_out);
LLAISYS_API int llaisysModelLastLogits(struct LlaisysModel *model, float *out_host, size_t capacity_floats);
LLAISYS_API double llaisysModelLastLoopMs(struct LlaisysModel *model);

/* Development aid, for models with an f32 residual stream: copies the stream after every layer run of the next steps to host
 * memory, [runs, rows, width]. Takes effect until called again; LLAISYS_E_INVALID from LayerStream when the last step was not
 * recorded. */
LLAISYS_API int llaisysModelRecordStream(struct LlaisysModel *model, int enable);
LLAISYS_API int llaisysModelLayerStream(struct LlaisysModel *model, float *out_host, size_t capacity_floats, size_t *floats_out);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MODELS_MODEL_H */
