/*
 * llaisys C ABI -- Vozozen: a decoder whose layers add up a sliding-window grouped-query attention (no positions) and a gated
 * linear attention of one normed input, then run a squared-relu MLP; a range of the
 * layers may be run several times over, each pass re-mixing the embedding into the stream. The model runs on NVIDIA
 * devices. All other functions are those of model.h.
 *
 * Weight names (llaisysModelLoadTensor): embed, loop.in, final.norm, head and, for layer i, l<i>.norm1, l<i>.norm2,
 * l<i>.mix.left.{q,k,v,q.norm,k.norm,g,o}, l<i>.mix.right.{q,k,v,g,o,norm,a1,a2,a2.b}, l<i>.mlp.{up,down}.
 */
#ifndef LLAISYS_MODELS_VOZOZEN_H
#define LLAISYS_MODELS_VOZOZEN_H

#include "model.h"

#ifdef __cplusplus
extern "C" {
#endif

/* Sliding-window attention: `heads` query heads share kv_heads key/value heads; window counts the query's own token. */
struct LlaisysWindowAttentionMeta {
    size_t heads, kv_heads, dim, vdim, window;
    float scale;
};

/* Gated linear attention: state [dim, vdim] per head, decay sigmoid(z)^(1/tau) per key channel from a rank-`rank` projection. */
struct LlaisysGatedLinearMeta {
    size_t heads, dim, vdim, rank;
    float tau;
};

struct LlaisysVozozenLayerMeta {
    struct LlaisysWindowAttentionMeta left;
    struct LlaisysGatedLinearMeta right;
    float left_scale, right_scale;
    size_t ff; /* 0 = no feed-forward */
};

struct LlaisysVozozenMeta {
    llaisysDataType_t dtype; /* of matrix products and activations: BF16, F16 or F32 */
    size_t nlayer;
    const struct LlaisysVozozenLayerMeta *layers;
    size_t width, voc, maxseq;
    float embed_scale, eps, logit_softcap; /* softcap 0 = none */
    /* layers [loop_start, loop_stop) run loop_times times in a row; loop_times 0 = no loop (and no loop.in) */
    size_t loop_start, loop_stop, loop_times;
    int64_t end_token;
};

/* NULL on failure (message on stderr and in llaisysGetLastError). */
LLAISYS_API struct LlaisysModel *llaisysVozozenModelCreate(const struct LlaisysVozozenMeta *meta, llaisysDeviceType_t device,
                                                           int device_id);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MODELS_VOZOZEN_H */
