/*
 * llaisys C ABI -- Lilovik: a decoder with norms before and after each sublayer. A layer's mixer is either grouped-query attention
 * without a softmax -- q and k normed over all their heads at once, a query factor that grows with the position, capped scores with a
 * penalty on distance, sigmoid weights mixed over the heads -- or a minGRU; a layer may lack its feed-forward (a gated relu). The
 * embedding adds sines and cosines of the position. The model runs on NVIDIA devices. All other functions are those of model.h.
 *
 * Weight names (llaisysModelLoadTensor): embed, final.norm, head and, for layer i, l<i>.norm1, l<i>.norm1b; attention:
 * l<i>.mix.{q,q.b,k,k.b,v,v.b,q.norm,k.norm,talk,pb,o}; minGRU: l<i>.mix.{z,z.b,x,x.b,g,o}; with a feed-forward l<i>.norm2,
 * l<i>.norm2b, l<i>.mlp.{gate,up,down}. Norms of the stream are stored around zero, q.norm and k.norm around one.
 */
#ifndef LLAISYS_MODELS_LILOVIK_H
#define LLAISYS_MODELS_LILOVIK_H

#include "model.h"

#ifdef __cplusplus
extern "C" {
#endif

/* See LlaisysGates and the row form of LlaisysNormAppend in mixers.h; head h takes 2^(-8 (h + 1) / heads) per token of distance off a
 * score. softcap <= 0: no cap; temp_coef 0: no query factor. */
struct LlaisysGatesAttentionMeta {
    size_t heads, kv_heads, dim, vdim;
    float scale, softcap, temp_coef, temp_every;
};

struct LlaisysLilovikLayerMeta {
    int recurrent; /* 1: minGRU of gru_width channels; 0: attention */
    struct LlaisysGatesAttentionMeta attn;
    size_t gru_width;
    size_t ff; /* 0 = no feed-forward */
};

struct LlaisysLilovikMeta {
    llaisysDataType_t dtype; /* of matrix products and activations: BF16, F16 or F32 */
    size_t nlayer;
    const struct LlaisysLilovikLayerMeta *layers;
    size_t width, voc, maxseq;
    float eps, logit_scale;
    int64_t end_token;
};

/* NULL on failure (message on stderr and in llaisysGetLastError). */
LLAISYS_API struct LlaisysModel *llaisysLilovikModelCreate(const struct LlaisysLilovikMeta *meta, llaisysDeviceType_t device,
                                                           int device_id);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MODELS_LILOVIK_H */
