/*
 * llaisys C ABI -- Doderax: a decoder whose layers add a token mixer and an MLP of one normed input to the stream. A mixer is
 * either a gated delta rule with a decay per key channel, or two mixers side by side -- sliding-window grouped-query attention
 * with rotary positions that keeps a sequence's first tokens, and a gated delta rule with one decay per head -- each normed over
 * the width, averaged. The embedding adds a row chosen by the hashed pair of the previous and the current token. The model runs
 * on NVIDIA devices. All other functions are those of model.h.
 *
 * Weight names (llaisysModelLoadTensor): embed, bigram, final.norm, head and, for layer i, l<i>.norm1, l<i>.mlp.{up,down};
 * delta rule with a decay per channel: l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,A_log,norm,a1,a2,dt_bias,g1,g2,o}; side by side:
 * l<i>.mix.left.{q,k,v,o,out}, l<i>.mix.right.{q,q.conv,k,k.conv,v,v.conv,b,A_log,norm,a,dt_bias,g,o,out}. Norms of the stream
 * (norm1, final.norm) are stored around zero, all others around one.
 */
#ifndef LLAISYS_MODELS_DODERAX_H
#define LLAISYS_MODELS_DODERAX_H

#include "model.h"

#ifdef __cplusplus
extern "C" {
#endif

/* Gated delta rule (see LlaisysGatedDelta in mixers.h): `heads` heads of values share kv_heads heads of queries and keys.
 * decay_rank 0: one decay per head; else one per key channel from a projection of that rank. gate_rank 0: output gate silu(W h);
 * else sigmoid of a projection of that rank. */
struct LlaisysDeltaMixerMeta {
    size_t heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank;
};

/* Attention of `heads` query heads over kv_heads key/value heads. The query at position i sees keys j <= i with i - j < window or
 * j < keep_first. The first rot_dims dims of q and k turn with their position (dim i with dim i + rot_dims / 2, frequency
 * rot_base^(-2 i / rot_dims)). */
struct LlaisysSinkAttentionMeta {
    size_t heads, kv_heads, dim, vdim, window, keep_first, rot_dims;
    double rot_base;
    float scale;
};

struct LlaisysDoderaxLayerMeta {
    int parallel; /* 1: attn beside delta; 0: delta alone */
    struct LlaisysSinkAttentionMeta attn;
    struct LlaisysDeltaMixerMeta delta;
    size_t ff; /* 0 = no feed-forward */
};

struct LlaisysDoderaxMeta {
    llaisysDataType_t dtype; /* of matrix products and activations: BF16, F16 or F32 */
    size_t nlayer;
    const struct LlaisysDoderaxLayerMeta *layers;
    size_t width, voc, maxseq;
    /* row (previous * pair_mul_prev + current * pair_mul_cur) mod pair_buckets of `bigram`, row pair_buckets for a sequence's
     * first token; pair_buckets 0 = no such table */
    size_t pair_buckets;
    int64_t pair_mul_prev, pair_mul_cur;
    float eps, logit_scale;
    int64_t end_token;
};

/* NULL on failure (message on stderr and in llaisysGetLastError). */
LLAISYS_API struct LlaisysModel *llaisysDoderaxModelCreate(const struct LlaisysDoderaxMeta *meta, llaisysDeviceType_t device,
                                                           int device_id);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MODELS_DODERAX_H */
