/*
 * llaisys C ABI -- Folivik: a decoder whose layers mix tokens by one of three mixers -- attention over latents, sliding-window
 * grouped-query attention with a penalty that grows with the logarithm of the distance, or a Mamba-2 state space -- and then pass a
 * mixture of experts with identity experts and a shared one. Every sublayer norms the stream before it reads it. The model runs on
 * NVIDIA devices. All other functions are those of model.h.
 *
 * Weight names (llaisysModelLoadTensor): embed, final.norm, head and, for layer i, l<i>.norm1, l<i>.norm2 (stream norms: one number
 * each); latent attention: l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}; windowed attention: l<i>.mix.{q,k,v,q.norm,k.norm,temp,r1,
 * r2,o}; state space: l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}; experts: l<i>.mlp.{router,correction}, l<i>.mlp.e<j>.{gate,up,
 * down}, l<i>.mlp.shared.{gate,up,down}.
 */
#ifndef LLAISYS_MODELS_FOLIVIK_H
#define LLAISYS_MODELS_FOLIVIK_H

#include "model.h"

#ifdef __cplusplus
extern "C" {
#endif

/* c_q = norm(W_dq h) [q_rank], per head (u, w) = W_uq c_q with w turned by the position; c = norm(first kv_rank rows of W_dkv h),
 * z = the last rot_dim rows turned, shared by all heads; key (W_uk c, z), value W_uv c, score scale * ((u, w) . key), all earlier keys;
 * a head's output is multiplied by sigmoid(W_g h). Dims 2 i and 2 i + 1 turn by position * rot_base^(-2 i / rot_dim). */
struct LlaisysLatentAttentionMeta {
    size_t heads, dim, rot_dim, vdim, q_rank, kv_rank;
    double rot_base;
    float scale;
};

/* q and k normed per head; score temp_h * scale * (q . k) - r1_h ln(1 + r2_h (i - j)) for keys 0 <= i - j < window. */
struct LlaisysFadingAttentionMeta {
    size_t heads, kv_heads, dim, vdim, window;
    float scale;
};

/* See LlaisysStateSpace in mixers.h. */
struct LlaisysStateSpaceMixerMeta {
    size_t heads, groups, state, vdim, taps, norm_groups;
};

/* See LlaisysExperts in mixers.h. top = 0: the layer has no feed-forward; groups = 1: no groups; shared_ff = 0: no shared expert. */
struct LlaisysExpertLayerMeta {
    size_t experts, identity, top, groups, keep, ff, shared_ff;
    float scale;
};

enum { LLAISYS_FOLIVIK_LATENT = 0, LLAISYS_FOLIVIK_ATTENTION = 1, LLAISYS_FOLIVIK_STATE_SPACE = 2 };

struct LlaisysFolivikLayerMeta {
    int mixer; /* LLAISYS_FOLIVIK_...: which of the next three counts */
    struct LlaisysLatentAttentionMeta latent;
    struct LlaisysFadingAttentionMeta attn;
    struct LlaisysStateSpaceMixerMeta ssm;
    struct LlaisysExpertLayerMeta mlp;
};

struct LlaisysFolivikMeta {
    llaisysDataType_t dtype; /* of matrix products and activations: BF16, F16 or F32 */
    size_t nlayer;
    const struct LlaisysFolivikLayerMeta *layers;
    size_t width, voc, maxseq;
    float eps;
    int64_t end_token;
};

/* NULL on failure (message on stderr and in llaisysGetLastError). */
LLAISYS_API struct LlaisysModel *llaisysFolivikModelCreate(const struct LlaisysFolivikMeta *meta, llaisysDeviceType_t device,
                                                           int device_id);

#ifdef __cplusplus
}
#endif
#endif /* LLAISYS_MODELS_FOLIVIK_H */
