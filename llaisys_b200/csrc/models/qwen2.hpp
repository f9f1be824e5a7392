// Qwen2 decoder (RMSNorm, GQA attention with q/k/v biases and half-split RoPE, SwiGLU MLP, untied output embedding)
// on the library's operators and the paged KV cache. The reference declares this model's C API and leaves it
// unimplemented (include/llaisys/models/qwen2.h:7-40; python/llaisys/models/qwen2.py:11-33 is a stub).
#pragma once

#include "../comm/collective.hpp"
#include "decoder.hpp"
#include "llaisys/models/qwen2.h"

#include <memory>
#include <vector>

namespace llaisys::models {

class Qwen2 : public Decoder {
public:
    // tp_rank / tp_world: tensor parallelism by heads. Rank r holds query heads [r nh/W, (r+1) nh/W), the KV heads they
    // use, and rows [r di/W, (r+1) di/W) of the MLP; the output and down projections produce partial sums that one
    // all-reduce each turns into the full activation (set the collective before the first step). Embeddings, norms and
    // the vocabulary projection are replicated, so every rank computes the same logits and tokens.
    Qwen2(const LlaisysQwen2Meta &meta, llaisysDeviceType_t device, int device_id, int tp_rank = 0, int tp_world = 1);
    void setCollective(std::unique_ptr<comm::Collective> c);
    int tpRank() const { return _tp_rank; }
    int tpWorld() const { return _tp_world; }
    ~Qwen2() override;

    LlaisysQwen2Weights *weights() { return &_weights; }
    const LlaisysQwen2Meta &meta() const { return _meta; } // this rank's share: nh, nkvh and di are per-rank under TP

    size_t vocab() const override { return _meta.voc; }
    size_t maxSeq() const override { return _meta.maxseq; }
    int64_t endToken() const override { return _meta.end_token; }

private:
    // q|k|v and gate|up live packed in one matrix each (one projection launch instead of three / two); the handles the
    // caller loads through are row slices of the packed tensors
    struct Layer {
        const std::byte *attn_norm, *qkv_w, *qkv_b, *o_w, *mlp_norm, *gate_up_w, *down_w;
    };
    llaisysTensor_t wrap(tensor_t t);
    llaisysTensor_t makeWeight(const std::vector<size_t> &shape);
    std::vector<Layer> layerPointers() const;
    kv::PagedKVConfig cacheShape() const override;
    void ensureActivations(size_t n_tokens, size_t n_out) override;
    void forward(const StepArrays &a, const StepShape &s) override;
    bool graphable() const override { return _tp_world == 1; }

    // operator shims: CPU loops or CUDA launches on the runtime stream, on raw device pointers
    void opEmbedding(void *out, const int64_t *idx, const void *w, size_t n, size_t d, size_t vocab);
    void opLinear(void *out, const void *in, const void *w, size_t m, size_t n, size_t k, bool accumulate = false);
    void opRmsNorm(void *out, const void *in, const void *w, size_t rows, size_t d);
    void opSwigluPacked(void *out, const void *gate_up, size_t rows, size_t di);
    void opAdd(void *c, const void *a, const void *b, size_t n);
    // x += in . w^T, through an all-reduce of the partial product when the model is sharded
    void projectIntoStream(void *x, void *tmp, const void *in, const void *w, size_t m, size_t n, size_t k);
    void opArgmax(int64_t *idx, const void *vals, size_t rows, size_t n);

    LlaisysQwen2Meta _meta; // per-rank dimensions
    int _tp_rank = 0, _tp_world = 1;
    std::unique_ptr<comm::Collective> _tp;

    LlaisysQwen2Weights _weights{};
    std::vector<llaisysTensor_t> _all_weights; // owns every handle in _weights
    std::vector<llaisysTensor_t> _per_layer[12];
    std::vector<tensor_t> _qkv_w, _qkv_b, _gate_up_w; // packed per-layer matrices behind the q/k/v and gate/up handles

    core::storage_t _x, _h, _qkv, _q, _attn, _gate_up, _act, _x_last;
};

} // namespace llaisys::models
