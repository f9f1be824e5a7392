// Lilovik decoder. Both sublayers of a layer norm the stream before and their output after: x += norm(mixer(norm(x))), then
// x += norm(W_down (relu(W_gate h) W_up h)), h = norm(x). The mixer is attention without a softmax whose weights are mixed over the
// heads, or a minGRU. The embedding adds sines and cosines of the position. The stream x is f32.
//
// What a sublayer launches: ONE projection for all that reads h, the mixer ([row norm + query factor + append] and attention, or the
// recurrence) or the gated relu, the output projection (f32, because a norm follows) and one kernel for that norm, the residual sum
// and the norm of the next sublayer.
#pragma once

#include "llaisys/models/lilovik.h"
#include "stream_decoder.hpp"

#include <vector>

namespace llaisys::models {

class Lilovik : public StreamDecoder {
public:
    Lilovik(const LlaisysLilovikMeta &meta, llaisysDeviceType_t device, int device_id);

    size_t vocab() const override { return _meta.voc; }
    size_t maxSeq() const override { return _meta.maxseq; }
    int64_t endToken() const override { return _meta.end_token; }

private:
    struct Layer {
        LlaisysLilovikLayerMeta meta;
        std::byte *norm1, *norm1b, *norm2, *norm2b;
        std::byte *proj, *bias, *out;              // bias: of every row of the projection (zero where it has none)
        std::byte *q_norm, *k_norm, *talk, *score_bias;
        std::byte *gate_up, *down;
        size_t at[3], n_proj;    // first row of q, k, v or z, x, g in the projection, parts padded to 8 rows; rows in all
        size_t n_mix, ff;        // columns of the mixer's output and of the feed-forward, padded to 8
        size_t index;            // among the layers of its type: layer of the cache, or of the state
        core::storage_t slopes;
    };

    kv::PagedKVConfig cacheShape() const override;
    std::vector<size_t> stateShape() const override;
    void ensureActivations(size_t n_tokens, size_t n_out) override;
    void forward(const StepArrays &a, const StepShape &s) override;
    void attention(const Layer &l, const StepArrays &a, const StepShape &s);
    void recurrence(const Layer &l, const StepArrays &a, const StepShape &s);

    LlaisysLilovikMeta _meta;
    std::vector<Layer> _layers;
    std::byte *_embed = nullptr, *_final_norm = nullptr, *_head = nullptr;
    core::storage_t _freq; // f64, of the position vectors

    core::storage_t _x, _y, _h, _proj, _q, _mix, _u, _scratch, _h_out;
};

} // namespace llaisys::models
