// Doderax decoder. A layer norms the stream once and adds both its sublayers' readings of it: x += mixer(h) + W_down gelu(W_up h).
// The mixer is a gated delta rule (decay per key channel, low-rank gates), or attention with rotary positions, a sliding window
// and kept first tokens beside a gated delta rule with one decay per head, each output normed, averaged. The stream x is f32.
//
// What a layer launches: norm, ONE projection for everything that reads h (both mixers and the MLP's up matrix), the delta rule
// (writing its gated heads into their columns of the mix buffer), gelu into the MLP's columns, and ONE output projection over
// all columns accumulated into the stream. Side by side: [rotation + append] and attention besides, an output projection per
// mixer, and one kernel that norms and adds both into the stream and norms that for the next layer.
#pragma once

#include "llaisys/models/doderax.h"
#include "stream_decoder.hpp"

#include <vector>

namespace llaisys::models {

class Doderax : public StreamDecoder {
public:
    Doderax(const LlaisysDoderaxMeta &meta, llaisysDeviceType_t device, int device_id);

    size_t vocab() const override { return _meta.voc; }
    size_t maxSeq() const override { return _meta.maxseq; }
    int64_t endToken() const override { return _meta.end_token; }

private:
    struct Layer {
        LlaisysDoderaxLayerMeta meta;
        std::byte *norm1, *proj;
        std::byte *conv_q, *conv_k, *conv_v, *a_log, *dt_bias, *decay_w, *gate_w, *head_norm;
        std::byte *out;                                  // over the whole mix buffer (delta rule alone)
        std::byte *out_left, *out_right, *left_norm, *right_norm, *down; // side by side
        // first row of each part in the packed projection, parts padded to 8 rows; n_proj rows in all
        size_t aq, ak, av, q, k, v, b, a, g, up, n_proj;
        size_t right, ff, n_mix; // first columns of the delta rule and of the MLP in the mix buffer, columns in all
        size_t kv_layer = 0, rotary = 0; // side by side: layer of the cache, entry of _rotary
    };
    struct Rotary { // one per (base, dims) in use
        double base;
        size_t dims;
        core::storage_t freq, table;
    };

    kv::PagedKVConfig cacheShape() const override;
    std::vector<size_t> stateShape() const override;
    void ensureActivations(size_t n_tokens, size_t n_out) override;
    void forward(const StepArrays &a, const StepShape &s) override;
    void delta(size_t layer, const StepArrays &a, const StepShape &s);
    void attention(const Layer &l, const StepArrays &a, const StepShape &s);
    size_t rotary(double base, size_t dims);

    LlaisysDoderaxMeta _meta;
    std::vector<Layer> _layers;
    std::vector<Rotary> _rotary;
    std::byte *_embed = nullptr, *_pairs = nullptr, *_final_norm = nullptr, *_head = nullptr;

    core::storage_t _x, _h, _proj, _gate, _q, _mix, _left, _right, _scratch, _segments, _h_out;
};

} // namespace llaisys::models
