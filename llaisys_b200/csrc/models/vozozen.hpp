// Vozozen decoder. A layer is pre-norm: x += mixer(norm1(x)), x += W_down relu(W_up norm2(x))^2. The mixer runs two head
// groups side by side on the same input -- sliding-window grouped-query attention with normed q / k, no positions and a
// sigmoid gate per head, and gated linear attention with a decay per key channel -- and adds the two outputs with a factor
// each. A range of layers may run several passes with the same weights; every pass has its own cache and state and starts
// from W_in [x; x0], x0 being the embedding output. The stream x is f32; logits go through a soft cap.
//
// What a layer launches: norm, ONE projection for everything both mixers read, [q/k norm + append + gates], the attention
// (writing its gated heads into the left columns of the mix buffer), the linear attention (the right columns), ONE output
// projection over both sides accumulated into the stream, norm, up, activation, down accumulated into the stream.
#pragma once

#include "stream_decoder.hpp"
#include "llaisys/models/vozozen.h"

#include <vector>

namespace llaisys::models {

class Vozozen : public StreamDecoder {
public:
    Vozozen(const LlaisysVozozenMeta &meta, llaisysDeviceType_t device, int device_id);

    size_t vocab() const override { return _meta.voc; }
    size_t maxSeq() const override { return _meta.maxseq; }
    int64_t endToken() const override { return _meta.end_token; }

private:
    kv::PagedKVConfig cacheShape() const override;
    std::vector<size_t> stateShape() const override;
    void ensureActivations(size_t n_tokens, size_t n_out) override;
    void forward(const StepArrays &a, const StepShape &s) override;

    struct Layer {
        LlaisysVozozenLayerMeta meta;
        std::byte *norm1, *norm2, *proj, *out, *up, *down, *q_norm, *k_norm, *decay_w, *decay_b, *gla_norm;
        // first row of each part in the packed projection, parts padded to 8 rows; `n_proj` rows in all
        size_t q, k, v, rq, rk, rv, rg, z, g, n_proj;
        size_t right, n_mix; // first column of the right mixer in the mix buffer, columns in all (padded to 8)
    };

    LlaisysVozozenMeta _meta;
    std::vector<Layer> _layers;
    std::vector<size_t> _runs;       // layer of every run, in order
    std::vector<bool> _starts_pass;  // run r is the first of a pass
    std::byte *_embed = nullptr, *_loop_in = nullptr, *_final_norm = nullptr, *_head = nullptr;

    core::storage_t _x, _pass_in, _h, _proj, _q, _row_scale, _mix, _raw, _decay, _segments, _u, _h_out;
};

} // namespace llaisys::models
