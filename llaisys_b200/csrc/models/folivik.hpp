// Folivik decoder: x += mixer(norm(x)), x += experts(norm(x)). The mixer is attention over latents, sliding-window attention with a
// logarithmic distance penalty, or a Mamba-2 state space; the feed-forward is a mixture of experts (or none). The stream x is f32.
//
// What a layer launches: ONE projection for all that reads h, the mixer, the output projection accumulated into the stream, the norm;
// then the router's product, the choice, the placing of rows, two products over the experts' rows, the shared expert (accumulated
// into the stream), and one kernel for the weighted sum, the residual and the norm of the next layer.
//
// Latent attention caches one row per token, [latent | turned key part], for all heads. The unrotated query is multiplied into the
// latent's space (W_uk of its head), attention runs over the rows as they are, and W_uv of each head follows. For long chunks that
// is more arithmetic than making keys and values of the contexts' rows once and running ordinary attention over them: chunks of at
// least kExpandFrom tokens do so, a pass over neighbouring sequences at a time.
#pragma once

#include "llaisys/models/folivik.h"
#include "stream_decoder.hpp"

#include <vector>

namespace llaisys::models {

class Folivik : public StreamDecoder {
public:
    Folivik(const LlaisysFolivikMeta &meta, llaisysDeviceType_t device, int device_id);

    size_t vocab() const override { return _meta.voc; }
    size_t maxSeq() const override { return _meta.maxseq; }
    int64_t endToken() const override { return _meta.end_token; }

private:
    struct Layer {
        LlaisysFolivikLayerMeta meta;
        float *norm1, *norm2;
        std::byte *proj, *out;
        size_t at[3], n_proj;                          // first row of each part of the projection, parts padded to 8 rows; rows in all
        size_t n_mix;                                  // columns of the mixer's output, padded to 8
        size_t index;                                  // layer of the cache, or of the state
        std::byte *q_norm, *k_norm;                    // both kinds of attention
        std::byte *uq, *uk, *uv;                       // latent attention
        size_t rotary, q_rank;                         // q_rank: padded columns of uq
        float *temp, *fade_a, *fade_b;                 // windowed attention
        std::byte *conv_w, *conv_b, *norm_w;           // state space
        float *a_log, *dt_bias, *d_skip;
        std::byte *router, *gate_up, *down, *shared_gate_up, *shared_down;
        float *correction;
        size_t ff, shared_ff;                          // padded
    };
    struct Rotary {
        double base;
        size_t dims;
        core::storage_t freq; // f64 [dims / 2]
        core::storage_t table; // of the step's rows
    };

    // Neighbouring sequences [from, to) of a step that are served alike, their rows, and for expanded ones the rows of their contexts
    struct LatentRange {
        bool expanded;
        size_t from, to, row, n_rows, max_q_len, max_kv_len, tokens;
    };

    kv::PagedKVConfig cacheShape() const override;
    std::vector<size_t> stateShape() const override;
    void ensureActivations(size_t n_tokens, size_t n_out) override;
    void forward(const StepArrays &a, const StepShape &s) override;
    void latentAttention(const Layer &l, const StepArrays &a, const StepShape &s);
    void latentRange(const Layer &l, const StepArrays &a, const StepShape &s, const LatentRange &r);
    void expandedRange(const Layer &l, const StepArrays &a, const StepShape &s, const LatentRange &r);
    void planLatents(const StepShape &s);
    void windowAttention(const Layer &l, const StepArrays &a, const StepShape &s);
    void stateSpace(const Layer &l, const StepArrays &a, const StepShape &s);
    void experts(const Layer &l, const StepShape &s, const float *next_gain);
    size_t rotary(double base, size_t dims); // index of the rotation, added when new

    LlaisysFolivikMeta _meta;
    std::vector<Layer> _layers;
    std::vector<Rotary> _rotary;
    std::byte *_embed = nullptr, *_head = nullptr;
    float *_final_norm = nullptr;

    core::storage_t _x, _h, _proj, _q, _q_wide, _latent, _scale, _mix, _scratch, _segments, _h_out;
    std::vector<LatentRange> _ranges; // of the current step
    std::vector<int32_t> _page_starts_host;
    core::storage_t _page_starts, _context, _keys, _values; // expanded: context rows, keys and values made of them
    core::storage_t _logits_e, _choice, _counts, _rows, _act, _expert_out, _shared; // experts
};

} // namespace llaisys::models
