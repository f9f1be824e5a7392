#include "vozozen.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <algorithm>
#include <cmath>
#include <cstring>

namespace llaisys::models {

// ---- construction -------------------------------------------------------------------------------------------------------

Vozozen::Vozozen(const LlaisysVozozenMeta &meta, llaisysDeviceType_t device, int device_id)
    : StreamDecoder("vozozen", device, device_id, meta.dtype), _meta(meta) {
    if (meta.nlayer == 0 || meta.layers == nullptr || meta.width == 0 || meta.voc == 0) {
        failModel(LLAISYS_E_INVALID, "inconsistent model dimensions");
    }
    const size_t W = meta.width, L = meta.nlayer;
    const bool loop = meta.loop_times > 0;
    if (loop && (meta.loop_start >= meta.loop_stop || meta.loop_stop > L)) {
        failModel(LLAISYS_E_INVALID, "the looped layers are not a range of the model's layers");
    }
    for (size_t i = 0; i < L; ++i) {
        const LlaisysVozozenLayerMeta &m = meta.layers[i];
        const LlaisysWindowAttentionMeta &l = m.left;
        const LlaisysGatedLinearMeta &r = m.right;
        if (l.heads == 0 || l.kv_heads == 0 || l.heads % l.kv_heads != 0 || l.dim == 0 || l.vdim == 0 || l.window == 0 ||
            r.heads == 0 || r.dim == 0 || r.vdim == 0 || r.rank == 0 || !(r.tau > 0.f)) {
            failModel(LLAISYS_E_INVALID, "layer " + std::to_string(i) + ": inconsistent mixer sizes");
        }
    }
    enter();

    // ---- weights ----
    _embed = matrix(meta.voc, W);
    place("embed", _embed, 0, 0, meta.voc, W, W);
    if (loop) {
        _loop_in = matrix(W, 2 * W);
        place("loop.in", _loop_in, 0, 0, W, 2 * W, 2 * W);
    }
    for (size_t i = 0; i < L; ++i) {
        Layer l{};
        l.meta = meta.layers[i];
        const LlaisysWindowAttentionMeta &a = l.meta.left;
        const LlaisysGatedLinearMeta &r = l.meta.right;
        const std::string p = "l" + std::to_string(i) + ".", ml = p + "mix.left.", mr = p + "mix.right.";
        size_t rows = 0;
        struct Part {
            std::string name;
            size_t *at, rows;
        };
        const Part parts[] = {{ml + "q", &l.q, a.heads * a.dim},     {ml + "k", &l.k, a.kv_heads * a.dim},
                              {ml + "v", &l.v, a.kv_heads * a.vdim}, {mr + "q", &l.rq, r.heads * r.dim},
                              {mr + "k", &l.rk, r.heads * r.dim},    {mr + "v", &l.rv, r.heads * r.vdim},
                              {mr + "g", &l.rg, r.heads * r.vdim},   {mr + "a1", &l.z, r.rank},
                              {ml + "g", &l.g, a.heads}};
        for (const Part &part : parts) {
            *part.at = rows;
            rows += pad8(part.rows);
        }
        l.n_proj = rows;
        l.proj = matrix(rows, W);
        for (const Part &part : parts) {
            place(part.name, l.proj, *part.at, 0, part.rows, W, W);
        }
        // both output projections side by side: one product over [left heads | right heads]
        l.right = pad8(a.heads * a.vdim);
        l.n_mix = l.right + pad8(r.heads * r.vdim);
        l.out = matrix(W, l.n_mix);
        place(ml + "o", l.out, 0, 0, W, a.heads * a.vdim, l.n_mix);
        place(mr + "o", l.out, 0, l.right, W, r.heads * r.vdim, l.n_mix);
        l.norm1 = vector(p + "norm1", W);
        l.q_norm = vector(ml + "q.norm", a.dim);
        l.k_norm = vector(ml + "k.norm", a.dim);
        l.decay_w = matrix(r.heads * r.dim, r.rank);
        place(mr + "a2", l.decay_w, 0, 0, r.heads * r.dim, r.rank, r.rank);
        l.decay_b = vector(mr + "a2.b", r.heads * r.dim);
        l.gla_norm = vector(mr + "norm", r.vdim);
        if (l.meta.ff != 0) {
            l.norm2 = vector(p + "norm2", W);
            l.up = matrix(l.meta.ff, W);
            place(p + "mlp.up", l.up, 0, 0, l.meta.ff, W, W);
            l.down = matrix(W, l.meta.ff);
            place(p + "mlp.down", l.down, 0, 0, W, l.meta.ff, l.meta.ff);
        }
        _layers.push_back(l);
    }
    _final_norm = vector("final.norm", W);
    _head = matrix(meta.voc, W);
    place("head", _head, 0, 0, meta.voc, W, W);
    _meta.layers = nullptr; // the caller's array; every layer keeps its own copy

    // ---- order of runs ----
    auto run = [&](size_t layer, bool starts_pass) {
        _runs.push_back(layer);
        _starts_pass.push_back(starts_pass);
    };
    const size_t start = loop ? meta.loop_start : L, stop = loop ? meta.loop_stop : L;
    for (size_t i = 0; i < start; ++i) {
        run(i, false);
    }
    for (size_t t = 0; t < meta.loop_times; ++t) {
        for (size_t i = start; i < stop; ++i) {
            run(i, i == start);
        }
    }
    for (size_t i = stop; i < L; ++i) {
        run(i, false);
    }
}

// ---- cache, state, workspace ------------------------------------------------------------------------------------------------

kv::PagedKVConfig Vozozen::cacheShape() const {
    kv::PagedKVConfig cfg;
    cfg.nlayer = _runs.size(); // every run of a looped layer has K/V (and state) of its own
    for (size_t layer : _runs) {
        const LlaisysWindowAttentionMeta &a = _layers[layer].meta.left;
        cfg.layers.push_back(kv::KVLayerShape{a.kv_heads, a.dim, a.vdim});
    }
    return cfg;
}

std::vector<size_t> Vozozen::stateShape() const {
    std::vector<size_t> floats;
    for (size_t layer : _runs) {
        const LlaisysGatedLinearMeta &r = _layers[layer].meta.right;
        floats.push_back(r.heads * r.dim * r.vdim);
    }
    return floats;
}

void Vozozen::ensureActivations(size_t n_tokens, size_t n_out) {
    auto &rt = enter();
    const size_t W = _meta.width;
    if (n_tokens > _ws_tokens) {
        ++_generation;
        size_t proj = 0, q = 0, heads = 0, mix = 0, raw = 0, decay = 0, ff = 0, segments = 0;
        for (const Layer &l : _layers) {
            proj = std::max(proj, l.n_proj);
            q = std::max(q, l.meta.left.heads * l.meta.left.dim);
            heads = std::max(heads, l.meta.left.heads);
            mix = std::max(mix, l.n_mix);
            raw = std::max(raw, l.meta.right.heads * l.meta.right.vdim);
            decay = std::max(decay, l.meta.right.heads * l.meta.right.dim);
            ff = std::max(ff, l.meta.ff);
#ifdef ENABLE_NVIDIA_API
            segments = std::max(segments, kernels::gated_linear_segment_floats(_dtype, l.meta.right.heads, l.meta.right.dim,
                                                                               l.meta.right.vdim));
#endif
        }
        _x = rt.allocateDeviceStorage(n_tokens * W * sizeof(float));
        _pass_in = rt.allocateDeviceStorage(n_tokens * 2 * W * _elem);
        _h = rt.allocateDeviceStorage(n_tokens * W * _elem);
        _proj = rt.allocateDeviceStorage(n_tokens * proj * _elem);
        _q = rt.allocateDeviceStorage(n_tokens * q * _elem);
        _row_scale = rt.allocateDeviceStorage(n_tokens * heads * sizeof(float));
        _mix = rt.allocateDeviceStorage(n_tokens * mix * _elem);
        _raw = rt.allocateDeviceStorage(n_tokens * raw * sizeof(float));
        _decay = rt.allocateDeviceStorage(n_tokens * decay * sizeof(float));
        if (segments != 0 && !_segments) {
            _segments = rt.allocateDeviceStorage(segments * sizeof(float));
        }
        _u = rt.allocateDeviceStorage(n_tokens * std::max<size_t>(ff, 1) * _elem);
#ifdef ENABLE_NVIDIA_API
        // the padding columns between and behind the two sides meet zero weights: they only have to be finite
        kernels::fill_zero(rt.stream(), _mix->memory(), _mix->size());
#endif
    }
    if (n_out > _ws_out) {
        _h_out = rt.allocateDeviceStorage(n_out * W * _elem);
    }
}

// ---- the network --------------------------------------------------------------------------------------------------------------

void Vozozen::forward(const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const size_t T = s.n_tokens, W = _meta.width;
    float *x = reinterpret_cast<float *>(_x->memory());
    std::byte *pass_in = _pass_in->memory(), *h = _h->memory(), *proj = _proj->memory(), *mix = _mix->memory(), *u = _u->memory();
    float *row_scale = reinterpret_cast<float *>(_row_scale->memory());
    beginRecord();

    // the right half of a pass's input is the embedding output, the same in every pass
    kernels::embed_scaled(_stream, _dtype, x, _loop_in != nullptr ? pass_in + W * _elem : nullptr, int64_t(2 * W), a.tokens, _embed,
                          _meta.embed_scale, T, W, _meta.voc);
    for (size_t run = 0; run < _runs.size(); ++run) {
        const Layer &l = _layers[_runs[run]];
        const LlaisysWindowAttentionMeta &la = l.meta.left;
        const LlaisysGatedLinearMeta &ra = l.meta.right;
        if (_starts_pass[run]) {
            kernels::stream_cast(_stream, _dtype, pass_in, int64_t(2 * W), x, T, W);
            kernels::linear_f32(_stream, _dtype, x, pass_in, _loop_in, T, W, 2 * W, false);
        }
        kernels::stream_rms_norm(_stream, _dtype, h, x, nullptr, l.norm1, _meta.eps, T, W);
        kernels::linear(_stream, _dtype, proj, h, l.proj, nullptr, T, l.n_proj, W);

        kernels::GatedLinearArgs g;
        g.proj = proj;
        g.row_stride = int64_t(l.n_proj);
        g.q_at = int64_t(l.rq);
        g.k_at = int64_t(l.rk);
        g.v_at = int64_t(l.rv);
        g.g_at = int64_t(l.rg);
        g.z_at = int64_t(l.z);
        g.decay_w = l.decay_w;
        g.decay_b = l.decay_b;
        g.norm_w = l.gla_norm;
        g.tau = ra.tau;
        g.q_scale = 1.f / std::sqrt(float(ra.dim));
        g.eps = _meta.eps;
        g.out_scale = l.meta.right_scale;
        g.heads = int32_t(ra.heads);
        g.dk = int32_t(ra.dim);
        g.dv = int32_t(ra.vdim);
        g.rank = int32_t(ra.rank);
        g.state = _state->data(run);
        g.slot_stride = int64_t(_state->slotStride(run));
        g.seq_ids = a.seq_list;
        g.q_starts = a.q_starts;
        g.kv_lens = a.kv_lens;
        g.n_seqs = int32_t(s.n_seqs);
        g.n_rows = int32_t(T);
        g.max_q_len = int32_t(s.max_q_len);
        g.out = mix + l.right * _elem;
        g.out_stride = int64_t(l.n_mix);
        g.raw = reinterpret_cast<float *>(_raw->memory());
        g.decay = reinterpret_cast<float *>(_decay->memory());
        g.segments = _segments ? reinterpret_cast<float *>(_segments->memory()) : nullptr;
        g.segment_floats = _segments ? _segments->size() / sizeof(float) : 0;
        if (s.decode_only) {
            kernels::gated_linear_decode(_stream, _dtype, g);
        } else {
            kernels::gated_linear_chunk(_stream, _dtype, g);
        }

        kernels::NormAppendArgs n;
        n.proj = proj;
        n.row_stride = int64_t(l.n_proj);
        n.q_at = int64_t(l.q);
        n.k_at = int64_t(l.k);
        n.v_at = int64_t(l.v);
        n.gate_at = int64_t(l.g);
        n.q_norm = l.q_norm;
        n.k_norm = l.k_norm;
        n.eps = _meta.eps;
        n.q_out = _q->memory();
        n.row_scale = row_scale;
        n.gate_scale = l.meta.left_scale;
        n.seq_ids = a.seq32;
        n.positions = a.pos32;
        n.n_rows = T;
        n.nh = int32_t(la.heads);
        _cache->normAppendDev(run, n, _stream);
        kv::AttnOptions opt;
        opt.window = la.window;
        opt.row_scale = row_scale;
        opt.row_stride = l.n_mix;
        if (s.decode_only) {
            _cache->decodeDev(run, mix, nullptr, _q->memory(), a.seq_list, a.kv_lens, s.n_seqs, s.max_kv_len, la.heads, la.scale,
                              _stream, opt);
        } else {
            _cache->prefillDev(run, mix, _q->memory(), a.seq_list, a.q_starts, a.kv_lens, s.n_seqs, T, s.max_q_len, s.max_kv_len,
                               la.heads, la.scale, _stream, opt);
        }
        kernels::linear_f32(_stream, _dtype, x, mix, l.out, T, W, l.n_mix, true);
        if (l.meta.ff != 0) {
            kernels::stream_rms_norm(_stream, _dtype, h, x, nullptr, l.norm2, _meta.eps, T, W);
            kernels::linear(_stream, _dtype, u, h, l.up, nullptr, T, l.meta.ff, W);
            kernels::relu_squared(_stream, _dtype, u, T * l.meta.ff);
            kernels::linear_f32(_stream, _dtype, x, u, l.down, T, W, l.meta.ff, true);
        }
        recordLayer(x, T * W);
    }
    if (s.n_out == 0) {
        return;
    }
    std::byte *h_out = _h_out->memory();
    float *logits = reinterpret_cast<float *>(_logits->memory());
    kernels::stream_rms_norm(_stream, _dtype, h_out, x, s.out_is_all ? nullptr : a.out_rows, _final_norm, _meta.eps, s.n_out, W);
    kernels::linear_f32(_stream, _dtype, logits, h_out, _head, s.n_out, _meta.voc, W, false);
    kernels::softcap_argmax(_stream, logits, _meta.logit_softcap, a.next, s.n_out, _meta.voc, _argmax_scratch->memory());
#else
    (void)a;
    (void)s;
    failModel(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
}

} // namespace llaisys::models
