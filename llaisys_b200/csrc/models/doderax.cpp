#include "doderax.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <algorithm>
#include <cmath>
#include <initializer_list>

namespace llaisys::models {

// ---- construction -------------------------------------------------------------------------------------------------------

Doderax::Doderax(const LlaisysDoderaxMeta &meta, llaisysDeviceType_t device, int device_id)
    : StreamDecoder("doderax", device, device_id, meta.dtype), _meta(meta) {
    if (meta.nlayer == 0 || meta.layers == nullptr || meta.width == 0 || meta.voc == 0) {
        failModel(LLAISYS_E_INVALID, "inconsistent model dimensions");
    }
    for (size_t i = 0; i < meta.nlayer; ++i) {
        const LlaisysDeltaMixerMeta &d = meta.layers[i].delta;
        const LlaisysSinkAttentionMeta &a = meta.layers[i].attn;
        const bool delta_ok = d.heads != 0 && d.kv_heads != 0 && d.heads % d.kv_heads == 0 && d.dim != 0 && d.vdim != 0 && d.taps != 0;
        const bool attn_ok = !meta.layers[i].parallel ||
                             (a.heads != 0 && a.kv_heads != 0 && a.heads % a.kv_heads == 0 && a.dim != 0 && a.vdim != 0 && a.window != 0 &&
                              a.rot_dims <= a.dim && a.rot_dims % 2 == 0 && (a.rot_dims == 0 || a.rot_base > 0.0));
        if (!delta_ok || !attn_ok) {
            failModel(LLAISYS_E_INVALID, "layer " + std::to_string(i) + ": inconsistent mixer sizes");
        }
    }
    enter();

    const size_t W = meta.width;
    _embed = matrix(meta.voc, W);
    place("embed", _embed, 0, 0, meta.voc, W, W);
    if (meta.pair_buckets != 0) {
        _pairs = matrix(meta.pair_buckets + 1, W);
        place("bigram", _pairs, 0, 0, meta.pair_buckets + 1, W, W);
    }
    size_t kv_layers = 0;
    for (size_t i = 0; i < meta.nlayer; ++i) {
        Layer l{};
        l.meta = meta.layers[i];
        const LlaisysSinkAttentionMeta &a = l.meta.attn;
        const LlaisysDeltaMixerMeta &d = l.meta.delta;
        const bool beside = l.meta.parallel != 0;
        const std::string p = "l" + std::to_string(i) + ".", ml = p + "mix.left.", md = p + (beside ? "mix.right." : "mix.");
        struct Part {
            std::string name;
            size_t *at, rows;
        };
        std::vector<Part> parts;
        if (beside) {
            parts = {{ml + "q", &l.aq, a.heads * a.dim}, {ml + "k", &l.ak, a.kv_heads * a.dim}, {ml + "v", &l.av, a.kv_heads * a.vdim}};
        }
        for (const Part &part : std::initializer_list<Part>{{md + "q", &l.q, d.kv_heads * d.dim},
                                                            {md + "k", &l.k, d.kv_heads * d.dim},
                                                            {md + "v", &l.v, d.heads * d.vdim},
                                                            {md + "b", &l.b, d.heads},
                                                            {md + (d.decay_rank ? "a1" : "a"), &l.a, d.decay_rank ? d.decay_rank : d.heads},
                                                            {md + (d.gate_rank ? "g1" : "g"), &l.g, d.gate_rank ? d.gate_rank : d.heads * d.vdim}}) {
            parts.push_back(part);
        }
        if (l.meta.ff != 0) {
            parts.push_back({p + "mlp.up", &l.up, l.meta.ff});
        }
        size_t rows = 0;
        for (const Part &part : parts) {
            *part.at = rows;
            rows += pad8(part.rows);
        }
        l.n_proj = rows;
        l.proj = matrix(rows, W);
        for (const Part &part : parts) {
            place(part.name, l.proj, *part.at, 0, part.rows, W, W);
        }
        auto whole = [&](const std::string &name, size_t r, size_t c, size_t ld) {
            std::byte *m = matrix(r, ld);
            place(name, m, 0, 0, r, c, ld);
            return m;
        };
        l.norm1 = vector(p + "norm1", W);
        l.conv_q = whole(md + "q.conv", d.kv_heads * d.dim, d.taps, d.taps);
        l.conv_k = whole(md + "k.conv", d.kv_heads * d.dim, d.taps, d.taps);
        l.conv_v = whole(md + "v.conv", d.heads * d.vdim, d.taps, d.taps);
        l.a_log = vector(md + "A_log", d.heads);
        l.dt_bias = vector(md + "dt_bias", d.decay_rank ? d.heads * d.dim : d.heads);
        l.head_norm = vector(md + "norm", d.vdim);
        if (d.decay_rank != 0) {
            l.decay_w = whole(md + "a2", d.heads * d.dim, d.decay_rank, pad8(d.decay_rank));
        }
        if (d.gate_rank != 0) {
            l.gate_w = whole(md + "g2", d.heads * d.vdim, d.gate_rank, pad8(d.gate_rank));
        }
        const size_t attn_cols = a.heads * a.vdim, delta_cols = d.heads * d.vdim;
        l.right = beside ? pad8(attn_cols) : 0;
        l.ff = l.right + pad8(delta_cols);
        l.n_mix = l.ff + pad8(l.meta.ff);
        if (beside) {
            l.out_left = whole(ml + "o", W, attn_cols, pad8(attn_cols));
            l.out_right = whole(md + "o", W, delta_cols, pad8(delta_cols));
            l.left_norm = vector(ml + "out", W);
            l.right_norm = vector(md + "out", W);
            if (l.meta.ff != 0) {
                l.down = whole(p + "mlp.down", W, l.meta.ff, pad8(l.meta.ff));
            }
            l.kv_layer = kv_layers++;
            l.rotary = a.rot_dims != 0 ? rotary(a.rot_base, a.rot_dims) : 0;
        } else {
            l.out = matrix(W, l.n_mix);
            place(md + "o", l.out, 0, 0, W, delta_cols, l.n_mix);
            if (l.meta.ff != 0) {
                place(p + "mlp.down", l.out, 0, l.ff, W, l.meta.ff, l.n_mix);
            }
        }
        _layers.push_back(l);
    }
    _final_norm = vector("final.norm", W);
    _head = matrix(meta.voc, W);
    place("head", _head, 0, 0, meta.voc, W, W);
    _meta.layers = nullptr; // the caller's array; every layer keeps its own copy
}

size_t Doderax::rotary(double base, size_t dims) {
    for (size_t i = 0; i < _rotary.size(); ++i) {
        if (_rotary[i].base == base && _rotary[i].dims == dims) {
            return i;
        }
    }
    std::vector<float> freq(dims / 2);
    for (size_t i = 0; i < freq.size(); ++i) {
        freq[i] = float(std::pow(base, -2.0 * double(i) / double(dims)));
    }
    auto &rt = enter();
    Rotary r{base, dims, rt.allocateDeviceStorage(freq.size() * sizeof(float)), nullptr};
    rt.api()->memcpy_sync(r.freq->memory(), freq.data(), freq.size() * sizeof(float), LLAISYS_MEMCPY_H2D);
    _rotary.push_back(std::move(r));
    return _rotary.size() - 1;
}

// ---- cache, state, workspace ------------------------------------------------------------------------------------------------

kv::PagedKVConfig Doderax::cacheShape() const {
    kv::PagedKVConfig cfg;
    for (const Layer &l : _layers) {
        if (l.meta.parallel) {
            cfg.layers.push_back(kv::KVLayerShape{l.meta.attn.kv_heads, l.meta.attn.dim, l.meta.attn.vdim});
        }
    }
    if (cfg.layers.empty()) { // without attention the pages only count tokens
        cfg.layers.push_back(kv::KVLayerShape{1, 8, 8});
    }
    cfg.nlayer = cfg.layers.size();
    return cfg;
}

std::vector<size_t> Doderax::stateShape() const {
    std::vector<size_t> floats;
#ifdef ENABLE_NVIDIA_API
    for (const Layer &l : _layers) {
        const LlaisysDeltaMixerMeta &d = l.meta.delta;
        floats.push_back(kernels::gated_delta_state_floats(d.heads, d.kv_heads, d.dim, d.vdim, d.taps));
    }
#endif
    return floats;
}

void Doderax::ensureActivations(size_t n_tokens, size_t n_out) {
    auto &rt = enter();
    const size_t W = _meta.width;
    if (n_tokens > _ws_tokens) {
        ++_generation;
        size_t proj = 0, gate = 0, q = 0, mix = 0, beside = 0, scratch = 0, segments = 0;
        for (const Layer &l : _layers) {
            const LlaisysDeltaMixerMeta &d = l.meta.delta;
            proj = std::max(proj, l.n_proj);
            mix = std::max(mix, l.n_mix);
            gate = std::max(gate, d.gate_rank != 0 ? pad8(d.heads * d.vdim) : 0);
            if (l.meta.parallel) {
                q = std::max(q, l.meta.attn.heads * l.meta.attn.dim);
                beside = W;
            }
#ifdef ENABLE_NVIDIA_API
            scratch = std::max(scratch, kernels::gated_delta_scratch_floats(_dtype, n_tokens, d.heads, d.kv_heads, d.dim, d.vdim));
            segments = std::max(segments, kernels::gated_delta_segment_floats(_dtype, d.heads, d.dim, d.vdim));
#endif
        }
        auto block = [&](size_t bytes) { return bytes != 0 ? rt.allocateDeviceStorage(bytes) : core::storage_t{}; };
        _x = block(n_tokens * W * sizeof(float));
        _h = block(n_tokens * W * _elem);
        _proj = block(n_tokens * proj * _elem);
        _gate = block(n_tokens * gate * _elem);
        _q = block(n_tokens * q * _elem);
        _mix = block(n_tokens * mix * _elem);
        _left = block(n_tokens * beside * sizeof(float));
        _right = block(n_tokens * beside * sizeof(float));
        _scratch = block(scratch * sizeof(float));
        for (Rotary &r : _rotary) {
            r.table = block(n_tokens * r.dims * sizeof(float));
        }
        if (segments != 0 && !_segments) {
            _segments = block(segments * sizeof(float));
        }
#ifdef ENABLE_NVIDIA_API
        // padding columns of the mix buffer meet zero weights: they only have to be finite
        kernels::fill_zero(rt.stream(), _mix->memory(), _mix->size());
#endif
    }
    if (n_out > _ws_out) {
        _h_out = rt.allocateDeviceStorage(n_out * W * _elem);
    }
}

// ---- the network --------------------------------------------------------------------------------------------------------------

void Doderax::delta(size_t layer, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const Layer &l = _layers[layer];
    const LlaisysDeltaMixerMeta &d = l.meta.delta;
    std::byte *proj = _proj->memory();
    kernels::GatedDeltaArgs g;
    g.gate = proj + l.g * _elem;
    g.gate_stride = int64_t(l.n_proj);
    if (d.gate_rank != 0) {
        const size_t cols = pad8(d.heads * d.vdim);
        kernels::linear(_stream, _dtype, _gate->memory(), proj + l.g * _elem, l.gate_w, nullptr, s.n_tokens, d.heads * d.vdim,
                        pad8(d.gate_rank), false, l.n_proj, cols);
        g.gate = _gate->memory();
        g.gate_stride = int64_t(cols);
    }
    g.gate_silu = d.gate_rank == 0 ? 1 : 0;
    g.proj = proj;
    g.row_stride = int64_t(l.n_proj);
    g.q_at = int64_t(l.q);
    g.k_at = int64_t(l.k);
    g.v_at = int64_t(l.v);
    g.b_at = int64_t(l.b);
    g.a_at = int64_t(l.a);
    g.conv_q = l.conv_q;
    g.conv_k = l.conv_k;
    g.conv_v = l.conv_v;
    g.taps = int32_t(d.taps);
    g.decay_w = l.decay_w;
    g.decay_ld = int64_t(pad8(d.decay_rank));
    g.a_log = l.a_log;
    g.dt_bias = l.dt_bias;
    g.norm_w = l.head_norm;
    g.q_scale = 1.f / std::sqrt(float(d.dim));
    g.eps = _meta.eps;
    g.heads = int32_t(d.heads);
    g.kv_heads = int32_t(d.kv_heads);
    g.dk = int32_t(d.dim);
    g.dv = int32_t(d.vdim);
    g.rank = int32_t(d.decay_rank);
    g.state = _state->data(layer);
    g.slot_stride = int64_t(_state->slotStride(layer));
    g.seq_ids = a.seq_list;
    g.q_starts = a.q_starts;
    g.kv_lens = a.kv_lens;
    g.n_seqs = int32_t(s.n_seqs);
    g.n_rows = int32_t(s.n_tokens);
    g.max_q_len = int32_t(s.max_q_len);
    g.out = _mix->memory() + l.right * _elem;
    g.out_stride = int64_t(l.n_mix);
    g.scratch = reinterpret_cast<float *>(_scratch->memory());
    g.scratch_floats = _scratch->size() / sizeof(float);
    g.segments = _segments ? reinterpret_cast<float *>(_segments->memory()) : nullptr;
    g.segment_floats = _segments ? _segments->size() / sizeof(float) : 0;
    if (s.decode_only) {
        kernels::gated_delta_decode(_stream, _dtype, g);
    } else {
        kernels::gated_delta_chunk(_stream, _dtype, g);
    }
#else
    (void)layer, (void)a, (void)s;
#endif
}

void Doderax::attention(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysSinkAttentionMeta &m = l.meta.attn;
    kernels::NormAppendArgs n;
    n.proj = _proj->memory();
    n.row_stride = int64_t(l.n_proj);
    n.q_at = int64_t(l.aq);
    n.k_at = int64_t(l.ak);
    n.v_at = int64_t(l.av);
    n.gate_at = -1;
    n.rot_dims = int32_t(m.rot_dims);
    n.rot_table = m.rot_dims != 0 ? reinterpret_cast<const float *>(_rotary[l.rotary].table->memory()) : nullptr;
    n.q_out = _q->memory();
    n.seq_ids = a.seq32;
    n.positions = a.pos32;
    n.n_rows = s.n_tokens;
    n.nh = int32_t(m.heads);
    _cache->normAppendDev(l.kv_layer, n, _stream);
    kv::AttnOptions opt;
    opt.window = m.window;
    opt.keep_first = m.keep_first;
    opt.row_stride = l.n_mix;
    if (s.decode_only) {
        _cache->decodeDev(l.kv_layer, _mix->memory(), nullptr, _q->memory(), a.seq_list, a.kv_lens, s.n_seqs, s.max_kv_len, m.heads, m.scale,
                          _stream, opt);
    } else {
        _cache->prefillDev(l.kv_layer, _mix->memory(), _q->memory(), a.seq_list, a.q_starts, a.kv_lens, s.n_seqs, s.n_tokens, s.max_q_len,
                           s.max_kv_len, m.heads, m.scale, _stream, opt);
    }
#else
    (void)l, (void)a, (void)s;
#endif
}

void Doderax::forward(const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const size_t T = s.n_tokens, W = _meta.width;
    float *x = reinterpret_cast<float *>(_x->memory());
    std::byte *h = _h->memory(), *proj = _proj->memory(), *mix = _mix->memory();
    beginRecord();
    if (_pairs != nullptr) {
        kernels::embed_pairs(_stream, _dtype, x, a.tokens, a.prev, _embed, _pairs, _meta.pair_mul_prev, _meta.pair_mul_cur,
                             int64_t(_meta.pair_buckets), T, W, _meta.voc);
    } else {
        kernels::embed_scaled(_stream, _dtype, x, nullptr, 0, a.tokens, _embed, 1.f, T, W, _meta.voc);
    }
    for (const Rotary &r : _rotary) {
        kernels::rotary_table(_stream, reinterpret_cast<float *>(r.table->memory()), a.pos32, reinterpret_cast<const float *>(r.freq->memory()),
                              T, r.dims / 2);
    }
    bool normed = false; // h holds the norm of x that the coming layer reads
    for (size_t i = 0; i < _layers.size(); ++i) {
        const Layer &l = _layers[i];
        const size_t ff = l.meta.ff;
        if (!normed) {
            kernels::stream_rms_norm(_stream, _dtype, h, x, nullptr, l.norm1, _meta.eps, T, W, 1.f);
        }
        kernels::linear(_stream, _dtype, proj, h, l.proj, nullptr, T, l.n_proj, W);
        delta(i, a, s);
        if (l.meta.parallel) {
            attention(l, a, s);
        }
        if (ff != 0) {
            kernels::gelu_tanh(_stream, _dtype, mix + l.ff * _elem, int64_t(l.n_mix), proj + l.up * _elem, int64_t(l.n_proj), T, ff);
        }
        normed = false;
        if (!l.meta.parallel) {
            kernels::linear_f32(_stream, _dtype, x, mix, l.out, T, W, l.n_mix, true);
        } else {
            float *left = reinterpret_cast<float *>(_left->memory()), *right = reinterpret_cast<float *>(_right->memory());
            kernels::linear_f32(_stream, _dtype, left, mix, l.out_left, T, W, l.right, false, 1.f, l.n_mix);
            kernels::linear_f32(_stream, _dtype, right, mix + l.right * _elem, l.out_right, T, W, l.ff - l.right, false, 1.f, l.n_mix);
            if (ff != 0) {
                kernels::linear_f32(_stream, _dtype, x, mix + l.ff * _elem, l.down, T, W, l.n_mix - l.ff, true, 1.f, l.n_mix);
            }
            normed = i + 1 < _layers.size();
            kernels::stream_add_normed(_stream, _dtype, x, left, l.left_norm, right, l.right_norm, 0.5f, _meta.eps, normed ? h : nullptr,
                                       normed ? _layers[i + 1].norm1 : nullptr, 1.f, T, W);
        }
        recordLayer(x, T * W);
    }
    if (s.n_out == 0) {
        return;
    }
    std::byte *h_out = _h_out->memory();
    float *logits = reinterpret_cast<float *>(_logits->memory());
    kernels::stream_rms_norm(_stream, _dtype, h_out, x, s.out_is_all ? nullptr : a.out_rows, _final_norm, _meta.eps, s.n_out, W, 1.f);
    kernels::linear_f32(_stream, _dtype, logits, h_out, _head, s.n_out, _meta.voc, W, false, _meta.logit_scale);
    kernels::softcap_argmax(_stream, logits, 0.f, a.next, s.n_out, _meta.voc, _argmax_scratch->memory());
#else
    (void)a, (void)s;
    failModel(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
}

} // namespace llaisys::models
