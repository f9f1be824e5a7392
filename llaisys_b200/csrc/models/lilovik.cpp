#include "lilovik.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <algorithm>
#include <cmath>

namespace llaisys::models {

namespace {
constexpr double kPositionBase = 10000.0, kSlopeExponent = 8.0;
}

// ---- construction -------------------------------------------------------------------------------------------------------

Lilovik::Lilovik(const LlaisysLilovikMeta &meta, llaisysDeviceType_t device, int device_id)
    : StreamDecoder("lilovik", device, device_id, meta.dtype), _meta(meta) {
    if (meta.nlayer == 0 || meta.layers == nullptr || meta.width == 0 || meta.voc == 0) {
        failModel(LLAISYS_E_INVALID, "inconsistent model dimensions");
    }
    for (size_t i = 0; i < meta.nlayer; ++i) {
        const LlaisysLilovikLayerMeta &m = meta.layers[i];
        const LlaisysGatesAttentionMeta &a = m.attn;
        const bool ok = m.recurrent ? m.gru_width != 0
                                    : a.heads != 0 && a.kv_heads != 0 && a.heads % a.kv_heads == 0 && a.dim != 0 && a.vdim != 0 &&
                                          (a.temp_coef == 0.f || a.temp_every > 0.f);
        if (!ok) {
            failModel(LLAISYS_E_INVALID, "layer " + std::to_string(i) + ": inconsistent mixer sizes");
        }
    }
    auto &rt = enter();

    const size_t W = meta.width;
    auto whole = [&](const std::string &name, size_t r, size_t c, size_t ld) {
        std::byte *m = matrix(r, ld);
        place(name, m, 0, 0, r, c, ld);
        return m;
    };
    _embed = whole("embed", meta.voc, W, W);
    size_t kv_layers = 0, state_layers = 0;
    for (size_t i = 0; i < meta.nlayer; ++i) {
        Layer l{};
        l.meta = meta.layers[i];
        const LlaisysGatesAttentionMeta &a = l.meta.attn;
        const bool gru = l.meta.recurrent != 0;
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
        const char *names[3] = {gru ? "z" : "q", gru ? "x" : "k", gru ? "g" : "v"};
        const size_t rows[3] = {gru ? l.meta.gru_width : a.heads * a.dim, gru ? l.meta.gru_width : a.kv_heads * a.dim,
                                gru ? l.meta.gru_width : a.kv_heads * a.vdim};
        for (int part = 0; part < 3; ++part) {
            l.at[part] = l.n_proj;
            l.n_proj += pad8(rows[part]);
        }
        l.proj = matrix(l.n_proj, W);
        l.bias = matrix(l.n_proj, 1);
        for (int part = 0; part < 3; ++part) {
            place(m + names[part], l.proj, l.at[part], 0, rows[part], W, W);
            if (!gru || part < 2) {
                place(m + names[part] + ".b", l.bias, l.at[part], 0, rows[part], 1, 1, 1);
            }
        }
        l.norm1 = vector(p + "norm1", W);
        l.norm1b = vector(p + "norm1b", W);
        const size_t mixed = gru ? l.meta.gru_width : a.heads * a.vdim;
        l.n_mix = pad8(mixed);
        l.out = whole(m + "o", W, mixed, l.n_mix);
        if (gru) {
            l.index = state_layers++;
        } else {
            l.index = kv_layers++;
            l.q_norm = vector(m + "q.norm", a.heads * a.dim);
            l.k_norm = vector(m + "k.norm", a.kv_heads * a.dim);
            l.talk = whole(m + "talk", a.heads, a.heads, a.heads);
            l.score_bias = vector(m + "pb", a.heads);
            std::vector<float> slopes(a.heads);
            for (size_t h = 0; h < a.heads; ++h) {
                slopes[h] = float(std::exp2(-kSlopeExponent * double(h + 1) / double(a.heads)));
            }
            l.slopes = rt.allocateDeviceStorage(a.heads * sizeof(float));
            rt.api()->memcpy_sync(l.slopes->memory(), slopes.data(), a.heads * sizeof(float), LLAISYS_MEMCPY_H2D);
        }
        if (l.meta.ff != 0) {
            l.ff = pad8(l.meta.ff);
            l.norm2 = vector(p + "norm2", W);
            l.norm2b = vector(p + "norm2b", W);
            l.gate_up = matrix(2 * l.ff, W);
            place(p + "mlp.gate", l.gate_up, 0, 0, l.meta.ff, W, W);
            place(p + "mlp.up", l.gate_up, l.ff, 0, l.meta.ff, W, W);
            l.down = whole(p + "mlp.down", W, l.meta.ff, l.ff);
        }
        _layers.push_back(std::move(l));
    }
    _final_norm = vector("final.norm", W);
    _head = whole("head", meta.voc, W, W);
    std::vector<double> freq((W + 1) / 2);
    for (size_t i = 0; i < freq.size(); ++i) {
        freq[i] = std::pow(kPositionBase, -2.0 * double(i) / double(W));
    }
    _freq = rt.allocateDeviceStorage(freq.size() * sizeof(double));
    rt.api()->memcpy_sync(_freq->memory(), freq.data(), freq.size() * sizeof(double), LLAISYS_MEMCPY_H2D);
    _meta.layers = nullptr; // the caller's array; every layer keeps its own copy
}

// ---- cache, state, workspace ------------------------------------------------------------------------------------------------

kv::PagedKVConfig Lilovik::cacheShape() const {
    kv::PagedKVConfig cfg;
    for (const Layer &l : _layers) {
        if (!l.meta.recurrent) {
            cfg.layers.push_back(kv::KVLayerShape{l.meta.attn.kv_heads, l.meta.attn.dim, l.meta.attn.vdim});
        }
    }
    if (cfg.layers.empty()) { // without attention the pages only count tokens
        cfg.layers.push_back(kv::KVLayerShape{1, 8, 8});
    }
    cfg.nlayer = cfg.layers.size();
    return cfg;
}

std::vector<size_t> Lilovik::stateShape() const {
    std::vector<size_t> floats;
    for (const Layer &l : _layers) {
        if (l.meta.recurrent) {
            floats.push_back(l.meta.gru_width);
        }
    }
    return floats;
}

void Lilovik::ensureActivations(size_t n_tokens, size_t n_out) {
    auto &rt = enter();
    const size_t W = _meta.width;
    if (n_tokens > _ws_tokens) {
        ++_generation;
        size_t proj = 0, q = 0, mix = 0, ff = 0, scratch = 0;
        for (const Layer &l : _layers) {
            proj = std::max({proj, l.n_proj, 2 * l.ff});
            mix = std::max(mix, l.n_mix);
            ff = std::max(ff, l.ff);
#ifdef ENABLE_NVIDIA_API
            scratch = std::max(scratch, l.meta.recurrent ? kernels::min_gru_scratch_floats(n_tokens, l.meta.gru_width) : 0);
#endif
            q = std::max(q, l.meta.recurrent ? 0 : l.meta.attn.heads * l.meta.attn.dim);
        }
        auto block = [&](size_t bytes) { return bytes != 0 ? rt.allocateDeviceStorage(bytes) : core::storage_t{}; };
        _x = block(n_tokens * W * sizeof(float));
        _y = block(n_tokens * W * sizeof(float));
        _h = block(n_tokens * W * _elem);
        _proj = block(n_tokens * proj * _elem);
        _q = block(n_tokens * q * _elem);
        _mix = block(n_tokens * mix * _elem);
        _u = block(n_tokens * ff * _elem);
        _scratch = block(scratch * sizeof(float));
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

void Lilovik::attention(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysGatesAttentionMeta &m = l.meta.attn;
    kernels::NormAppendArgs n;
    n.proj = _proj->memory();
    n.row_stride = int64_t(l.n_proj);
    n.q_at = int64_t(l.at[0]);
    n.k_at = int64_t(l.at[1]);
    n.v_at = int64_t(l.at[2]);
    n.gate_at = -1;
    n.row_norm = 1;
    n.bias = l.bias;
    n.q_norm = l.q_norm;
    n.k_norm = l.k_norm;
    n.eps = _meta.eps;
    n.temp_coef = m.temp_coef;
    n.temp_every = m.temp_coef != 0.f ? m.temp_every : 1.f;
    n.q_out = _q->memory();
    n.seq_ids = a.seq32;
    n.positions = a.pos32;
    n.n_rows = s.n_tokens;
    n.nh = int32_t(m.heads);
    _cache->normAppendDev(l.index, n, _stream);
    kernels::GateArgs gates;
    gates.softcap = m.softcap;
    gates.slopes = reinterpret_cast<const float *>(l.slopes->memory());
    gates.bias = l.score_bias;
    gates.talk = l.talk;
    kv::AttnOptions opt;
    opt.gates = &gates;
    opt.row_stride = l.n_mix;
    if (s.decode_only) {
        _cache->decodeDev(l.index, _mix->memory(), nullptr, _q->memory(), a.seq_list, a.kv_lens, s.n_seqs, s.max_kv_len, m.heads, m.scale,
                          _stream, opt);
    } else {
        _cache->prefillDev(l.index, _mix->memory(), _q->memory(), a.seq_list, a.q_starts, a.kv_lens, s.n_seqs, s.n_tokens, s.max_q_len,
                           s.max_kv_len, m.heads, m.scale, _stream, opt);
    }
#else
    (void)l, (void)a, (void)s;
#endif
}

void Lilovik::recurrence(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    kernels::MinGruArgs g;
    g.proj = _proj->memory();
    g.row_stride = int64_t(l.n_proj);
    g.z_at = int64_t(l.at[0]);
    g.x_at = int64_t(l.at[1]);
    g.g_at = int64_t(l.at[2]);
    g.bias_z = l.bias + l.at[0] * _elem;
    g.bias_x = l.bias + l.at[1] * _elem;
    g.width = int32_t(l.meta.gru_width);
    g.state = _state->data(l.index);
    g.slot_stride = int64_t(_state->slotStride(l.index));
    g.seq_ids = a.seq_list;
    g.q_starts = a.q_starts;
    g.kv_lens = a.kv_lens;
    g.n_seqs = int32_t(s.n_seqs);
    g.n_rows = int32_t(s.n_tokens);
    g.max_q_len = int32_t(s.max_q_len);
    g.out = _mix->memory();
    g.out_stride = int64_t(l.n_mix);
    g.scratch = reinterpret_cast<float *>(_scratch->memory());
    g.scratch_floats = _scratch->size() / sizeof(float);
    if (s.decode_only) {
        kernels::min_gru_decode(_stream, _dtype, g);
    } else {
        kernels::min_gru_chunk(_stream, _dtype, g);
    }
#else
    (void)l, (void)a, (void)s;
#endif
}

void Lilovik::forward(const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const size_t T = s.n_tokens, W = _meta.width;
    float *x = reinterpret_cast<float *>(_x->memory()), *y = reinterpret_cast<float *>(_y->memory());
    std::byte *h = _h->memory(), *proj = _proj->memory(), *mix = _mix->memory();
    beginRecord();
    kernels::embed_positions(_stream, _dtype, x, a.tokens, a.pos32, reinterpret_cast<const double *>(_freq->memory()), _embed, T, W, _meta.voc);
    kernels::stream_rms_norm(_stream, _dtype, h, x, nullptr, _layers[0].norm1, _meta.eps, T, W, 1.f);
    for (size_t i = 0; i < _layers.size(); ++i) {
        const Layer &l = _layers[i];
        // the norm of y into the stream, and h = the norm that comes next
        auto add = [&](const std::byte *norm, const std::byte *next) {
            kernels::stream_add_normed(_stream, _dtype, x, y, norm, nullptr, nullptr, 1.f, _meta.eps, next != nullptr ? h : nullptr, next, 1.f,
                                       T, W, 1.f);
        };
        const std::byte *next_layer = i + 1 < _layers.size() ? _layers[i + 1].norm1 : nullptr;
        kernels::linear(_stream, _dtype, proj, h, l.proj, nullptr, T, l.n_proj, W);
        l.meta.recurrent ? recurrence(l, a, s) : attention(l, a, s);
        kernels::linear_f32(_stream, _dtype, y, mix, l.out, T, W, l.n_mix, false);
        add(l.norm1b, l.ff != 0 ? l.norm2 : next_layer);
        if (l.ff != 0) {
            kernels::linear(_stream, _dtype, proj, h, l.gate_up, nullptr, T, 2 * l.ff, W);
            kernels::relu_glu_packed(_stream, _dtype, _u->memory(), proj, T, l.ff);
            kernels::linear_f32(_stream, _dtype, y, _u->memory(), l.down, T, W, l.ff, false);
            add(l.norm2b, next_layer);
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
