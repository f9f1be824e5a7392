#include "folivik.hpp"

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
constexpr size_t kExpandFrom = 128;    // tokens of a chunk from which keys and values of its context are made
constexpr size_t kPassTokens = 65536;  // context rows that are expanded together (one sequence alone may have more)
constexpr size_t kTailRows = 64;       // zero rows behind the last context: key blocks of 64 may reach into them
} // namespace

// ---- construction -------------------------------------------------------------------------------------------------------

Folivik::Folivik(const LlaisysFolivikMeta &meta, llaisysDeviceType_t device, int device_id)
    : StreamDecoder("folivik", device, device_id, meta.dtype), _meta(meta) {
    if (meta.nlayer == 0 || meta.layers == nullptr || meta.width == 0 || meta.voc == 0) {
        failModel(LLAISYS_E_INVALID, "inconsistent model dimensions");
    }
    for (size_t i = 0; i < meta.nlayer; ++i) {
        const LlaisysFolivikLayerMeta &m = meta.layers[i];
        const LlaisysLatentAttentionMeta &t = m.latent;
        const LlaisysFadingAttentionMeta &a = m.attn;
        const LlaisysStateSpaceMixerMeta &d = m.ssm;
        const LlaisysExpertLayerMeta &e = m.mlp;
        bool ok = false;
        switch (m.mixer) {
        case LLAISYS_FOLIVIK_LATENT:
            ok = t.heads != 0 && t.dim != 0 && t.rot_dim % 2 == 0 && t.vdim != 0 && t.q_rank != 0 && t.kv_rank != 0 &&
                 (t.rot_dim == 0 || t.rot_base > 0.0);
            break;
        case LLAISYS_FOLIVIK_ATTENTION:
            ok = a.heads != 0 && a.kv_heads != 0 && a.heads % a.kv_heads == 0 && a.dim != 0 && a.vdim != 0 && a.window != 0;
            break;
        case LLAISYS_FOLIVIK_STATE_SPACE:
            ok = d.heads != 0 && d.groups != 0 && d.heads % d.groups == 0 && d.state != 0 && d.vdim != 0 && d.taps != 0 && d.norm_groups != 0 &&
                 d.heads * d.vdim % d.norm_groups == 0;
            break;
        default:
            break;
        }
        if (!ok) {
            failModel(LLAISYS_E_INVALID, "layer " + std::to_string(i) + ": inconsistent mixer sizes");
        }
        if (e.top != 0 && (e.experts == 0 || e.ff == 0 || e.groups == 0 || e.keep == 0 || e.keep > e.groups || (e.experts + e.identity) % e.groups != 0 ||
                           e.top > e.keep * ((e.experts + e.identity) / e.groups))) {
            failModel(LLAISYS_E_INVALID, "layer " + std::to_string(i) + ": inconsistent expert sizes");
        }
    }
    enter();

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
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
        struct Part {
            const char *name;
            size_t rows;
        };
        auto project = [&](const std::vector<Part> &parts) {
            for (size_t k = 0; k < parts.size(); ++k) {
                l.at[k] = l.n_proj;
                l.n_proj += pad8(parts[k].rows);
            }
            l.proj = matrix(l.n_proj, W);
            for (size_t k = 0; k < parts.size(); ++k) {
                place(m + parts[k].name, l.proj, l.at[k], 0, parts[k].rows, W, W);
            }
        };
        l.norm1 = floats(p + "norm1", 0);
        size_t mixed = 0;
        if (l.meta.mixer == LLAISYS_FOLIVIK_LATENT) {
            const LlaisysLatentAttentionMeta &t = l.meta.latent;
            project({{"dq", t.q_rank}, {"dkv", t.kv_rank + t.rot_dim}, {"g", t.heads}});
            l.q_norm = vector(m + "dq.norm", t.q_rank);
            l.k_norm = vector(m + "dkv.norm", t.kv_rank);
            l.q_rank = pad8(t.q_rank);
            l.uq = whole(m + "uq", t.heads * (t.dim + t.rot_dim), t.q_rank, l.q_rank);
            l.uk = whole(m + "uk", t.heads * t.dim, t.kv_rank, t.kv_rank);
            l.uv = whole(m + "uv", t.heads * t.vdim, t.kv_rank, t.kv_rank);
            l.index = kv_layers++;
            l.rotary = t.rot_dim != 0 ? rotary(t.rot_base, t.rot_dim) : 0;
            mixed = t.heads * t.vdim;
        } else if (l.meta.mixer == LLAISYS_FOLIVIK_ATTENTION) {
            const LlaisysFadingAttentionMeta &a = l.meta.attn;
            project({{"q", a.heads * a.dim}, {"k", a.kv_heads * a.dim}, {"v", a.kv_heads * a.vdim}});
            l.q_norm = vector(m + "q.norm", a.dim);
            l.k_norm = vector(m + "k.norm", a.dim);
            l.temp = floats(m + "temp", a.heads);
            l.fade_a = floats(m + "r1", a.heads);
            l.fade_b = floats(m + "r2", a.heads);
            l.index = kv_layers++;
            mixed = a.heads * a.vdim;
        } else {
            const LlaisysStateSpaceMixerMeta &d = l.meta.ssm;
            const size_t inner = d.heads * d.vdim, channels = inner + 2 * d.groups * d.state;
            project({{"in", inner + channels + d.heads}});
            l.at[1] = inner;
            l.at[2] = inner + channels;
            l.conv_w = whole(m + "conv", channels, d.taps, d.taps);
            l.conv_b = vector(m + "conv.b", channels);
            l.a_log = floats(m + "A_log", d.heads);
            l.dt_bias = floats(m + "dt_bias", d.heads);
            l.d_skip = floats(m + "D", d.heads);
            l.norm_w = vector(m + "norm", inner);
            l.index = state_layers++;
            mixed = inner;
        }
        l.n_mix = pad8(mixed);
        l.out = whole(m + "o", W, mixed, l.n_mix);
        const LlaisysExpertLayerMeta &e = l.meta.mlp;
        if (e.top != 0) {
            const std::string f = p + "mlp.";
            l.norm2 = floats(p + "norm2", 0);
            l.router = whole(f + "router", e.experts + e.identity, W, W);
            l.correction = floats(f + "correction", e.experts + e.identity);
            l.ff = pad8(e.ff);
            l.gate_up = matrix(e.experts * 2 * l.ff, W);
            l.down = matrix(e.experts * W, l.ff);
            for (size_t j = 0; j < e.experts; ++j) {
                const std::string name = f + "e" + std::to_string(j) + ".";
                place(name + "gate", l.gate_up, 2 * j * l.ff, 0, e.ff, W, W);
                place(name + "up", l.gate_up, (2 * j + 1) * l.ff, 0, e.ff, W, W);
                place(name + "down", l.down, j * W, 0, W, e.ff, l.ff);
            }
            if (e.shared_ff != 0) {
                l.shared_ff = pad8(e.shared_ff);
                l.shared_gate_up = matrix(2 * l.shared_ff, W);
                place(f + "shared.gate", l.shared_gate_up, 0, 0, e.shared_ff, W, W);
                place(f + "shared.up", l.shared_gate_up, l.shared_ff, 0, e.shared_ff, W, W);
                l.shared_down = whole(f + "shared.down", W, e.shared_ff, l.shared_ff);
            }
        }
        _layers.push_back(l);
    }
    _final_norm = floats("final.norm", 0);
    _head = whole("head", meta.voc, W, W);
    _meta.layers = nullptr; // the caller's array; every layer keeps its own copy
}

size_t Folivik::rotary(double base, size_t dims) {
    for (size_t i = 0; i < _rotary.size(); ++i) {
        if (_rotary[i].base == base && _rotary[i].dims == dims) {
            return i;
        }
    }
    std::vector<double> freq(dims / 2);
    for (size_t i = 0; i < freq.size(); ++i) {
        freq[i] = std::pow(base, -2.0 * double(i) / double(dims));
    }
    auto &rt = enter();
    Rotary r{base, dims, rt.allocateDeviceStorage(freq.size() * sizeof(double)), nullptr};
    rt.api()->memcpy_sync(r.freq->memory(), freq.data(), freq.size() * sizeof(double), LLAISYS_MEMCPY_H2D);
    _rotary.push_back(std::move(r));
    return _rotary.size() - 1;
}

// ---- cache, state, workspace ------------------------------------------------------------------------------------------------

kv::PagedKVConfig Folivik::cacheShape() const {
    kv::PagedKVConfig cfg;
    for (const Layer &l : _layers) {
        if (l.meta.mixer == LLAISYS_FOLIVIK_LATENT) {
            const LlaisysLatentAttentionMeta &t = l.meta.latent;
            cfg.layers.push_back(kv::KVLayerShape{1, t.kv_rank + t.rot_dim, t.kv_rank, true});
        } else if (l.meta.mixer == LLAISYS_FOLIVIK_ATTENTION) {
            cfg.layers.push_back(kv::KVLayerShape{l.meta.attn.kv_heads, l.meta.attn.dim, l.meta.attn.vdim});
        }
    }
    if (cfg.layers.empty()) { // without attention the pages only count tokens
        cfg.layers.push_back(kv::KVLayerShape{1, 8, 8});
    }
    cfg.nlayer = cfg.layers.size();
    return cfg;
}

std::vector<size_t> Folivik::stateShape() const {
    std::vector<size_t> floats;
#ifdef ENABLE_NVIDIA_API
    for (const Layer &l : _layers) {
        if (l.meta.mixer == LLAISYS_FOLIVIK_STATE_SPACE) {
            const LlaisysStateSpaceMixerMeta &d = l.meta.ssm;
            floats.push_back(kernels::state_space_state_floats(d.heads, d.groups, d.state, d.vdim, d.taps));
        }
    }
#endif
    return floats;
}

void Folivik::ensureActivations(size_t n_tokens, size_t n_out) {
    auto &rt = enter();
    const size_t W = _meta.width;
    if (n_tokens > _ws_tokens) {
        ++_generation;
        size_t proj = 0, q = 0, q_wide = 0, latent = 0, scale = 0, mix = 0, scratch = 0, segments = 0, lane_out = 0;
        size_t router = 0, choice = 0, experts = 0, rows = 0, act = 0, out = 0, shared = 0;
        for (const Layer &l : _layers) {
            proj = std::max(proj, l.n_proj);
            mix = std::max(mix, l.n_mix);
            if (l.meta.mixer == LLAISYS_FOLIVIK_LATENT) {
                const LlaisysLatentAttentionMeta &t = l.meta.latent;
                q = std::max(q, t.heads * (t.dim + t.rot_dim));
                q_wide = std::max(q_wide, t.heads * (t.kv_rank + t.rot_dim));
                lane_out = std::max(lane_out, t.heads * t.kv_rank);
                latent = std::max(latent, l.q_rank);
                scale = std::max(scale, t.heads);
            } else if (l.meta.mixer == LLAISYS_FOLIVIK_ATTENTION) {
                q = std::max(q, l.meta.attn.heads * l.meta.attn.dim);
            } else {
#ifdef ENABLE_NVIDIA_API
                const LlaisysStateSpaceMixerMeta &d = l.meta.ssm;
                scratch = std::max(scratch, kernels::state_space_scratch_floats(_dtype, n_tokens, d.heads, d.groups, d.state, d.vdim));
                segments = std::max(segments, kernels::state_space_segment_floats(_dtype, d.heads, d.state, d.vdim));
#endif
            }
            const LlaisysExpertLayerMeta &e = l.meta.mlp;
            if (e.top != 0) {
                router = std::max(router, e.experts + e.identity);
                choice = std::max(choice, e.top);
                experts = std::max(experts, e.experts);
                rows = std::max(rows, e.top * W);
                act = std::max(act, e.top * l.ff);
                out = std::max(out, e.top * W);
                shared = std::max(shared, 2 * l.shared_ff);
            }
        }
        auto block = [&](size_t bytes) { return bytes != 0 ? rt.allocateDeviceStorage(bytes) : core::storage_t{}; };
        _x = block(n_tokens * W * sizeof(float));
        _h = block(n_tokens * W * _elem);
        _proj = block(n_tokens * std::max(proj, shared) * _elem);
        _q = block(n_tokens * q * _elem);
        _q_wide = block(n_tokens * (q_wide + lane_out) * _elem); // queries over latents, then outputs over latents
        _latent = block(n_tokens * latent * _elem);
        _scale = block(n_tokens * scale * sizeof(float));
        _mix = block(n_tokens * mix * _elem);
        _scratch = block(scratch * sizeof(float));
        _logits_e = block(n_tokens * router * sizeof(float));
        _choice = block(n_tokens * choice * 16); // chosen, weights, place, line
        _counts = block(experts * sizeof(int32_t));
        _rows = block(n_tokens * rows * _elem);
        _act = block(n_tokens * act * _elem);
        _expert_out = block(n_tokens * out * _elem);
        _shared = block(n_tokens * shared / 2 * _elem);
        for (Rotary &r : _rotary) {
            r.table = block(n_tokens * r.dims * sizeof(float));
        }
        if (segments != 0 && !_segments) {
            _segments = block(segments * sizeof(float));
        }
#ifdef ENABLE_NVIDIA_API
        // padding columns meet zero weights: they only have to be finite
        for (const core::storage_t &b : {_mix, _latent}) {
            if (b) {
                kernels::fill_zero(rt.stream(), b->memory(), b->size());
            }
        }
#endif
    }
    if (n_out > _ws_out) {
        _h_out = rt.allocateDeviceStorage(n_out * W * _elem);
    }
}

// ---- the network --------------------------------------------------------------------------------------------------------------

void Folivik::latentAttention(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysLatentAttentionMeta &m = l.meta.latent;
    const size_t T = s.n_tokens, H = m.heads;
    kernels::LatentAppendArgs n;
    n.proj = _proj->memory();
    n.row_stride = int64_t(l.n_proj);
    n.q_at = int64_t(l.at[0]);
    n.kv_at = int64_t(l.at[1]);
    n.gate_at = int64_t(l.at[2]);
    n.q_rank = int32_t(m.q_rank);
    n.rank = int32_t(m.kv_rank);
    n.rot_dims = int32_t(m.rot_dim);
    n.nh = int32_t(H);
    n.q_norm = l.q_norm;
    n.kv_norm = l.k_norm;
    n.eps = _meta.eps;
    n.rot_table = m.rot_dim != 0 ? reinterpret_cast<const float *>(_rotary[l.rotary].table->memory()) : nullptr;
    n.q_latent = _latent->memory();
    n.q_latent_stride = int64_t(l.q_rank);
    n.row_scale = reinterpret_cast<float *>(_scale->memory());
    n.seq_ids = a.seq32;
    n.positions = a.pos32;
    n.n_rows = T;
    _cache->latentAppendDev(l.index, n, _stream);
    kernels::linear(_stream, _dtype, _q->memory(), _latent->memory(), l.uq, nullptr, T, H * (m.dim + m.rot_dim), l.q_rank);
    if (s.decode_only || !_cache->latentTc(l.index, H) || !_cache->canExpand(l.index, m.dim, m.rot_dim, m.vdim)) {
        latentRange(l, a, s, LatentRange{false, 0, s.n_seqs, 0, T, s.max_q_len, s.max_kv_len, 0});
        return;
    }
    for (const LatentRange &r : _ranges) {
        r.expanded ? expandedRange(l, a, s, r) : latentRange(l, a, s, r);
    }
#else
    (void)l, (void)a, (void)s;
#endif
}

// Sequences whose queries are multiplied into the latents' space
void Folivik::latentRange(const Layer &l, const StepArrays &a, const StepShape &s, const LatentRange &r) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysLatentAttentionMeta &m = l.meta.latent;
    const size_t T = s.n_tokens, H = m.heads, row = m.kv_rank + m.rot_dim, dim = m.dim + m.rot_dim;
    const float *table = m.rot_dim != 0 ? reinterpret_cast<const float *>(_rotary[l.rotary].table->memory()) + r.row * m.rot_dim : nullptr;
    std::byte *wide = _q_wide->memory(), *out = wide + T * H * row * _elem; // (whole steps: the attention kernels take absolute rows)
    const std::byte *q = _q->memory() + r.row * H * dim * _elem;
    std::byte *q_rows = wide + r.row * H * row * _elem;
    kernels::linear_heads(_stream, _dtype, q_rows, q, l.uk, r.n_rows, H, m.kv_rank, m.dim, true, H * dim, dim, H * row, row);
    kernels::rotate_pairs(_stream, _dtype, q_rows, row, m.kv_rank, q, m.dim, m.rot_dim, table, r.n_rows, H);
    kv::AttnOptions opt;
    opt.row_scale = reinterpret_cast<const float *>(_scale->memory());
    const size_t n = r.to - r.from;
    if (s.decode_only) {
        _cache->decodeDev(l.index, out, nullptr, wide, a.seq_list, a.kv_lens, n, s.max_kv_len, H, m.scale, _stream, opt);
    } else {
        _cache->prefillDev(l.index, out, wide, a.seq_list + r.from, a.q_starts + r.from, a.kv_lens + r.from, n, r.n_rows, r.max_q_len,
                           r.max_kv_len, H, m.scale, _stream, opt);
    }
    kernels::linear_heads(_stream, _dtype, _mix->memory() + r.row * l.n_mix * _elem, out + r.row * H * m.kv_rank * _elem, l.uv, r.n_rows, H,
                          m.vdim, m.kv_rank, false, H * m.kv_rank, m.kv_rank, l.n_mix, m.vdim);
#else
    (void)l, (void)a, (void)s, (void)r;
#endif
}

// Sequences whose contexts' rows become keys and values
void Folivik::expandedRange(const Layer &l, const StepArrays &a, const StepShape &s, const LatentRange &r) {
#ifdef ENABLE_NVIDIA_API
    (void)s;
    const LlaisysLatentAttentionMeta &m = l.meta.latent;
    const size_t H = m.heads, row = m.kv_rank + m.rot_dim, dim = m.dim + m.rot_dim, n = r.to - r.from;
    const int32_t *starts = reinterpret_cast<const int32_t *>(_page_starts->memory()) + r.from;
    const float *table = reinterpret_cast<const float *>(_rotary[l.rotary].table->memory()) + r.row * m.rot_dim;
    std::byte *context = _context->memory(), *q = _q->memory() + r.row * H * dim * _elem;
    _cache->latentGatherDev(l.index, context, int64_t(row), a.seq_list + r.from, starts, a.kv_lens + r.from, n, r.max_kv_len, _stream);
    kernels::fill_zero(_stream, context + (r.tokens - kTailRows) * row * _elem, kTailRows * row * _elem);
    kernels::linear(_stream, _dtype, _keys->memory(), context, l.uk, nullptr, r.tokens, H * m.dim, m.kv_rank, false, row);
    kernels::linear(_stream, _dtype, _values->memory(), context, l.uv, nullptr, r.tokens, H * m.vdim, m.kv_rank, false, row);
    kernels::rotate_pairs(_stream, _dtype, q, dim, m.dim, q, m.dim, m.rot_dim, table, r.n_rows, H);
    kernels::ExpandedArgs e;
    e.q = _q->memory();
    e.k = _keys->memory();
    e.k_shared = context + m.kv_rank * _elem;
    e.shared_stride = int64_t(row);
    e.v = _values->memory();
    e.tokens = int64_t(r.tokens);
    e.nh = int32_t(H);
    e.dim = int32_t(m.dim);
    e.rot_dim = int32_t(m.rot_dim);
    e.vdim = int32_t(m.vdim);
    e.page_starts = starts;
    e.q_starts = a.q_starts + r.from;
    e.kv_lens = a.kv_lens + r.from;
    e.n_seqs = int32_t(n);
    e.scale = m.scale;
    e.out = _mix->memory();
    e.out_stride = int64_t(l.n_mix);
    e.row_scale = reinterpret_cast<const float *>(_scale->memory());
    _cache->expandedDev(e, _stream);
#else
    (void)l, (void)a, (void)s, (void)r;
#endif
}

// Cuts a step's sequences into ranges, and makes room for the contexts of those that are expanded.
void Folivik::planLatents(const StepShape &s) {
    _ranges.clear();
    size_t row = 0, keys = 0, values = 0, tokens = 0;
    for (const Layer &l : _layers) {
        const LlaisysLatentAttentionMeta &m = l.meta.latent;
        if (l.meta.mixer == LLAISYS_FOLIVIK_LATENT && _cache->canExpand(l.index, m.dim, m.rot_dim, m.vdim)) {
            row = std::max(row, m.kv_rank + m.rot_dim);
            keys = std::max(keys, m.heads * m.dim);
            values = std::max(values, m.heads * m.vdim);
        }
    }
    if (row == 0 || s.decode_only) {
        return;
    }
    _page_starts_host.assign(s.n_seqs, -1);
    bool any = false;
    for (size_t i = 0; i < s.n_seqs; ++i) {
        const size_t first = size_t(s.host_q_starts[i]), n = size_t(s.host_q_starts[i + 1]) - first, len = size_t(s.host_kv_lens[i]);
        const size_t padded = (len + 15) / 16 * 16;
        const bool expanded = n >= kExpandFrom;
        if (_ranges.empty() || _ranges.back().expanded != expanded || (expanded && _ranges.back().tokens + padded > kPassTokens)) {
            _ranges.push_back(LatentRange{expanded, i, i, first, 0, 0, 0, expanded ? kTailRows : 0});
        }
        LatentRange &r = _ranges.back();
        if (expanded) {
            _page_starts_host[i] = int32_t((r.tokens - kTailRows) / 16);
            r.tokens += padded;
            any = true;
        }
        r.to = i + 1;
        r.n_rows += n;
        r.max_q_len = std::max(r.max_q_len, n);
        r.max_kv_len = std::max(r.max_kv_len, len);
        tokens = std::max(tokens, r.tokens);
    }
    if (!any) {
        return;
    }
    auto &rt = enter();
    auto grow = [&](core::storage_t &block, size_t bytes) {
        if (!block || block->size() < bytes) {
            block = rt.allocateDeviceStorage(bytes);
        }
    };
    grow(_page_starts, s.n_seqs * sizeof(int32_t));
    grow(_context, tokens * row * _elem);
    grow(_keys, tokens * keys * _elem);
    grow(_values, tokens * values * _elem);
    copyToDevice(_page_starts->memory(), _page_starts_host.data(), s.n_seqs * sizeof(int32_t));
}

void Folivik::windowAttention(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysFadingAttentionMeta &m = l.meta.attn;
    kernels::NormAppendArgs n;
    n.proj = _proj->memory();
    n.row_stride = int64_t(l.n_proj);
    n.q_at = int64_t(l.at[0]);
    n.k_at = int64_t(l.at[1]);
    n.v_at = int64_t(l.at[2]);
    n.gate_at = -1;
    n.q_norm = l.q_norm;
    n.k_norm = l.k_norm;
    n.eps = _meta.eps;
    n.head_scale = l.temp;
    n.q_out = _q->memory();
    n.seq_ids = a.seq32;
    n.positions = a.pos32;
    n.n_rows = s.n_tokens;
    n.nh = int32_t(m.heads);
    _cache->normAppendDev(l.index, n, _stream);
    kv::AttnOptions opt;
    opt.window = m.window;
    opt.fade_a = l.fade_a;
    opt.fade_b = l.fade_b;
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

void Folivik::stateSpace(const Layer &l, const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysStateSpaceMixerMeta &m = l.meta.ssm;
    kernels::StateSpaceArgs g;
    g.proj = _proj->memory();
    g.row_stride = int64_t(l.n_proj);
    g.z_at = int64_t(l.at[0]);
    g.x_at = int64_t(l.at[1]);
    g.dt_at = int64_t(l.at[2]);
    g.conv_w = l.conv_w;
    g.conv_b = l.conv_b;
    g.norm_w = l.norm_w;
    g.a_log = l.a_log;
    g.dt_bias = l.dt_bias;
    g.d_skip = l.d_skip;
    g.taps = int32_t(m.taps);
    g.heads = int32_t(m.heads);
    g.groups = int32_t(m.groups);
    g.dk = int32_t(m.state);
    g.dv = int32_t(m.vdim);
    g.norm_groups = int32_t(m.norm_groups);
    g.eps = _meta.eps;
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
    g.segments = _segments ? reinterpret_cast<float *>(_segments->memory()) : nullptr;
    g.segment_floats = _segments ? _segments->size() / sizeof(float) : 0;
    if (s.decode_only) {
        kernels::state_space_decode(_stream, _dtype, g);
    } else {
        kernels::state_space_chunk(_stream, _dtype, g);
    }
#else
    (void)l, (void)a, (void)s;
#endif
}

// h holds the norm of x; afterwards that of the next layer (next_gain != null)
void Folivik::experts(const Layer &l, const StepShape &s, const float *next_gain) {
#ifdef ENABLE_NVIDIA_API
    const LlaisysExpertLayerMeta &m = l.meta.mlp;
    const size_t T = s.n_tokens, W = _meta.width, n = m.experts + m.identity;
    float *x = reinterpret_cast<float *>(_x->memory()), *logits = reinterpret_cast<float *>(_logits_e->memory());
    std::byte *h = _h->memory();
    kernels::linear_f32(_stream, _dtype, logits, h, l.router, T, n, W, false);
    kernels::ExpertArgs e;
    e.experts = int32_t(m.experts);
    e.identity = int32_t(m.identity);
    e.top = int32_t(m.top);
    e.groups = int32_t(m.groups);
    e.keep = int32_t(m.keep);
    e.scale = m.scale;
    e.width = int32_t(W);
    e.ff = int32_t(l.ff);
    e.gate_up = l.gate_up;
    e.down = l.down;
    e.correction = l.correction;
    e.logits = logits;
    e.h = h;
    e.n_rows = int32_t(T);
    e.chosen = reinterpret_cast<int32_t *>(_choice->memory());
    e.weights = reinterpret_cast<float *>(e.chosen + T * m.top);
    e.place = e.chosen + 2 * T * m.top;
    e.line = e.chosen + 3 * T * m.top;
    e.counts = reinterpret_cast<int32_t *>(_counts->memory());
    e.rows = _rows->memory();
    e.act = _act->memory();
    e.out = _expert_out->memory();
    kernels::experts_route(_stream, _dtype, e);
    if (m.shared_ff != 0) {
        kernels::linear(_stream, _dtype, _proj->memory(), h, l.shared_gate_up, nullptr, T, 2 * l.shared_ff, W);
        kernels::swiglu_packed(_stream, _dtype, _shared->memory(), _proj->memory(), T, l.shared_ff);
        kernels::linear_f32(_stream, _dtype, x, _shared->memory(), l.shared_down, T, W, l.shared_ff, true);
    }
    kernels::experts_apply(_stream, _dtype, e);
    kernels::experts_combine(_stream, _dtype, e, x, next_gain != nullptr ? h : nullptr, next_gain, _meta.eps);
#else
    (void)l, (void)s, (void)next_gain;
#endif
}

void Folivik::forward(const StepArrays &a, const StepShape &s) {
#ifdef ENABLE_NVIDIA_API
    const size_t T = s.n_tokens, W = _meta.width;
    float *x = reinterpret_cast<float *>(_x->memory());
    std::byte *h = _h->memory();
    beginRecord();
    if (_counts) {
        kernels::fill_zero(_stream, _counts->memory(), _counts->size()); // (every layer leaves it zero; a step that failed may not have)
    }
    kernels::embed_scaled(_stream, _dtype, x, nullptr, 0, a.tokens, _embed, 1.f, T, W, _meta.voc);
    for (const Rotary &r : _rotary) {
        kernels::rotary_table(_stream, reinterpret_cast<float *>(r.table->memory()), a.pos32, reinterpret_cast<const double *>(r.freq->memory()),
                              T, r.dims / 2);
    }
    planLatents(s);
    bool normed = false; // h holds the norm of x that the coming layer reads
    for (size_t i = 0; i < _layers.size(); ++i) {
        const Layer &l = _layers[i];
        if (!normed) {
            kernels::stream_rms_norm_gain(_stream, _dtype, h, x, nullptr, l.norm1, _meta.eps, T, W);
        }
        kernels::linear(_stream, _dtype, _proj->memory(), h, l.proj, nullptr, T, l.n_proj, W);
        switch (l.meta.mixer) {
        case LLAISYS_FOLIVIK_LATENT:
            latentAttention(l, a, s);
            break;
        case LLAISYS_FOLIVIK_ATTENTION:
            windowAttention(l, a, s);
            break;
        default:
            stateSpace(l, a, s);
            break;
        }
        kernels::linear_f32(_stream, _dtype, x, _mix->memory(), l.out, T, W, l.n_mix, true);
        normed = false;
        if (l.meta.mlp.top != 0) {
            kernels::stream_rms_norm_gain(_stream, _dtype, h, x, nullptr, l.norm2, _meta.eps, T, W);
            normed = i + 1 < _layers.size();
            experts(l, s, normed ? _layers[i + 1].norm1 : nullptr);
        }
        recordLayer(x, T * W);
    }
    if (s.n_out == 0) {
        return;
    }
    std::byte *h_out = _h_out->memory();
    float *logits = reinterpret_cast<float *>(_logits->memory());
    kernels::stream_rms_norm_gain(_stream, _dtype, h_out, x, s.out_is_all ? nullptr : a.out_rows, _final_norm, _meta.eps, s.n_out, W);
    kernels::linear_f32(_stream, _dtype, logits, h_out, _head, s.n_out, _meta.voc, W, false);
    kernels::softcap_argmax(_stream, logits, 0.f, a.next, s.n_out, _meta.voc, _argmax_scratch->memory());
#else
    (void)a, (void)s;
    failModel(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
}

} // namespace llaisys::models
