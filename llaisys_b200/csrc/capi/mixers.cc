// extern "C" thunks of include/llaisys/mixers.h.
#include "llaisys/mixers.h"

#include "../core/core.hpp"
#include "paged_kv_handle.hpp"
#include "status.hpp"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

using llaisys::capi::guarded;

namespace {
int bad(const char *what) {
    llaisys::kernels::set_last_error(what);
    return LLAISYS_E_INVALID;
}
} // namespace

extern "C" {

int llaisysPagedKVCreateLayers(llaisysPagedKV_t *kv_out, llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype,
                               size_t nlayer, const size_t *nkvh, const size_t *k_dim, const size_t *v_dim, size_t num_pages,
                               size_t page_size, size_t max_seqs, size_t max_pages_per_seq) {
    if (kv_out == nullptr || nkvh == nullptr || k_dim == nullptr || v_dim == nullptr) {
        return bad("paged KV: null argument");
    }
    return guarded([&] {
        *kv_out = nullptr;
        llaisys::kv::PagedKVConfig cfg;
        cfg.device_type = device_type;
        cfg.device_id = device_id;
        cfg.dtype = dtype;
        cfg.nlayer = nlayer;
        for (size_t l = 0; l < nlayer; ++l) {
            cfg.layers.push_back(llaisys::kv::KVLayerShape{nkvh[l], k_dim[l], v_dim[l]});
        }
        cfg.num_pages = num_pages;
        cfg.page_size = page_size;
        cfg.max_seqs = max_seqs;
        cfg.max_pages_per_seq = max_pages_per_seq;
        *kv_out = new LlaisysPagedKV(cfg);
    });
}

int llaisysPagedKVCreateLatents(llaisysPagedKV_t *kv_out, llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype,
                                size_t nlayer, const size_t *rank, const size_t *rot_dim, size_t num_pages, size_t page_size,
                                size_t max_seqs, size_t max_pages_per_seq) {
    if (kv_out == nullptr || rank == nullptr || rot_dim == nullptr) {
        return bad("paged KV: null argument");
    }
    return guarded([&] {
        *kv_out = nullptr;
        llaisys::kv::PagedKVConfig cfg;
        cfg.device_type = device_type;
        cfg.device_id = device_id;
        cfg.dtype = dtype;
        cfg.nlayer = nlayer;
        for (size_t l = 0; l < nlayer; ++l) {
            cfg.layers.push_back(llaisys::kv::KVLayerShape{1, rank[l] + rot_dim[l], rank[l], true});
        }
        cfg.num_pages = num_pages;
        cfg.page_size = page_size;
        cfg.max_seqs = max_seqs;
        cfg.max_pages_per_seq = max_pages_per_seq;
        *kv_out = new LlaisysPagedKV(cfg);
    });
}

int llaisysPagedKVLatentAppendDev(llaisysPagedKV_t kv, size_t layer, const LlaisysLatentAppend *a, llaisysStream_t stream) {
    if (kv == nullptr || a == nullptr || a->proj == nullptr || a->q_norm == nullptr || a->kv_norm == nullptr || a->q_latent == nullptr ||
        a->seq_ids_dev == nullptr || a->positions_dev == nullptr || (a->rot_dims != 0 && a->rot_table == nullptr)) {
        return bad("paged KV latent append: null argument");
    }
    return guarded([&] {
        llaisys::kernels::LatentAppendArgs n;
        n.proj = a->proj;
        n.row_stride = a->row_stride;
        n.q_at = a->q_at;
        n.kv_at = a->kv_at;
        n.gate_at = a->gate_at;
        n.q_rank = int32_t(a->q_rank);
        n.rank = int32_t(a->rank);
        n.rot_dims = int32_t(a->rot_dims);
        n.nh = int32_t(a->nh);
        n.q_norm = a->q_norm;
        n.kv_norm = a->kv_norm;
        n.eps = a->eps;
        n.rot_table = a->rot_table;
        n.q_latent = a->q_latent;
        n.q_latent_stride = a->q_latent_stride;
        n.row_scale = a->row_scale;
        n.seq_ids = a->seq_ids_dev;
        n.positions = a->positions_dev;
        n.n_rows = a->n_rows;
        kv->impl.latentAppendDev(layer, n, stream);
    });
}

int llaisysPagedKVLatentGatherDev(llaisysPagedKV_t kv, size_t layer, void *out, int64_t out_stride, const int32_t *seq_ids_dev,
                                  const int32_t *page_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t max_kv_len,
                                  llaisysStream_t stream) {
    if (kv == nullptr || out == nullptr || seq_ids_dev == nullptr || page_starts_dev == nullptr || kv_lens_dev == nullptr) {
        return bad("paged KV latent gather: null argument");
    }
    return guarded([&] { kv->impl.latentGatherDev(layer, out, out_stride, seq_ids_dev, page_starts_dev, kv_lens_dev, n_seqs, max_kv_len, stream); });
}

int llaisysPagedAttentionExpandedDev(llaisysPagedKV_t kv, const LlaisysExpandedAttention *a, llaisysStream_t stream) {
    if (kv == nullptr || a == nullptr || a->q == nullptr || a->k == nullptr || a->k_shared == nullptr || a->v == nullptr || a->out == nullptr ||
        a->page_starts_dev == nullptr || a->q_starts_dev == nullptr || a->kv_lens_dev == nullptr) {
        return bad("expanded attention: null argument");
    }
    return guarded([&] {
        llaisys::kernels::ExpandedArgs e;
        e.q = a->q;
        e.k = a->k;
        e.k_shared = a->k_shared;
        e.shared_stride = a->shared_stride;
        e.v = a->v;
        e.tokens = int64_t(a->tokens);
        e.nh = int32_t(a->nh);
        e.dim = int32_t(a->dim);
        e.rot_dim = int32_t(a->rot_dim);
        e.vdim = int32_t(a->vdim);
        e.page_starts = a->page_starts_dev;
        e.q_starts = a->q_starts_dev;
        e.kv_lens = a->kv_lens_dev;
        e.n_seqs = int32_t(a->n_seqs);
        e.scale = a->scale;
        e.out = a->out;
        e.out_stride = a->out_stride;
        e.row_scale = a->row_scale;
        kv->impl.expandedDev(e, stream);
    });
}

int llaisysRotatePairsDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, void *out, size_t out_dim, size_t out_at,
                          const void *q, size_t dim, size_t rot_dims, const float *rot_table, size_t n_rows, size_t nh, llaisysStream_t stream) {
    if (out == nullptr || q == nullptr || rot_table == nullptr) {
        return bad("rotate pairs: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("rotate pairs: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::rotate_pairs(stream, dtype, out, out_dim, out_at, q, dim, rot_dims, rot_table, n_rows, nh);
#else
        (void)device_id, (void)dtype, (void)out_dim, (void)out_at, (void)dim, (void)rot_dims, (void)n_rows, (void)nh, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysStateSpaceDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const LlaisysStateSpace *a, int decode,
                         llaisysStream_t stream) {
    if (a == nullptr || a->proj == nullptr || a->conv_w == nullptr || a->conv_b == nullptr || a->norm_w == nullptr || a->a_log == nullptr ||
        a->dt_bias == nullptr || a->d_skip == nullptr || a->state == nullptr || a->seq_ids_dev == nullptr || a->kv_lens_dev == nullptr ||
        a->out == nullptr || a->scratch == nullptr || (decode == 0 && a->q_starts_dev == nullptr)) {
        return bad("state space: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("state space: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::StateSpaceArgs g;
        g.proj = a->proj;
        g.row_stride = a->row_stride;
        g.z_at = a->z_at;
        g.x_at = a->x_at;
        g.dt_at = a->dt_at;
        g.conv_w = a->conv_w;
        g.conv_b = a->conv_b;
        g.norm_w = a->norm_w;
        g.a_log = a->a_log;
        g.dt_bias = a->dt_bias;
        g.d_skip = a->d_skip;
        g.taps = int32_t(a->taps);
        g.heads = int32_t(a->heads);
        g.groups = int32_t(a->groups);
        g.dk = int32_t(a->dk);
        g.dv = int32_t(a->dv);
        g.norm_groups = int32_t(a->norm_groups);
        g.eps = a->eps;
        g.state = a->state;
        g.slot_stride = a->slot_stride;
        g.seq_ids = a->seq_ids_dev;
        g.q_starts = a->q_starts_dev;
        g.kv_lens = a->kv_lens_dev;
        g.n_seqs = int32_t(a->n_seqs);
        g.n_rows = int32_t(a->n_rows);
        g.max_q_len = int32_t(a->max_q_len);
        g.out = a->out;
        g.out_stride = a->out_stride;
        g.scratch = a->scratch;
        g.scratch_floats = a->scratch_floats;
        g.segments = a->scratch_segments;
        g.segment_floats = a->scratch_segment_floats;
        if (decode != 0) {
            llaisys::kernels::state_space_decode(stream, dtype, g);
        } else {
            llaisys::kernels::state_space_chunk(stream, dtype, g);
        }
#else
        (void)dtype, (void)device_id, (void)decode, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

void llaisysStateSpaceSizes(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t groups, size_t dk, size_t dv, size_t taps,
                            size_t *state_floats, size_t *scratch_floats, size_t *segment_floats) {
    size_t state = 0, scratch = 0, segments = 0;
#ifdef ENABLE_NVIDIA_API
    state = llaisys::kernels::state_space_state_floats(heads, groups, dk, dv, taps);
    scratch = llaisys::kernels::state_space_scratch_floats(dtype, n_rows, heads, groups, dk, dv);
    segments = llaisys::kernels::state_space_segment_floats(dtype, heads, dk, dv);
#else
    (void)dtype, (void)n_rows, (void)heads, (void)groups, (void)dk, (void)dv, (void)taps;
#endif
    if (state_floats != nullptr) {
        *state_floats = state;
    }
    if (scratch_floats != nullptr) {
        *scratch_floats = scratch;
    }
    if (segment_floats != nullptr) {
        *segment_floats = segments;
    }
}

int llaisysExpertsDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const LlaisysExperts *a, llaisysStream_t stream) {
    if (a == nullptr || a->gate_up == nullptr || a->down == nullptr || a->correction == nullptr || a->logits == nullptr || a->h == nullptr ||
        a->chosen == nullptr || a->weights == nullptr || a->place == nullptr || a->counts == nullptr || a->line == nullptr || a->rows == nullptr ||
        a->act == nullptr || a->out == nullptr || a->x == nullptr || (a->next != nullptr && a->gain == nullptr)) {
        return bad("experts: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("experts: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::ExpertArgs e;
        e.experts = int32_t(a->experts);
        e.identity = int32_t(a->identity);
        e.top = int32_t(a->top);
        e.groups = int32_t(a->groups);
        e.keep = int32_t(a->keep);
        e.scale = a->scale;
        e.width = int32_t(a->width);
        e.ff = int32_t(a->ff);
        e.gate_up = a->gate_up;
        e.down = a->down;
        e.correction = a->correction;
        e.logits = a->logits;
        e.h = a->h;
        e.n_rows = int32_t(a->n_rows);
        e.chosen = a->chosen;
        e.weights = a->weights;
        e.place = a->place;
        e.counts = a->counts;
        e.line = a->line;
        e.rows = a->rows;
        e.act = a->act;
        e.out = a->out;
        llaisys::kernels::experts_route(stream, dtype, e);
        llaisys::kernels::experts_apply(stream, dtype, e);
        llaisys::kernels::experts_combine(stream, dtype, e, a->x, a->next, a->gain, a->eps);
#else
        (void)dtype, (void)device_id, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysPagedKVNormAppendDev(llaisysPagedKV_t kv, size_t layer, const LlaisysNormAppend *a, llaisysStream_t stream) {
    if (kv == nullptr || a == nullptr) {
        return bad("paged KV norm append: null argument");
    }
    return guarded([&] {
        llaisys::kernels::NormAppendArgs n;
        n.proj = a->proj;
        n.row_stride = a->row_stride;
        n.q_at = a->q_at;
        n.k_at = a->k_at;
        n.v_at = a->v_at;
        n.gate_at = a->gate_at;
        n.q_norm = a->q_norm;
        n.k_norm = a->k_norm;
        n.eps = a->eps;
        n.rot_dims = int32_t(a->rot_dims);
        n.rot_table = a->rot_table;
        n.gate_scale = a->gate_scale;
        n.q_out = a->q_out;
        n.row_scale = a->row_scale;
        n.seq_ids = a->seq_ids_dev;
        n.positions = a->positions_dev;
        n.n_rows = a->n_rows;
        n.nh = int32_t(a->nh);
        n.row_norm = a->row_norm;
        n.bias = a->bias;
        n.temp_coef = a->temp_coef;
        n.temp_every = a->temp_every;
        n.head_scale = a->head_scale;
        kv->impl.normAppendDev(layer, n, stream);
    });
}

int llaisysPagedAttentionOptDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q, const int32_t *seq_ids_dev,
                                const int32_t *q_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t total_q,
                                size_t max_q_len, size_t max_kv_len, size_t nh, float scale, size_t window, size_t keep_first,
                                const float *row_scale, size_t row_stride, llaisysStream_t stream) {
    if (kv == nullptr) {
        return bad("paged attention: null cache handle");
    }
    return guarded([&] {
        llaisys::kv::AttnOptions opt;
        opt.window = window;
        opt.keep_first = keep_first;
        opt.row_scale = row_scale;
        opt.row_stride = row_stride;
        if (q_starts_dev == nullptr) {
            kv->impl.decodeDev(layer, out, nullptr, q, seq_ids_dev, kv_lens_dev, n_seqs, max_kv_len, nh, scale, stream, opt);
        } else {
            kv->impl.prefillDev(layer, out, q, seq_ids_dev, q_starts_dev, kv_lens_dev, n_seqs, total_q, max_q_len, max_kv_len, nh,
                                scale, stream, opt);
        }
    });
}

int llaisysPagedAttentionFadeDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q, const int32_t *seq_ids_dev,
                                 const int32_t *q_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t total_q, size_t max_q_len,
                                 size_t max_kv_len, size_t nh, float scale, size_t window, const float *fade_a, const float *fade_b,
                                 size_t row_stride, llaisysStream_t stream) {
    if (kv == nullptr || fade_a == nullptr || fade_b == nullptr) {
        return bad("attention with a distance penalty: null argument");
    }
    return guarded([&] {
        llaisys::kv::AttnOptions opt;
        opt.window = window;
        opt.fade_a = fade_a;
        opt.fade_b = fade_b;
        opt.row_stride = row_stride;
        if (q_starts_dev == nullptr) {
            kv->impl.decodeDev(layer, out, nullptr, q, seq_ids_dev, kv_lens_dev, n_seqs, max_kv_len, nh, scale, stream, opt);
        } else {
            kv->impl.prefillDev(layer, out, q, seq_ids_dev, q_starts_dev, kv_lens_dev, n_seqs, total_q, max_q_len, max_kv_len, nh,
                                scale, stream, opt);
        }
    });
}

int llaisysPagedAttentionGatesDev(llaisysPagedKV_t kv, size_t layer, void *out, const void *q, const int32_t *seq_ids_dev,
                                  const int32_t *q_starts_dev, const int32_t *kv_lens_dev, size_t n_seqs, size_t total_q,
                                  size_t max_q_len, size_t max_kv_len, size_t nh, float scale, size_t window,
                                  const LlaisysGates *gates, size_t row_stride, llaisysStream_t stream) {
    if (kv == nullptr || gates == nullptr) {
        return bad("gated attention: null argument");
    }
    return guarded([&] {
        llaisys::kernels::GateArgs g;
        g.softcap = gates->softcap;
        g.slopes = gates->slopes;
        g.bias = gates->bias;
        g.talk = gates->talk;
        llaisys::kv::AttnOptions opt;
        opt.window = window;
        opt.row_stride = row_stride;
        opt.gates = &g;
        if (q_starts_dev == nullptr) {
            kv->impl.decodeDev(layer, out, nullptr, q, seq_ids_dev, kv_lens_dev, n_seqs, max_kv_len, nh, scale, stream, opt);
        } else {
            kv->impl.prefillDev(layer, out, q, seq_ids_dev, q_starts_dev, kv_lens_dev, n_seqs, total_q, max_q_len, max_kv_len, nh,
                                scale, stream, opt);
        }
    });
}

size_t llaisysMinGruScratchFloats(size_t n_rows, size_t width) {
#ifdef ENABLE_NVIDIA_API
    return llaisys::kernels::min_gru_scratch_floats(n_rows, width);
#else
    (void)n_rows, (void)width;
    return 0;
#endif
}

int llaisysMinGruDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const LlaisysMinGru *a, int decode,
                     llaisysStream_t stream) {
    if (a == nullptr || a->proj == nullptr || a->bias_z == nullptr || a->bias_x == nullptr || a->state == nullptr ||
        a->seq_ids_dev == nullptr || a->kv_lens_dev == nullptr || a->out == nullptr || (decode == 0 && a->q_starts_dev == nullptr)) {
        return bad("minGRU: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("minGRU: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::MinGruArgs g;
        g.proj = a->proj;
        g.row_stride = a->row_stride;
        g.z_at = a->z_at;
        g.x_at = a->x_at;
        g.g_at = a->g_at;
        g.bias_z = a->bias_z;
        g.bias_x = a->bias_x;
        g.width = int32_t(a->width);
        g.state = a->state;
        g.slot_stride = a->slot_stride;
        g.seq_ids = a->seq_ids_dev;
        g.q_starts = a->q_starts_dev;
        g.kv_lens = a->kv_lens_dev;
        g.n_seqs = int32_t(a->n_seqs);
        g.n_rows = int32_t(a->n_rows);
        g.max_q_len = int32_t(a->max_q_len);
        g.out = a->out;
        g.out_stride = a->out_stride;
        g.scratch = a->scratch;
        g.scratch_floats = a->scratch_floats;
        if (decode != 0) {
            llaisys::kernels::min_gru_decode(stream, dtype, g);
        } else {
            llaisys::kernels::min_gru_chunk(stream, dtype, g);
        }
#else
        (void)dtype, (void)device_id, (void)decode, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysGatedLinearDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const LlaisysGatedLinear *a,
                          int decode, llaisysStream_t stream) {
    if (a == nullptr || a->proj == nullptr || a->decay_w == nullptr || a->decay_b == nullptr || a->norm_w == nullptr ||
        a->state == nullptr || a->seq_ids_dev == nullptr || a->kv_lens_dev == nullptr || a->out == nullptr ||
        (decode == 0 && a->q_starts_dev == nullptr)) {
        return bad("gated linear attention: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("gated linear attention: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::GatedLinearArgs g;
        g.proj = a->proj;
        g.row_stride = a->row_stride;
        g.q_at = a->q_at;
        g.k_at = a->k_at;
        g.v_at = a->v_at;
        g.g_at = a->g_at;
        g.z_at = a->z_at;
        g.decay_w = a->decay_w;
        g.decay_b = a->decay_b;
        g.norm_w = a->norm_w;
        g.tau = a->tau;
        g.q_scale = a->q_scale;
        g.eps = a->eps;
        g.out_scale = a->out_scale;
        g.heads = int32_t(a->heads);
        g.dk = int32_t(a->dk);
        g.dv = int32_t(a->dv);
        g.rank = int32_t(a->rank);
        g.state = a->state;
        g.slot_stride = a->slot_stride;
        g.seq_ids = a->seq_ids_dev;
        g.q_starts = a->q_starts_dev;
        g.kv_lens = a->kv_lens_dev;
        g.n_seqs = int32_t(a->n_seqs);
        g.n_rows = int32_t(a->n_rows);
        g.max_q_len = int32_t(a->max_q_len);
        g.out = a->out;
        g.out_stride = a->out_stride;
        g.raw = a->scratch_raw;
        g.decay = a->scratch_decay;
        g.segments = a->scratch_segments;
        g.segment_floats = a->scratch_segment_floats;
        if (decode != 0) {
            llaisys::kernels::gated_linear_decode(stream, dtype, g);
        } else {
            llaisys::kernels::gated_linear_chunk(stream, dtype, g);
        }
#else
        (void)dtype;
        (void)device_id;
        (void)decode;
        (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysRotaryTableDev(llaisysDeviceType_t device_type, int device_id, float *table, const int32_t *positions_dev,
                          const float *freq_dev, size_t n_rows, size_t half, llaisysStream_t stream) {
    if (table == nullptr || positions_dev == nullptr || freq_dev == nullptr) {
        return bad("rotary table: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("rotary table: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::rotary_table(stream, table, positions_dev, freq_dev, n_rows, half);
#else
        (void)device_id, (void)n_rows, (void)half, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysRotaryTableWideDev(llaisysDeviceType_t device_type, int device_id, float *table, const int32_t *positions_dev,
                              const double *freq_dev, size_t n_rows, size_t half, llaisysStream_t stream) {
    if (table == nullptr || positions_dev == nullptr || freq_dev == nullptr) {
        return bad("rotary table: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("rotary table: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::rotary_table(stream, table, positions_dev, freq_dev, n_rows, half);
#else
        (void)device_id, (void)n_rows, (void)half, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

int llaisysGatedDeltaDev(llaisysDeviceType_t device_type, int device_id, llaisysDataType_t dtype, const LlaisysGatedDelta *a,
                         int decode, llaisysStream_t stream) {
    if (a == nullptr || a->proj == nullptr || a->conv_q == nullptr || a->conv_k == nullptr || a->conv_v == nullptr ||
        a->a_log == nullptr || a->dt_bias == nullptr || a->norm_w == nullptr || a->gate == nullptr || a->state == nullptr ||
        a->seq_ids_dev == nullptr || a->kv_lens_dev == nullptr || a->out == nullptr ||
        (decode == 0 && (a->q_starts_dev == nullptr || a->scratch == nullptr))) {
        return bad("gated delta rule: null argument");
    }
    if (device_type != LLAISYS_DEVICE_NVIDIA) {
        llaisys::kernels::set_last_error("gated delta rule: NVIDIA devices only");
        return LLAISYS_E_UNSUPPORTED;
    }
    return guarded([&] {
#ifdef ENABLE_NVIDIA_API
        llaisys::core::context().setDevice(device_type, device_id);
        llaisys::kernels::GatedDeltaArgs g;
        g.proj = a->proj;
        g.row_stride = a->row_stride;
        g.q_at = a->q_at;
        g.k_at = a->k_at;
        g.v_at = a->v_at;
        g.b_at = a->b_at;
        g.a_at = a->a_at;
        g.conv_q = a->conv_q;
        g.conv_k = a->conv_k;
        g.conv_v = a->conv_v;
        g.taps = int32_t(a->taps);
        g.decay_w = a->decay_w;
        g.decay_ld = a->decay_ld;
        g.a_log = a->a_log;
        g.dt_bias = a->dt_bias;
        g.norm_w = a->norm_w;
        g.gate = a->gate;
        g.gate_stride = a->gate_stride;
        g.gate_silu = a->gate_silu;
        g.q_scale = a->q_scale;
        g.eps = a->eps;
        g.unit_eps = a->unit_eps;
        g.heads = int32_t(a->heads);
        g.kv_heads = int32_t(a->kv_heads);
        g.dk = int32_t(a->dk);
        g.dv = int32_t(a->dv);
        g.rank = int32_t(a->rank);
        g.state = a->state;
        g.slot_stride = a->slot_stride;
        g.seq_ids = a->seq_ids_dev;
        g.q_starts = a->q_starts_dev;
        g.kv_lens = a->kv_lens_dev;
        g.n_seqs = int32_t(a->n_seqs);
        g.n_rows = int32_t(a->n_rows);
        g.max_q_len = int32_t(a->max_q_len);
        g.out = a->out;
        g.out_stride = a->out_stride;
        g.scratch = a->scratch;
        g.scratch_floats = a->scratch_floats;
        g.segments = a->scratch_segments;
        g.segment_floats = a->scratch_segment_floats;
        if (decode != 0) {
            llaisys::kernels::gated_delta_decode(stream, dtype, g);
        } else {
            llaisys::kernels::gated_delta_chunk(stream, dtype, g);
        }
#else
        (void)dtype, (void)device_id, (void)decode, (void)stream;
        throw llaisys::kv::StatusError(LLAISYS_E_UNSUPPORTED, "this build has no NVIDIA backend");
#endif
    });
}

void llaisysGatedDeltaSizes(llaisysDataType_t dtype, size_t n_rows, size_t heads, size_t kv_heads, size_t dk, size_t dv, size_t taps,
                            size_t *state_floats, size_t *scratch_floats, size_t *segment_floats) {
    size_t state = 0, scratch = 0, segments = 0;
#ifdef ENABLE_NVIDIA_API
    state = llaisys::kernels::gated_delta_state_floats(heads, kv_heads, dk, dv, taps);
    scratch = llaisys::kernels::gated_delta_scratch_floats(dtype, n_rows, heads, kv_heads, dk, dv);
    segments = llaisys::kernels::gated_delta_segment_floats(dtype, heads, dk, dv);
#else
    (void)dtype, (void)n_rows, (void)heads, (void)kv_heads, (void)dk, (void)dv, (void)taps;
#endif
    if (state_floats != nullptr) {
        *state_floats = state;
    }
    if (scratch_floats != nullptr) {
        *scratch_floats = scratch;
    }
    if (segment_floats != nullptr) {
        *segment_floats = segments;
    }
}

size_t llaisysGatedLinearSegmentFloats(llaisysDataType_t dtype, size_t heads, size_t dk, size_t dv) {
#ifdef ENABLE_NVIDIA_API
    return llaisys::kernels::gated_linear_segment_floats(dtype, heads, dk, dv);
#else
    (void)dtype, (void)heads, (void)dk, (void)dv;
    return 0;
#endif
}

} // extern "C"
