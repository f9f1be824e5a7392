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
