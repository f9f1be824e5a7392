#include "qwen2.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "../cpu/cpu_kernels.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <cmath>

namespace llaisys::models {

namespace {
[[noreturn]] void fail(int code, const std::string &msg) { throw kv::StatusError(code, msg); }
} // namespace

// ---- construction -------------------------------------------------------------------------------------------------

namespace {
LlaisysQwen2Meta shard_meta(LlaisysQwen2Meta meta, int tp_rank, int tp_world) {
    if (tp_world < 1 || tp_rank < 0 || tp_rank >= tp_world) {
        fail(LLAISYS_E_INVALID, "qwen2: bad tensor-parallel rank or world size");
    }
    const size_t w = size_t(tp_world);
    if (meta.nkvh % w != 0 || meta.nh % w != 0 || meta.di % w != 0) {
        fail(LLAISYS_E_INVALID, "qwen2: the tensor-parallel world size must divide nkvh, nh and di");
    }
    meta.nh /= w;
    meta.nkvh /= w;
    meta.di /= w;
    return meta;
}
} // namespace

Qwen2::Qwen2(const LlaisysQwen2Meta &global_meta, llaisysDeviceType_t device, int device_id, int tp_rank, int tp_world)
    : Decoder("qwen2", device, device_id, global_meta.dtype, global_meta.dtype),
      _meta(shard_meta(global_meta, tp_rank, tp_world)), _tp_rank(tp_rank), _tp_world(tp_world) {
    const LlaisysQwen2Meta &meta = _meta;
    if (meta.nlayer == 0 || meta.hs == 0 || meta.nh == 0 || meta.nkvh == 0 || meta.dh == 0 || meta.di == 0 || meta.voc == 0 ||
        meta.nh % meta.nkvh != 0 || meta.dh % 2 != 0) {
        fail(LLAISYS_E_INVALID, "qwen2: inconsistent model dimensions");
    }
    enter();

    const size_t L = meta.nlayer, hs = meta.hs, qd = meta.nh * meta.dh, kd = meta.nkvh * meta.dh, di = meta.di;
    _weights.in_embed = makeWeight({meta.voc, hs});
    _weights.out_embed = makeWeight({meta.voc, hs});
    _weights.out_norm_w = makeWeight({hs});
    for (auto &v : _per_layer) {
        v.resize(L);
    }
    _qkv_w.resize(L);
    _qkv_b.resize(L);
    _gate_up_w.resize(L);
    const std::vector<std::byte> zeros((qd + 2 * kd) * _elem);
    for (size_t l = 0; l < L; ++l) {
        _qkv_w[l] = Tensor::create({qd + 2 * kd, hs}, meta.dtype, device, device_id);
        _qkv_b[l] = Tensor::create({qd + 2 * kd}, meta.dtype, device, device_id);
        _qkv_b[l]->load(zeros.data()); // a caller that loads no biases gets none
        _gate_up_w[l] = Tensor::create({2 * di, hs}, meta.dtype, device, device_id);
        _per_layer[0][l] = makeWeight({hs});
        _per_layer[1][l] = wrap(_qkv_w[l]->slice(0, 0, qd));
        _per_layer[2][l] = wrap(_qkv_b[l]->slice(0, 0, qd));
        _per_layer[3][l] = wrap(_qkv_w[l]->slice(0, qd, qd + kd));
        _per_layer[4][l] = wrap(_qkv_b[l]->slice(0, qd, qd + kd));
        _per_layer[5][l] = wrap(_qkv_w[l]->slice(0, qd + kd, qd + 2 * kd));
        _per_layer[6][l] = wrap(_qkv_b[l]->slice(0, qd + kd, qd + 2 * kd));
        _per_layer[7][l] = makeWeight({hs, qd});
        _per_layer[8][l] = makeWeight({hs});
        _per_layer[9][l] = wrap(_gate_up_w[l]->slice(0, 0, di));
        _per_layer[10][l] = wrap(_gate_up_w[l]->slice(0, di, 2 * di));
        _per_layer[11][l] = makeWeight({hs, di});
    }
    _weights.attn_norm_w = _per_layer[0].data();
    _weights.attn_q_w = _per_layer[1].data();
    _weights.attn_q_b = _per_layer[2].data();
    _weights.attn_k_w = _per_layer[3].data();
    _weights.attn_k_b = _per_layer[4].data();
    _weights.attn_v_w = _per_layer[5].data();
    _weights.attn_v_b = _per_layer[6].data();
    _weights.attn_o_w = _per_layer[7].data();
    _weights.mlp_norm_w = _per_layer[8].data();
    _weights.mlp_gate_w = _per_layer[9].data();
    _weights.mlp_up_w = _per_layer[10].data();
    _weights.mlp_down_w = _per_layer[11].data();
}

Qwen2::~Qwen2() {
    for (llaisysTensor_t h : _all_weights) {
        delete h;
    }
}

llaisysTensor_t Qwen2::wrap(tensor_t t) {
    auto *h = new LlaisysTensor{std::move(t)};
    _all_weights.push_back(h);
    return h;
}

llaisysTensor_t Qwen2::makeWeight(const std::vector<size_t> &shape) {
    return wrap(Tensor::create(shape, _meta.dtype, _device, _device_id));
}

std::vector<Qwen2::Layer> Qwen2::layerPointers() const {
    std::vector<Layer> layers(_meta.nlayer);
    for (size_t l = 0; l < _meta.nlayer; ++l) {
        auto p = [&](int w) { return static_cast<const std::byte *>(_per_layer[w][l]->tensor->data()); };
        auto packed = [](const tensor_t &t) { return static_cast<const std::byte *>(t->data()); };
        layers[l] = Layer{p(0), packed(_qkv_w[l]), packed(_qkv_b[l]), p(7), p(8), packed(_gate_up_w[l]), p(11)};
    }
    return layers;
}

// ---- workspace -------------------------------------------------------------------------------------------------------

kv::PagedKVConfig Qwen2::cacheShape() const {
    kv::PagedKVConfig cfg;
    cfg.nlayer = _meta.nlayer;
    cfg.nkvh = _meta.nkvh;
    cfg.head_dim = _meta.dh;
    return cfg;
}

void Qwen2::ensureActivations(size_t n_tokens, size_t n_out) {
    auto &rt = enter();
    if (n_tokens > _ws_tokens) {
        ++_generation;
        const size_t hs = _meta.hs, qd = _meta.nh * _meta.dh, kd = _meta.nkvh * _meta.dh;
        _x = rt.allocateDeviceStorage(n_tokens * hs * _elem);
        _h = rt.allocateDeviceStorage(n_tokens * hs * _elem);
        _qkv = rt.allocateDeviceStorage(n_tokens * (qd + 2 * kd) * _elem);
        _q = rt.allocateDeviceStorage(n_tokens * qd * _elem);
        _attn = rt.allocateDeviceStorage(n_tokens * qd * _elem);
        _gate_up = rt.allocateDeviceStorage(n_tokens * 2 * _meta.di * _elem);
        _act = rt.allocateDeviceStorage(n_tokens * _meta.di * _elem);
    }
    if (n_out > _ws_out) {
        _x_last = rt.allocateDeviceStorage(n_out * _meta.hs * _elem);
    }
}

// ---- operator shims ----------------------------------------------------------------------------------------------------

#ifdef ENABLE_NVIDIA_API
#define QWEN2_DISPATCH(CPU_CALL, CUDA_CALL) \
    if (_on_gpu) {                          \
        CUDA_CALL;                          \
    } else {                                \
        CPU_CALL;                           \
    }
#else
#define QWEN2_DISPATCH(CPU_CALL, CUDA_CALL) CPU_CALL;
#endif

void Qwen2::opEmbedding(void *out, const int64_t *idx, const void *w, size_t n, size_t d, size_t vocab) {
    QWEN2_DISPATCH(cpu::embedding(_elem, out, idx, w, n, d, vocab), kernels::embedding(_stream, _elem, out, idx, w, n, d, vocab));
}
void Qwen2::opLinear(void *out, const void *in, const void *w, size_t m, size_t n, size_t k, bool accumulate) {
    QWEN2_DISPATCH(cpu::linear(_meta.dtype, out, in, w, nullptr, m, n, k, accumulate),
                   kernels::linear(_stream, _meta.dtype, out, in, w, nullptr, m, n, k, accumulate));
}
void Qwen2::opRmsNorm(void *out, const void *in, const void *w, size_t rows, size_t d) {
    QWEN2_DISPATCH(cpu::rms_norm(_meta.dtype, out, in, w, _meta.epsilon, rows, d),
                   kernels::rms_norm(_stream, _meta.dtype, out, in, w, _meta.epsilon, rows, d));
}
void Qwen2::opSwigluPacked(void *out, const void *gate_up, size_t rows, size_t di) {
    QWEN2_DISPATCH(cpu::swiglu_packed(_meta.dtype, out, gate_up, rows, di),
                   kernels::swiglu_packed(_stream, _meta.dtype, out, gate_up, rows, di));
}
void Qwen2::opAdd(void *c, const void *a, const void *b, size_t n) {
    QWEN2_DISPATCH(cpu::add(_meta.dtype, c, a, b, n), kernels::add(_stream, _meta.dtype, c, a, b, n));
}

void Qwen2::setCollective(std::unique_ptr<comm::Collective> c) {
    if (!c || c->rank() != _tp_rank || c->world() != _tp_world) {
        fail(LLAISYS_E_INVALID, "qwen2: the collective's rank / world size differ from the model's");
    }
    _tp = std::move(c);
}

void Qwen2::projectIntoStream(void *x, void *tmp, const void *in, const void *w, size_t m, size_t n, size_t k) {
    if (_tp_world == 1) {
        opLinear(x, in, w, m, n, k, true); // the residual add folded into the projection
        return;
    }
    if (!_tp) {
        fail(LLAISYS_E_INVALID, "qwen2: a sharded model needs its all-reduce (llaisysQwen2ModelSetAllReduce...) before the first step");
    }
    opLinear(tmp, in, w, m, n, k);
    _tp->allReduceSum(tmp, m * n, _meta.dtype, _stream);
    opAdd(x, x, tmp, m * n);
}

void Qwen2::opArgmax(int64_t *idx, const void *vals, size_t rows, size_t n) {
    QWEN2_DISPATCH(cpu::argmax_rows(_meta.dtype, idx, nullptr, vals, rows, n),
                   kernels::argmax_rows_split(_stream, _meta.dtype, idx, vals, rows, n, _argmax_scratch->memory()));
}

// ---- the network ---------------------------------------------------------------------------------------------------------

void Qwen2::forward(const StepArrays &a, const StepShape &s) {
    const size_t T = s.n_tokens, n_seqs = s.n_seqs;
    const size_t hs = _meta.hs, qd = _meta.nh * _meta.dh, kd = _meta.nkvh * _meta.dh, di = _meta.di;
    const float scale = 1.f / std::sqrt(float(_meta.dh));
    std::byte *x = _x->memory(), *h = _h->memory(), *qkv = _qkv->memory(), *q = _q->memory();
    std::byte *attn = _attn->memory(), *gate_up = _gate_up->memory(), *act = _act->memory();
    const std::vector<Layer> layers = layerPointers();

    // Per layer: norm, packed q|k|v projection, [bias + rope + append], attention, output projection accumulated into the
    // residual stream, norm, packed gate|up projection, activation, down projection accumulated into the stream.
    opEmbedding(x, a.tokens, _weights.in_embed->tensor->data(), T, hs, _meta.voc);
    for (size_t l = 0; l < _meta.nlayer; ++l) {
        const Layer &w = layers[l];
        opRmsNorm(h, x, w.attn_norm, T, hs);
        opLinear(qkv, h, w.qkv_w, T, qd + 2 * kd, hs);
        _cache->ropeAppendDev(l, q, qkv, w.qkv_b, a.seq32, a.pos32, T, _meta.nh, _meta.theta, _stream);
        if (s.decode_only) {
            _cache->decodeDev(l, attn, nullptr, q, a.seq_list, a.kv_lens, n_seqs, s.max_kv_len, _meta.nh, scale, _stream);
        } else {
            _cache->prefillDev(l, attn, q, a.seq_list, a.q_starts, a.kv_lens, n_seqs, T, s.max_q_len, s.max_kv_len, _meta.nh,
                               scale, _stream);
        }
        projectIntoStream(x, h, attn, w.o_w, T, hs, qd);
        opRmsNorm(h, x, w.mlp_norm, T, hs);
        opLinear(gate_up, h, w.gate_up_w, T, 2 * di, hs);
        opSwigluPacked(act, gate_up, T, di);
        projectIntoStream(x, h, act, w.down_w, T, hs, di);
    }
    if (s.n_out == 0) {
        return;
    }
    // the rows that are asked for (the last token of every sequence) -> final norm -> vocabulary projection -> greedy choice
    const std::byte *last = x;
    if (!s.out_is_all) {
        opEmbedding(_x_last->memory(), a.out_rows, x, s.n_out, hs, T);
        last = _x_last->memory();
    }
    opRmsNorm(_x_last->memory(), last, _weights.out_norm_w->tensor->data(), s.n_out, hs);
    opLinear(_logits->memory(), _x_last->memory(), _weights.out_embed->tensor->data(), s.n_out, _meta.voc, hs);
    opArgmax(a.next, _logits->memory(), s.n_out, _meta.voc);
}

} // namespace llaisys::models
