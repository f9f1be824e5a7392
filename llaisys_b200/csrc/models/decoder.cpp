#include "decoder.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <algorithm>
#include <chrono>
#include <cstring>
#include <limits>

namespace llaisys::models {

namespace {
constexpr size_t kPageSize = 16;
constexpr size_t kNotLive = std::numeric_limits<size_t>::max();
size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }
} // namespace

Decoder::Decoder(const char *name, llaisysDeviceType_t device, int device_id, llaisysDataType_t dtype,
                 llaisysDataType_t logits_dtype)
    : _name(name), _device(device), _device_id(device_id), _dtype(dtype), _logits_dtype(logits_dtype) {
    if (dtype != LLAISYS_DTYPE_F32 && dtype != LLAISYS_DTYPE_F16 && dtype != LLAISYS_DTYPE_BF16) {
        failModel(LLAISYS_E_INVALID, "dtype must be F32, F16 or BF16");
    }
    _elem = utils::dsize(dtype);
    _on_gpu = device != LLAISYS_DEVICE_CPU;
    _stream = enter().stream();
}

Decoder::~Decoder() {
    dropStepGraphs();
    for (ModelObserver *o : std::vector<ModelObserver *>(_observers)) {
        o->modelDestroyed();
    }
}

void Decoder::removeObserver(ModelObserver *o) {
    _observers.erase(std::remove(_observers.begin(), _observers.end(), o), _observers.end());
}

void Decoder::failModel(int code, const std::string &msg) const {
    throw kv::StatusError(code, std::string(_name) + ": " + msg);
}

bool Decoder::loadTensor(const std::string &, llaisysDataType_t, const std::vector<size_t> &, const void *) {
    failModel(LLAISYS_E_UNSUPPORTED, "this model's weights are loaded through their handles");
}

void Decoder::recordStream(bool) { failModel(LLAISYS_E_UNSUPPORTED, "this model keeps no record of its stream"); }
size_t Decoder::layerStream(float *, size_t) { failModel(LLAISYS_E_UNSUPPORTED, "this model keeps no record of its stream"); }

void Decoder::dropStepGraphs() {
#ifdef ENABLE_NVIDIA_API
    for (StepGraph &g : _step_graphs) {
        if (g.exec != nullptr) {
            kernels::graph_destroy(g.exec);
        }
    }
#endif
    _step_graphs.clear();
}

core::Runtime &Decoder::enter() const {
    auto &ctx = core::context();
    ctx.setDevice(_device, _device_id);
    return ctx.runtime();
}

// ---- cache and sequences --------------------------------------------------------------------------------------------

void Decoder::configureCache(size_t max_seqs, size_t max_tokens, size_t pool_tokens) {
    if (max_seqs == 0 || max_tokens == 0) {
        failModel(LLAISYS_E_INVALID, "cache sizes must be positive");
    }
    kv::PagedKVConfig cfg = cacheShape();
    cfg.device_type = _device;
    cfg.device_id = _device_id;
    cfg.dtype = _dtype;
    cfg.page_size = kPageSize;
    cfg.max_seqs = max_seqs;
    cfg.max_pages_per_seq = (max_tokens + kPageSize - 1) / kPageSize;
    cfg.num_pages = pool_tokens == 0 ? cfg.max_seqs * cfg.max_pages_per_seq : (pool_tokens + kPageSize - 1) / kPageSize;
    dropStepGraphs();
    _cache.reset(); // the old pool first: two need not fit beside each other
    _state.reset();
    _seq_len.clear();
    _implicit_seq = -1;
    _cache = std::make_unique<kv::PagedKV>(cfg);
    const std::vector<size_t> state = stateShape();
    if (!state.empty()) {
        _state = std::make_unique<kv::StatePool>(_device, _device_id, max_seqs, state);
    }
    // [position-wise work + append] -> decode attention run as a programmatic pair: the attention kernel's set-up and its
    // copies of older pages overlap the append (which writes each sequence's last page only, as the overlap contract asks)
    _cache->setLaunchOverlap(_on_gpu);
    _max_tokens_per_seq = cfg.max_pages_per_seq * kPageSize;
    _seq_len.assign(max_seqs, kNotLive);
    _seq_last.assign(max_seqs, -1);
    _seq_tokens.assign(max_seqs, {});
}

size_t &Decoder::seqLen(int32_t seq) {
    if (!_cache || seq < 0 || size_t(seq) >= _seq_len.size() || _seq_len[seq] == kNotLive) {
        failModel(LLAISYS_E_NO_SEQ, "sequence " + std::to_string(seq) + " does not exist");
    }
    return _seq_len[seq];
}

int32_t Decoder::seqAdd() {
    if (!_cache) {
        failModel(LLAISYS_E_INVALID, "configure the cache first");
    }
    const int32_t s = _cache->seqAdd();
    _seq_len[s] = 0;
    _seq_last[s] = -1;
    _seq_tokens[s].clear();
    return s;
}

int32_t Decoder::seqAddWithPrefix(const int64_t *tokens, size_t n, size_t *matched) {
    const int32_t s = seqAdd();
    size_t got = 0;
    if (n > 1 && tokens != nullptr && !_state) {
        try {
            got = _cache->seqMatchPrefix(s, tokens, n - 1); // whole pages inside the first n - 1 tokens
        } catch (...) {
            seqFree(s);
            throw;
        }
        _seq_tokens[s].assign(tokens, tokens + got);
        _seq_last[s] = got != 0 ? tokens[got - 1] : -1;
    }
    _seq_len[s] = got;
    if (matched != nullptr) {
        *matched = got;
    }
    return s;
}

void Decoder::seqReserve(int32_t seq, size_t n_tokens) {
    seqLen(seq);
    if (n_tokens > _max_tokens_per_seq) {
        failModel(LLAISYS_E_INVALID, "sequence would exceed the configured maximum length");
    }
    _cache->seqReserve(seq, n_tokens);
}

// The sequence now holds K/V for n more tokens: remember their ids and publish the pages they completed.
void Decoder::recordTokens(int32_t seq, const int64_t *tokens, size_t n) {
    _seq_last[seq] = tokens[n - 1];
    if (_state) {
        return; // pages of a network with recurrent state are not a whole prefix: never shared
    }
    std::vector<int64_t> &held = _seq_tokens[seq];
    const size_t before = held.size() / kPageSize;
    held.insert(held.end(), tokens, tokens + n);
    if (held.size() / kPageSize != before) {
        _cache->seqPublish(seq, held.data(), held.size());
    }
}

void Decoder::seqFree(int32_t seq) {
    seqLen(seq);
    _cache->seqFree(seq);
    _seq_len[seq] = kNotLive;
    _seq_tokens[seq].clear();
    if (seq == _implicit_seq) {
        _implicit_seq = -1;
    }
}

void Decoder::reset() {
    if (_implicit_seq >= 0) {
        seqFree(_implicit_seq);
    }
}

int64_t Decoder::infer(const int64_t *tokens, size_t n) {
    if (n == 0 || tokens == nullptr) {
        failModel(LLAISYS_E_INVALID, "infer needs at least one token");
    }
    if (!_cache) {
        configureCache(1, std::max<size_t>(maxSeq(), n + 1));
    }
    if (_implicit_seq < 0) {
        _implicit_seq = seqAdd();
    }
    const int32_t n32 = int32_t(n);
    int64_t next = 0;
    step(&_implicit_seq, &n32, 1, tokens, &next);
    return next;
}

// ---- workspace -------------------------------------------------------------------------------------------------------

void Decoder::ensureWorkspace(size_t n_tokens, size_t n_seqs, size_t n_out) {
    auto &rt = enter();
    ensureActivations(n_tokens, n_out);
    _ws_tokens = std::max(_ws_tokens, n_tokens);
    if (n_out > _ws_out) {
        ++_generation;
        _ws_out = n_out;
        _logits = rt.allocateDeviceStorage(n_out * vocab() * utils::dsize(_logits_dtype));
        // keys and counters of the split argmax: zero once, the kernel leaves them zero
        _argmax_scratch = rt.allocateDeviceStorage(n_out * 12);
        const std::vector<std::byte> zeros(n_out * 12);
        copyToDevice(_argmax_scratch->memory(), zeros.data(), zeros.size());
    }
    // tokens, pos64, prev, out_rows, next (int64) then seq32, pos32, kv_lens, seq_list, q_starts (int32), 16-byte aligned
    const size_t need = align_up(n_tokens * 8, 16) * 3 + align_up(n_out * 8, 16) * 2 + align_up(n_tokens * 4, 16) * 2 +
                        align_up(n_seqs * 4, 16) * 2 + align_up((n_seqs + 1) * 4, 16);
    if (need > _meta_bytes) {
        ++_generation;
        _meta_bytes = need * 2;
        _meta_block = rt.allocateDeviceStorage(_meta_bytes);
    }
}

Decoder::StepArrays Decoder::carveStepArrays(size_t n_tokens, size_t n_seqs, size_t n_out) {
    StepArrays a;
    size_t at = 0;
    auto take = [&](size_t bytes) {
        const size_t here = at;
        at += align_up(bytes, 16);
        return here;
    };
    std::byte *base = _meta_block->memory();
    a.tokens = reinterpret_cast<int64_t *>(base + take(n_tokens * 8));
    a.pos64 = reinterpret_cast<int64_t *>(base + take(n_tokens * 8));
    a.prev = reinterpret_cast<int64_t *>(base + take(n_tokens * 8));
    a.out_rows = reinterpret_cast<int64_t *>(base + take(n_out * 8));
    a.next = reinterpret_cast<int64_t *>(base + take(n_out * 8));
    a.seq32 = reinterpret_cast<int32_t *>(base + take(n_tokens * 4));
    a.pos32 = reinterpret_cast<int32_t *>(base + take(n_tokens * 4));
    a.kv_lens = reinterpret_cast<int32_t *>(base + take(n_seqs * 4));
    a.seq_list = reinterpret_cast<int32_t *>(base + take(n_seqs * 4));
    a.q_starts = reinterpret_cast<int32_t *>(base + take((n_seqs + 1) * 4));
    return a;
}

void Decoder::copyToDevice(void *dst, const void *src, size_t bytes) {
    auto &rt = enter();
    if (_on_gpu) {
        rt.api()->memcpy_async(dst, src, bytes, LLAISYS_MEMCPY_H2D, _stream);
    } else {
        std::memcpy(dst, src, bytes);
    }
}

void Decoder::copyToHost(void *dst, const void *src, size_t bytes) {
    auto &rt = enter();
    if (_on_gpu) {
        rt.api()->memcpy_async(dst, src, bytes, LLAISYS_MEMCPY_D2H, _stream);
        rt.synchronize();
    } else {
        std::memcpy(dst, src, bytes);
    }
}

// ---- steps ------------------------------------------------------------------------------------------------------------

void Decoder::step(const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs, const int64_t *tokens, int64_t *next_out) {
    if (n_seqs != 0 && (n_tokens == nullptr || next_out == nullptr)) {
        failModel(LLAISYS_E_INVALID, "null argument");
    }
    std::vector<int32_t> rows(n_seqs);
    int32_t row = -1;
    for (size_t i = 0; i < n_seqs; ++i) {
        rows[i] = row += n_tokens[i];
    }
    stepRows(seq_ids, n_tokens, n_seqs, tokens, rows.data(), n_seqs, next_out);
}

void Decoder::stepRows(const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs, const int64_t *tokens,
                       const int32_t *rows, size_t n_rows, int64_t *next_out) {
    if (n_seqs == 0) {
        return;
    }
    if (seq_ids == nullptr || n_tokens == nullptr || tokens == nullptr ||
        (n_rows != 0 && (rows == nullptr || next_out == nullptr))) {
        failModel(LLAISYS_E_INVALID, "null argument");
    }
    size_t T = 0, max_q = 0, max_kv = 0;
    for (size_t i = 0; i < n_seqs; ++i) {
        const size_t len = seqLen(seq_ids[i]);
        if (n_tokens[i] < 1) {
            failModel(LLAISYS_E_INVALID, "every sequence of a step needs at least one new token");
        }
        if (len + size_t(n_tokens[i]) > _max_tokens_per_seq) {
            failModel(LLAISYS_E_INVALID, "sequence would exceed the configured maximum length");
        }
        for (size_t j = 0; j < i; ++j) {
            if (seq_ids[j] == seq_ids[i]) {
                failModel(LLAISYS_E_INVALID, "a sequence appears twice in one step");
            }
        }
        T += size_t(n_tokens[i]);
        max_q = std::max(max_q, size_t(n_tokens[i]));
        max_kv = std::max(max_kv, len + size_t(n_tokens[i]));
    }
    for (size_t i = 0; i < T; ++i) {
        if (tokens[i] < 0 || size_t(tokens[i]) >= vocab()) {
            failModel(LLAISYS_E_INVALID, "token id out of range");
        }
    }
    bool out_is_all = n_rows == T;
    for (size_t i = 0; i < n_rows; ++i) {
        if (rows[i] < 0 || size_t(rows[i]) >= T) {
            failModel(LLAISYS_E_INVALID, "a row with logits lies outside the step's tokens");
        }
        out_is_all = out_is_all && size_t(rows[i]) == i;
    }
    for (size_t i = 0; i < n_seqs; ++i) {
        _cache->seqReserve(seq_ids[i], seqLen(seq_ids[i]) + size_t(n_tokens[i]));
    }
    enter();
    ensureWorkspace(T, n_seqs, n_rows);
    const StepArrays a = carveStepArrays(T, n_seqs, n_rows);
    // the same carving over a host image, then one copy
    _meta_host.assign(_meta_bytes, std::byte{0});
    std::byte *dev0 = _meta_block->memory(), *host0 = _meta_host.data();
    auto host = [&](auto *dev_ptr) { return reinterpret_cast<decltype(dev_ptr)>(host0 + (reinterpret_cast<std::byte *>(dev_ptr) - dev0)); };
    size_t row = 0;
    bool decode_only = true;
    host(a.q_starts)[0] = 0;
    for (size_t i = 0; i < n_seqs; ++i) {
        const size_t len = seqLen(seq_ids[i]), n = size_t(n_tokens[i]);
        decode_only = decode_only && n == 1;
        for (size_t t = 0; t < n; ++t, ++row) {
            host(a.tokens)[row] = tokens[row];
            host(a.prev)[row] = t != 0 ? tokens[row - 1] : _seq_last[seq_ids[i]];
            host(a.pos64)[row] = int64_t(len + t);
            host(a.pos32)[row] = int32_t(len + t);
            host(a.seq32)[row] = seq_ids[i];
        }
        host(a.kv_lens)[i] = int32_t(len + n);
        host(a.seq_list)[i] = seq_ids[i];
        host(a.q_starts)[i + 1] = int32_t(row);
    }
    for (size_t i = 0; i < n_rows; ++i) {
        host(a.out_rows)[i] = rows[i];
    }
    StepShape shape;
    shape.n_tokens = T;
    shape.n_seqs = n_seqs;
    shape.n_out = n_rows;
    shape.max_q_len = max_q;
    shape.max_kv_len = max_kv;
    shape.decode_only = decode_only;
    shape.out_is_all = out_is_all;
    if (!decode_only) {
        shape.host_q_starts = host(a.q_starts);
        shape.host_kv_lens = host(a.kv_lens);
    }
    copyToDevice(dev0, host0, _meta_bytes);
    _cache->flush();
    bool replayed = false;
#ifdef ENABLE_NVIDIA_API
    if (_on_gpu && decode_only && out_is_all && graphable()) {
        // The launch-bound case (about nine kernels per layer): replay the step as a graph. The graph is captured with the
        // cache's maximum length as the attention kernels' bound, so it is valid for every later step of this batch size.
        if (_step_graphs.size() <= n_seqs) {
            _step_graphs.resize(n_seqs + 1);
        }
        StepGraph &g = _step_graphs[n_seqs];
        if (g.exec != nullptr && g.generation != _generation) {
            kernels::graph_destroy(g.exec);
            g = StepGraph{};
        }
        if (g.exec == nullptr && g.seen && g.generation == _generation) {
            enter().synchronize();
            kernels::graph_capture_begin(_stream);
            try {
                shape.max_kv_len = _max_tokens_per_seq;
                forward(a, shape);
            } catch (...) {
                kernels::graph_destroy(kernels::graph_capture_end(_stream));
                throw;
            }
            g.exec = kernels::graph_capture_end(_stream);
        }
        if (g.exec != nullptr) {
            kernels::graph_launch(g.exec, _stream);
            replayed = true;
        } else {
            g.seen = true;
            g.generation = _generation;
            shape.max_kv_len = _max_tokens_per_seq; // the eager step sizes scratch for what the capture will ask for
        }
    }
#endif
    if (!replayed) {
        forward(a, shape);
    }
    _last_n_out = n_rows;
    if (n_rows != 0) {
        copyToHost(next_out, a.next, n_rows * sizeof(int64_t));
    }
    for (size_t i = 0, at = 0; i < n_seqs; ++i) {
        seqLen(seq_ids[i]) += size_t(n_tokens[i]);
        recordTokens(seq_ids[i], tokens + at, size_t(n_tokens[i]));
        at += size_t(n_tokens[i]);
    }
    checkKernels();
}

void Decoder::decodeLoop(const int32_t *seq_ids, size_t n_seqs, const int64_t *first_tokens, size_t n_steps,
                       int64_t *tokens_out) {
    if (n_seqs == 0 || n_steps == 0) {
        return;
    }
    if (seq_ids == nullptr || first_tokens == nullptr || tokens_out == nullptr) {
        failModel(LLAISYS_E_INVALID, "null argument");
    }
    size_t max_kv = 0;
    for (size_t i = 0; i < n_seqs; ++i) {
        const size_t len = seqLen(seq_ids[i]);
        if (len + n_steps > _max_tokens_per_seq) {
            failModel(LLAISYS_E_INVALID, "sequence would exceed the configured maximum length");
        }
        if (first_tokens[i] < 0 || size_t(first_tokens[i]) >= vocab()) {
            failModel(LLAISYS_E_INVALID, "token id out of range");
        }
        max_kv = std::max(max_kv, len + n_steps);
    }
    for (size_t i = 0; i < n_seqs; ++i) {
        _cache->seqReserve(seq_ids[i], seqLen(seq_ids[i]) + n_steps); // every page of the loop, up front
    }
    auto &rt = enter();
    ensureWorkspace(n_seqs, n_seqs, n_seqs);
    const StepArrays a = carveStepArrays(n_seqs, n_seqs, n_seqs);
    _meta_host.assign(_meta_bytes, std::byte{0});
    std::byte *dev0 = _meta_block->memory(), *host0 = _meta_host.data();
    auto host = [&](auto *dev_ptr) { return reinterpret_cast<decltype(dev_ptr)>(host0 + (reinterpret_cast<std::byte *>(dev_ptr) - dev0)); };
    for (size_t i = 0; i < n_seqs; ++i) {
        const size_t len = seqLen(seq_ids[i]);
        host(a.tokens)[i] = first_tokens[i];
        host(a.prev)[i] = _seq_last[seq_ids[i]];
        host(a.pos64)[i] = int64_t(len);
        host(a.pos32)[i] = int32_t(len);
        host(a.seq32)[i] = seq_ids[i];
        host(a.kv_lens)[i] = int32_t(len + 1);
        host(a.seq_list)[i] = seq_ids[i];
        host(a.q_starts)[i] = int32_t(i);
        host(a.out_rows)[i] = int64_t(i);
    }
    host(a.q_starts)[n_seqs] = int32_t(n_seqs);
    copyToDevice(dev0, host0, _meta_bytes);
    _cache->flush();
    // the token log and the step counter the advance kernel writes through
    core::storage_t log = rt.allocateDeviceStorage(n_steps * n_seqs * sizeof(int64_t));
    core::storage_t counter = rt.allocateDeviceStorage(sizeof(int32_t));
    const int32_t zero = 0;
    copyToDevice(counter->memory(), &zero, sizeof(zero));
    auto *log_dev = reinterpret_cast<int64_t *>(log->memory());
    auto *counter_dev = reinterpret_cast<int32_t *>(counter->memory());

    StepShape shape;
    shape.n_tokens = shape.n_seqs = shape.n_out = n_seqs;
    shape.max_q_len = 1;
    shape.max_kv_len = max_kv;
    shape.decode_only = shape.out_is_all = true;
    auto one_step = [&]() {
        forward(a, shape);
#ifdef ENABLE_NVIDIA_API
        if (_on_gpu) {
            kernels::advance_decode_state(_stream, a.tokens, a.prev, a.next, a.pos64, a.pos32, a.kv_lens, log_dev, counter_dev,
                                          int(n_seqs));
            return;
        }
#endif
        int32_t &step = *counter_dev;
        for (size_t i = 0; i < n_seqs; ++i) {
            a.prev[i] = a.tokens[i];
            a.tokens[i] = a.next[i];
            log_dev[size_t(step) * n_seqs + i] = a.next[i];
            a.pos64[i] += 1;
            a.pos32[i] += 1;
            a.kv_lens[i] += 1;
        }
        ++step;
    };

    if (_on_gpu) {
#ifdef ENABLE_NVIDIA_API
        one_step(); // eager: sizes every lazily grown scratch before the capture
        size_t timed_steps = 0;
        float ms = 0.f;
        if (n_steps > 1) {
            rt.synchronize();
            kernels::graph_capture_begin(_stream);
            try {
                one_step();
            } catch (...) {
                kernels::graph_destroy(kernels::graph_capture_end(_stream));
                throw;
            }
            void *exec = kernels::graph_capture_end(_stream);
            void *e0 = kernels::event_create(), *e1 = kernels::event_create();
            kernels::event_record(e0, _stream);
            for (size_t s = 1; s < n_steps; ++s) {
                kernels::graph_launch(exec, _stream);
            }
            kernels::event_record(e1, _stream);
            ms = kernels::event_elapsed_ms(e0, e1);
            timed_steps = n_steps - 1;
            kernels::event_destroy(e0);
            kernels::event_destroy(e1);
            kernels::graph_destroy(exec);
        }
        _last_loop_ms = timed_steps ? double(ms) / double(timed_steps) : 0.0;
#endif
    } else {
        const auto t0 = std::chrono::steady_clock::now();
        for (size_t s = 0; s < n_steps; ++s) {
            one_step();
        }
        _last_loop_ms = std::chrono::duration<double, std::milli>(std::chrono::steady_clock::now() - t0).count() / double(n_steps);
    }
    _last_n_out = n_seqs;
    copyToHost(tokens_out, log_dev, n_steps * n_seqs * sizeof(int64_t));
    std::vector<int64_t> fed(n_steps);
    for (size_t i = 0; i < n_seqs; ++i) {
        seqLen(seq_ids[i]) += n_steps;
        fed[0] = first_tokens[i]; // step s consumed the token step s - 1 produced
        for (size_t st = 1; st < n_steps; ++st) {
            fed[st] = tokens_out[(st - 1) * n_seqs + i];
        }
        recordTokens(seq_ids[i], fed.data(), n_steps);
    }
    checkKernels();
}

// Error words of the kernels a step ran: the cache's (bad block-table entries, a wait that ran out in an attention
// kernel) and the projection kernel's.
void Decoder::checkKernels() {
    _cache->check();
#ifdef ENABLE_NVIDIA_API
    if (_on_gpu) {
        const int status = kernels::linear_tc_status(_stream);
        if (status != 0) {
            failModel(LLAISYS_E_KERNEL, "the projection kernel reported error word " + std::to_string(status));
        }
    }
#endif
}

void Decoder::lastLogits(float *out_host, size_t capacity_floats) {
    const size_t n = _last_n_out * vocab();
    if (n == 0) {
        failModel(LLAISYS_E_INVALID, "no step has run yet");
    }
    if (out_host == nullptr || capacity_floats < n) {
        failModel(LLAISYS_E_INVALID, "logits buffer too small");
    }
    std::vector<std::byte> raw(n * utils::dsize(_logits_dtype));
    copyToHost(raw.data(), _logits->memory(), raw.size());
    for (size_t i = 0; i < n; ++i) {
        switch (_logits_dtype) {
        case LLAISYS_DTYPE_F32:
            out_host[i] = reinterpret_cast<const float *>(raw.data())[i];
            break;
        case LLAISYS_DTYPE_F16:
            out_host[i] = utils::cast<float>(reinterpret_cast<const fp16_t *>(raw.data())[i]);
            break;
        default:
            out_host[i] = utils::cast<float>(reinterpret_cast<const bf16_t *>(raw.data())[i]);
            break;
        }
    }
}

} // namespace llaisys::models
