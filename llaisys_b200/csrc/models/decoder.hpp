// The network-independent half of a decoder-only model: sequences over a paged KV cache (and recurrent-state slots where
// the network has them), batched steps, the device-resident decode loop, captured decode steps and logits. A model
// derives from Decoder and supplies its weights, its cache geometry, its activations and forward().
//
// All state of a forward pass lives on the model's device: activations in a workspace sized for the largest batch
// seen, per-step index arrays (tokens, positions, sequence rows, lengths) in one staging block. A decode loop keeps
// even the loop-carried state there: the chosen tokens feed the next step's embedding lookup, positions and lengths
// are advanced by a kernel, and on NVIDIA one step is captured as a CUDA graph and replayed.
#pragma once

#include "../capi/handles.hpp"
#include "../kv/paged_kv.hpp"
#include "../kv/state_pool.hpp"

#include <memory>
#include <string>
#include <vector>

namespace llaisys::models {

// Objects that borrow a model (a serving engine) hear about its destruction instead of touching freed memory when the
// owner destroys the two in the wrong order.
struct ModelObserver {
    virtual void modelDestroyed() = 0;

protected:
    ~ModelObserver() = default;
};

class Decoder {
public:
    Decoder(const char *name, llaisysDeviceType_t device, int device_id, llaisysDataType_t dtype, llaisysDataType_t logits_dtype);
    virtual ~Decoder();
    Decoder(const Decoder &) = delete;
    Decoder &operator=(const Decoder &) = delete;

    void addObserver(ModelObserver *o) { _observers.push_back(o); }
    void removeObserver(ModelObserver *o);

    llaisysDeviceType_t deviceType() const { return _device; }
    int deviceId() const { return _device_id; }
    llaisysDataType_t dtype() const { return _dtype; }
    virtual size_t vocab() const = 0;
    virtual size_t maxSeq() const = 0;      // default length of the implicit sequence's cache
    virtual int64_t endToken() const = 0;   // < 0: none

    // Copies one checkpoint tensor (host memory, F32 or BF16, row-major) into the weight of that name. False: the model
    // has no such weight. Throws on a wrong shape. Models whose weights are loaded through handles have no names.
    virtual bool loadTensor(const std::string &name, llaisysDataType_t dtype, const std::vector<size_t> &shape, const void *data);
    // Names of weights that no loadTensor call has filled yet.
    virtual std::vector<std::string> missingTensors() const { return {}; }

    // Development aid, for models that have it: keep the residual stream after every layer run of the steps that follow;
    // layerStream gives [runs, rows, width] of the last such step (-> its floats; out_host may be null).
    virtual void recordStream(bool enable);
    virtual size_t layerStream(float *out_host, size_t capacity_floats);

    // A cache of max_seqs sequences of at most max_tokens tokens each. pool_tokens: how many tokens all live sequences
    // together can hold (whole pages); 0 = max_seqs * max_tokens.
    void configureCache(size_t max_seqs, size_t max_tokens, size_t pool_tokens = 0);
    int32_t seqAdd();
    // New sequence that starts from the cached K/V of the longest published whole-page prefix of tokens[0, n) that leaves
    // at least one token to run; *matched = tokens already covered (feed tokens[*matched, n) to step()). A model with
    // recurrent state never matches: pages alone do not hold what its prefix left behind.
    int32_t seqAddWithPrefix(const int64_t *tokens, size_t n, size_t *matched);
    void seqReserve(int32_t seq, size_t n_tokens); // pages for n_tokens now, so that later steps cannot run out
    size_t seqLength(int32_t seq) { return seqLen(seq); }
    size_t freePages() const { return _cache ? _cache->numFreePages() : 0; }
    size_t maxTokensPerSeq() const { return _max_tokens_per_seq; }
    void seqFree(int32_t seq);
    void reset();
    int64_t infer(const int64_t *tokens, size_t n);
    // Appends n_tokens[i] tokens to sequence seq_ids[i]; next_out[i] = greedy token after its last one.
    void step(const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs, const int64_t *tokens, int64_t *next_out);
    // The same step with logits (and greedy tokens) at chosen rows of the packed tokens instead of at each sequence's last
    // token: rows[n_rows], any order, n_rows may be 0 (the vocabulary projection is then skipped). next_out[n_rows].
    void stepRows(const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs, const int64_t *tokens, const int32_t *rows,
                  size_t n_rows, int64_t *next_out);
    void decodeLoop(const int32_t *seq_ids, size_t n_seqs, const int64_t *first_tokens, size_t n_steps,
                    int64_t *tokens_out);
    void lastLogits(float *out_host, size_t capacity_floats);
    double lastLoopMs() const { return _last_loop_ms; }

protected:
    // device pointers of one step's index arrays (all inside _meta_block)
    struct StepArrays {
        int64_t *tokens = nullptr, *pos64 = nullptr, *out_rows = nullptr, *next = nullptr;
        int64_t *prev = nullptr; // the token before each row's in its sequence, -1 for the first
        int32_t *seq32 = nullptr, *pos32 = nullptr, *kv_lens = nullptr, *q_starts = nullptr, *seq_list = nullptr;
    };
    struct StepShape {
        size_t n_tokens = 0, n_seqs = 0, n_out = 0; // rows, sequences, rows with logits
        size_t max_q_len = 0, max_kv_len = 0;
        bool decode_only = false;   // one token per sequence
        bool out_is_all = false;    // logits are wanted for every row, in order (no gather needed)
        // the same as StepArrays::q_starts and kv_lens in host memory, valid during forward(); null in decode steps
        const int32_t *host_q_starts = nullptr, *host_kv_lens = nullptr;
    };

    // ---- what a model supplies ----
    // layers, heads and head dims of the cache; pool and table sizes are filled in by configureCache
    virtual kv::PagedKVConfig cacheShape() const = 0;
    // floats of recurrent state per sequence, one entry per state-carrying layer; empty = none
    virtual std::vector<size_t> stateShape() const { return {}; }
    // activations for up to n_tokens rows (bump _generation when a buffer moves)
    virtual void ensureActivations(size_t n_tokens, size_t n_out) = 0;
    // the network itself: logits into _logits [n_out, vocab], greedy tokens into a.next
    virtual void forward(const StepArrays &a, const StepShape &s) = 0;
    virtual bool graphable() const { return true; } // decode steps may be captured as CUDA graphs

    core::Runtime &enter() const;
    [[noreturn]] void failModel(int code, const std::string &msg) const;
    void copyToDevice(void *dst, const void *src, size_t bytes);
    void copyToHost(void *dst, const void *src, size_t bytes);
    void dropStepGraphs();

    const char *_name;
    llaisysDeviceType_t _device;
    int _device_id;
    llaisysDataType_t _dtype, _logits_dtype;
    size_t _elem = 0;
    bool _on_gpu = false;
    llaisysStream_t _stream = nullptr;

    std::unique_ptr<kv::PagedKV> _cache;
    std::unique_ptr<kv::StatePool> _state;
    core::storage_t _logits, _argmax_scratch;
    size_t _ws_tokens = 0, _ws_out = 0;
    uint64_t _generation = 1;

private:
    void ensureWorkspace(size_t n_tokens, size_t n_seqs, size_t n_out);
    StepArrays carveStepArrays(size_t n_tokens, size_t n_seqs, size_t n_out);
    size_t &seqLen(int32_t seq);
    void recordTokens(int32_t seq, const int64_t *tokens, size_t n);
    void checkKernels();

    size_t _max_tokens_per_seq = 0;
    std::vector<size_t> _seq_len; // by sequence id; SIZE_MAX = not live
    std::vector<int64_t> _seq_last;  // by sequence id: its newest token, -1 when it has none
    std::vector<std::vector<int64_t>> _seq_tokens; // ids of the tokens each sequence holds (keys of the prefix cache)
    int32_t _implicit_seq = -1;
    core::storage_t _meta_block;
    size_t _meta_bytes = 0;
    std::vector<std::byte> _meta_host;
    // Decode steps of step() (every sequence one token) replayed as CUDA graphs, one per batch size: the first step of
    // a size runs eagerly (it sizes scratch), the second is captured, later ones are replayed. A graph is dropped when
    // a buffer it points into is reallocated (generation) or the cache is reconfigured.
    struct StepGraph {
        void *exec = nullptr;
        uint64_t generation = 0;
        bool seen = false;
    };
    std::vector<StepGraph> _step_graphs; // by n_seqs
    std::vector<ModelObserver *> _observers;
    size_t _last_n_out = 0;
    double _last_loop_ms = 0.0;
};

} // namespace llaisys::models
