// extern "C" thunks of the generic model API and of the families that have no older ABI of their own.
#include "llaisys/models/doderax.h"
#include "llaisys/models/folivik.h"
#include "llaisys/models/lilovik.h"
#include "llaisys/models/model.h"
#include "llaisys/models/vozozen.h"
#include "llaisys/paged_kv.h"

#include "model_handle.hpp"

#include <cstring>
#include <iostream>

using llaisys::capi::guarded;
using llaisys::capi::null_model;

template <typename Model, typename Meta>
static LlaisysModel *create_model(const char *function, const Meta *meta, llaisysDeviceType_t device, int device_id) {
    LlaisysModel *model = nullptr;
    const int rc = meta == nullptr ? null_model()
                                   : guarded([&] { model = new LlaisysModel(std::make_unique<Model>(*meta, device, device_id)); });
    if (rc != LLAISYS_OK) {
        std::cerr << "[ERROR] " << function << ": " << llaisysGetLastError() << std::endl;
        return nullptr;
    }
    return model;
}

extern "C" {

void llaisysModelDestroy(LlaisysModel *model) { delete model; }
size_t llaisysModelVocab(LlaisysModel *model) { return model ? model->impl->vocab() : 0; }

int llaisysModelLoadTensor(LlaisysModel *model, const char *name, llaisysDataType_t dtype, const size_t *shape, size_t ndim,
                           const void *data, int *known_out) {
    if (model == nullptr || name == nullptr || (shape == nullptr && ndim != 0) || data == nullptr) {
        return null_model();
    }
    return guarded([&] {
        const bool known = model->impl->loadTensor(name, dtype, std::vector<size_t>(shape, shape + ndim), data);
        if (known_out != nullptr) {
            *known_out = known ? 1 : 0;
        }
    });
}
size_t llaisysModelMissingTensors(LlaisysModel *model, char *name_out, size_t cap) {
    if (model == nullptr) {
        return 0;
    }
    const std::vector<std::string> missing = model->impl->missingTensors();
    if (name_out != nullptr && cap > 0) {
        std::strncpy(name_out, missing.empty() ? "" : missing[0].c_str(), cap - 1);
        name_out[cap - 1] = '\0';
    }
    return missing.size();
}

int llaisysModelConfigureCache(LlaisysModel *model, size_t max_seqs, size_t max_tokens, size_t pool_tokens) {
    return model ? guarded([&] { model->impl->configureCache(max_seqs, max_tokens, pool_tokens); }) : null_model();
}
int llaisysModelSeqAdd(LlaisysModel *model, int32_t *seq_out) {
    return model && seq_out ? guarded([&] { *seq_out = model->impl->seqAdd(); }) : null_model();
}
int llaisysModelSeqAddWithPrefix(LlaisysModel *model, const int64_t *tokens, size_t n, int32_t *seq_out, size_t *matched_out) {
    if (model == nullptr || seq_out == nullptr || matched_out == nullptr) {
        return null_model();
    }
    return guarded([&] { *seq_out = model->impl->seqAddWithPrefix(tokens, n, matched_out); });
}
int llaisysModelSeqFree(LlaisysModel *model, int32_t seq) {
    return model ? guarded([&] { model->impl->seqFree(seq); }) : null_model();
}
size_t llaisysModelFreePages(LlaisysModel *model) { return model ? model->impl->freePages() : 0; }
int llaisysModelInfer(LlaisysModel *model, const int64_t *tokens, size_t n, int64_t *next_out) {
    return model && next_out ? guarded([&] { *next_out = model->impl->infer(tokens, n); }) : null_model();
}
int llaisysModelReset(LlaisysModel *model) {
    return model ? guarded([&] { model->impl->reset(); }) : null_model();
}
int llaisysModelStep(LlaisysModel *model, const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs, const int64_t *tokens,
                     int64_t *next_out) {
    return model ? guarded([&] { model->impl->step(seq_ids, n_tokens, n_seqs, tokens, next_out); }) : null_model();
}
int llaisysModelStepRows(LlaisysModel *model, const int32_t *seq_ids, const int32_t *n_tokens, size_t n_seqs,
                         const int64_t *tokens, const int32_t *rows, size_t n_rows, int64_t *next_out) {
    return model ? guarded([&] { model->impl->stepRows(seq_ids, n_tokens, n_seqs, tokens, rows, n_rows, next_out); })
                 : null_model();
}
int llaisysModelDecodeLoop(LlaisysModel *model, const int32_t *seq_ids, size_t n_seqs, const int64_t *first_tokens, size_t n_steps,
                           int64_t *tokens_out) {
    return model ? guarded([&] { model->impl->decodeLoop(seq_ids, n_seqs, first_tokens, n_steps, tokens_out); }) : null_model();
}
int llaisysModelLastLogits(LlaisysModel *model, float *out_host, size_t capacity_floats) {
    return model ? guarded([&] { model->impl->lastLogits(out_host, capacity_floats); }) : null_model();
}
double llaisysModelLastLoopMs(LlaisysModel *model) { return model ? model->impl->lastLoopMs() : 0.0; }

LlaisysModel *llaisysVozozenModelCreate(const LlaisysVozozenMeta *meta, llaisysDeviceType_t device, int device_id) {
    return create_model<llaisys::models::Vozozen>("llaisysVozozenModelCreate", meta, device, device_id);
}
LlaisysModel *llaisysDoderaxModelCreate(const LlaisysDoderaxMeta *meta, llaisysDeviceType_t device, int device_id) {
    return create_model<llaisys::models::Doderax>("llaisysDoderaxModelCreate", meta, device, device_id);
}
LlaisysModel *llaisysLilovikModelCreate(const LlaisysLilovikMeta *meta, llaisysDeviceType_t device, int device_id) {
    return create_model<llaisys::models::Lilovik>("llaisysLilovikModelCreate", meta, device, device_id);
}

LlaisysModel *llaisysFolivikModelCreate(const LlaisysFolivikMeta *meta, llaisysDeviceType_t device, int device_id) {
    return create_model<llaisys::models::Folivik>("llaisysFolivikModelCreate", meta, device, device_id);
}

int llaisysModelRecordStream(LlaisysModel *model, int enable) {
    return model ? guarded([&] { model->impl->recordStream(enable != 0); }) : null_model();
}
int llaisysModelLayerStream(LlaisysModel *model, float *out_host, size_t capacity_floats, size_t *floats_out) {
    return model && floats_out ? guarded([&] { *floats_out = model->impl->layerStream(out_host, capacity_floats); }) : null_model();
}

} // extern "C"
