#include "state_pool.hpp"

#include "llaisys/paged_kv.h"
#include "paged_kv.hpp"

namespace llaisys::kv {

StatePool::StatePool(llaisysDeviceType_t device_type, int device_id, size_t n_slots, const std::vector<size_t> &layer_floats)
    : _n_slots(n_slots) {
    if (n_slots == 0 || layer_floats.empty()) {
        throw StatusError(LLAISYS_E_INVALID, "state pool: no slots or no layers");
    }
    size_t total = 0;
    for (size_t n : layer_floats) {
        if (n == 0) {
            throw StatusError(LLAISYS_E_INVALID, "state pool: a layer without state");
        }
        _stride.push_back((n + 3) / 4 * 4);
        _offset.push_back(total);
        total += n_slots * _stride.back();
    }
    auto &ctx = core::context();
    ctx.setDevice(device_type, device_id);
    _block = ctx.runtime().allocateDeviceStorage(total * sizeof(float));
}

float *StatePool::data(size_t layer) const { return reinterpret_cast<float *>(_block->memory()) + _offset[layer]; }

} // namespace llaisys::kv
