// Recurrent state of sequences: one slot per sequence, f32, for every layer that carries state. The slot of a sequence is
// its id in the paged cache, so slots come and go with sequences and need no allocator of their own. A slot is not
// cleared when a sequence takes it: kernels start a sequence whose first token is in the step from a zero state and
// never read what an earlier owner left.
#pragma once

#include "../core/core.hpp"

#include <vector>

namespace llaisys::kv {

class StatePool {
public:
    // layer_floats[l] = floats of state per sequence in layer l
    StatePool(llaisysDeviceType_t device_type, int device_id, size_t n_slots, const std::vector<size_t> &layer_floats);
    StatePool(const StatePool &) = delete;
    StatePool &operator=(const StatePool &) = delete;

    size_t numSlots() const { return _n_slots; }
    size_t numLayers() const { return _stride.size(); }
    // slot s of a layer starts at data(layer) + s * slotStride(layer)
    float *data(size_t layer) const;
    size_t slotStride(size_t layer) const { return _stride[layer]; } // floats, a multiple of 4 (16 bytes)

private:
    size_t _n_slots;
    std::vector<size_t> _stride, _offset; // floats
    core::storage_t _block;
};

} // namespace llaisys::kv
