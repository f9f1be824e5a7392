#include "kernels.hpp"
#include "state_space.cuh"

namespace llaisys::kernels {

bool state_space_tiles_fit(llaisysDataType_t, const StateSpaceArgs &) { return false; }
void state_space_tiles(stream_t, const StateSpaceArgs &) {}
size_t state_space_segment_floats(llaisysDataType_t, size_t, size_t, size_t) { return 0; }

} // namespace llaisys::kernels
