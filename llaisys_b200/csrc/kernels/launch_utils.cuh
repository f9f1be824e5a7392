// Launch helpers shared by kernels that take part in programmatic launches.
#pragma once

#include "device_utils.cuh"
#include "kernels.hpp"

#include <utility>

namespace llaisys::kernels {

// Programmatic launch: the kernel waits for its predecessor (grid_dependency_wait) before it touches anything, then lets its successor be
// scheduled, so that a launch hides under the kernel before it (see rms_norm_vec_kernel).
template <typename... KArgs, typename... Args>
void launch_programmatic_smem(void (*kernel)(KArgs...), dim3 grid, unsigned block, size_t smem, cudaStream_t s, Args &&...args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(block);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    LLAISYS_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, KArgs(std::forward<Args>(args))...));
}
template <typename... KArgs, typename... Args>
void launch_programmatic(void (*kernel)(KArgs...), dim3 grid, unsigned block, cudaStream_t s, Args &&...args) {
    launch_programmatic_smem(kernel, grid, block, 0, s, std::forward<Args>(args)...);
}

inline bool aligned16(const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

// body(T{}) with the element type of dtype
template <typename F>
void dispatch(llaisysDataType_t dtype, F &&body) {
    switch (dtype) {
    case LLAISYS_DTYPE_F32:
        body(float{});
        break;
    case LLAISYS_DTYPE_F16:
        body(__half{});
        break;
    case LLAISYS_DTYPE_BF16:
        body(__nv_bfloat16{});
        break;
    default:
        EXCEPTION_UNSUPPORTED_DATATYPE(dtype);
    }
}

} // namespace llaisys::kernels
