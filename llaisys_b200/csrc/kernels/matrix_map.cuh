// Tensor maps over plain matrices and the error word of the kernels that use them (defined in skinny_gemm_tc.cu).
#pragma once

#include <cuda.h>

#include <cstdint>

namespace llaisys::kernels {

constexpr int kErrGemmTimeout = 16; // bit of the error word: a bounded wait ran out

// Row-major [rows, k] 16-bit matrix -> 2-D map with a box of 64 elements x box_rows rows, 128-byte swizzle; elements outside read as
// zero. Maps are cached: a decode loop asks for the same handful of (pointer, shape) pairs every step.
bool matrix_map(CUtensorMap *out, const void *ptr, uint64_t rows, uint64_t k, uint32_t box_rows, bool bf16);
// The current device's error word (see linear_tc_status).
int32_t *gemm_error_word();

} // namespace llaisys::kernels
