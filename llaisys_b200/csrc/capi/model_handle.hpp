// The structs behind the opaque model handles of the C ABI. A family's handle IS a model handle: the generic functions take
// either.
#pragma once

#include "../models/doderax.hpp"
#include "../models/folivik.hpp"
#include "../models/lilovik.hpp"
#include "../models/qwen2.hpp"
#include "../models/vozozen.hpp"

#include "status.hpp"

#include <memory>

struct LlaisysModel {
    explicit LlaisysModel(std::unique_ptr<llaisys::models::Decoder> decoder) : impl(std::move(decoder)) {}
    std::unique_ptr<llaisys::models::Decoder> impl;
};

struct LlaisysQwen2Model : LlaisysModel {
    LlaisysQwen2Model(const LlaisysQwen2Meta &meta, llaisysDeviceType_t device, int device_id, int tp_rank = 0, int tp_world = 1)
        : LlaisysModel(std::make_unique<llaisys::models::Qwen2>(meta, device, device_id, tp_rank, tp_world)) {}
    llaisys::models::Qwen2 &qwen2() { return static_cast<llaisys::models::Qwen2 &>(*impl); }
};

namespace llaisys::capi {

inline int null_model() {
    kernels::set_last_error("model: null handle or argument");
    return LLAISYS_E_INVALID;
}

} // namespace llaisys::capi
