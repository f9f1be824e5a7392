// The struct behind the opaque cache handle of the C ABI, shared by the thunks that take one.
#pragma once

#include "../kv/paged_kv.hpp"

struct LlaisysPagedKV {
    llaisys::kv::PagedKV impl;
    explicit LlaisysPagedKV(const llaisys::kv::PagedKVConfig &cfg) : impl(cfg) {}
};
