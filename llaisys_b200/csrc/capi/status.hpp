// Exceptions to status codes, for the thunks of the status-returning ABI.
#pragma once

#include "../kv/paged_kv.hpp"
#include "llaisys/paged_kv.h"

#include <stdexcept>
#include <string>

namespace llaisys::kernels {
void set_last_error(const std::string &msg);
}

namespace llaisys::capi {

// Runs `body`; every failure becomes a status code plus a thread-local message (llaisysGetLastError).
template <typename F>
int guarded(F &&body) {
    try {
        body();
        return LLAISYS_OK;
    } catch (const kv::StatusError &e) {
        kernels::set_last_error(e.what());
        return e.code;
    } catch (const std::invalid_argument &e) {
        kernels::set_last_error(e.what());
        return LLAISYS_E_INVALID;
    } catch (const std::exception &e) {
        kernels::set_last_error(e.what());
        return LLAISYS_E_DEVICE;
    }
}

} // namespace llaisys::capi
