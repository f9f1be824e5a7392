#include "stream_decoder.hpp"

#include "../common/check.hpp"
#include "../common/dtypes.hpp"
#include "llaisys/paged_kv.h"
#ifdef ENABLE_NVIDIA_API
#include "../kernels/kernels.hpp"
#endif

#include <algorithm>

namespace llaisys::models {

StreamDecoder::StreamDecoder(const char *name, llaisysDeviceType_t device, int device_id, llaisysDataType_t dtype)
    : Decoder(name, device, device_id, dtype, LLAISYS_DTYPE_F32) {
    if (!_on_gpu) {
        failModel(LLAISYS_E_UNSUPPORTED, "this model runs on NVIDIA devices only");
    }
}

std::byte *StreamDecoder::matrix(size_t rows, size_t cols) {
    auto &rt = enter();
    _weight_blocks.push_back(rt.allocateDeviceStorage(rows * cols * _elem));
    std::byte *p = _weight_blocks.back()->memory();
#ifdef ENABLE_NVIDIA_API
    kernels::fill_zero(rt.stream(), p, rows * cols * _elem);
#endif
    return p;
}

void StreamDecoder::place(const std::string &name, std::byte *base, size_t row, size_t col, size_t rows, size_t cols, size_t ld,
                    size_t ndim) {
    _slots.emplace(name, Slot{base, row, col, rows, cols, ld, ndim, _dtype});
}

std::byte *StreamDecoder::vector(const std::string &name, size_t n) {
    std::byte *p = matrix(n, 1);
    place(name, p, 0, 0, n, 1, 1, 1);
    return p;
}

float *StreamDecoder::floats(const std::string &name, size_t n) {
    auto &rt = enter();
    const size_t rows = std::max<size_t>(n, 1);
    _weight_blocks.push_back(rt.allocateDeviceStorage(rows * sizeof(float)));
    std::byte *p = _weight_blocks.back()->memory();
    _slots.emplace(name, Slot{p, 0, 0, rows, 1, 1, n == 0 ? size_t(0) : size_t(1), LLAISYS_DTYPE_F32});
    return reinterpret_cast<float *>(p);
}

bool StreamDecoder::loadTensor(const std::string &name, llaisysDataType_t dtype, const std::vector<size_t> &shape, const void *data) {
    auto it = _slots.find(name);
    if (it == _slots.end()) {
        return false;
    }
    Slot &slot = it->second;
    const bool fits = shape.size() == slot.ndim && (slot.ndim < 1 || shape[0] == slot.rows) && (slot.ndim < 2 || shape[1] == slot.cols);
    if (!fits) {
        failModel(LLAISYS_E_INVALID, "tensor " + name + " has another shape than the configuration gives it");
    }
    if (dtype != LLAISYS_DTYPE_F32 && dtype != LLAISYS_DTYPE_BF16 && dtype != LLAISYS_DTYPE_F16) {
        failModel(LLAISYS_E_INVALID, "tensor " + name + ": F32, F16 or BF16 expected");
    }
    const size_t n = slot.rows * slot.cols, elem = utils::dsize(slot.dtype);
    std::vector<std::byte> converted;
    const std::byte *src = static_cast<const std::byte *>(data);
    if (dtype != slot.dtype) {
        converted.resize(n * elem);
        for (size_t i = 0; i < n; ++i) {
            float v = 0.f;
            switch (dtype) {
            case LLAISYS_DTYPE_F32:
                v = static_cast<const float *>(data)[i];
                break;
            case LLAISYS_DTYPE_F16:
                v = utils::cast<float>(static_cast<const fp16_t *>(data)[i]);
                break;
            default:
                v = utils::cast<float>(static_cast<const bf16_t *>(data)[i]);
                break;
            }
            switch (slot.dtype) {
            case LLAISYS_DTYPE_F32:
                reinterpret_cast<float *>(converted.data())[i] = v;
                break;
            case LLAISYS_DTYPE_F16:
                reinterpret_cast<fp16_t *>(converted.data())[i] = utils::cast<fp16_t>(v);
                break;
            default:
                reinterpret_cast<bf16_t *>(converted.data())[i] = utils::cast<bf16_t>(v);
                break;
            }
        }
        src = converted.data();
    }
    auto &rt = enter();
    rt.synchronize(); // the zero fill of the packed matrix comes first
    std::byte *dst = slot.base + (slot.row * slot.ld + slot.col) * elem;
    if (slot.cols == slot.ld) {
        rt.api()->memcpy_sync(dst, src, n * elem, LLAISYS_MEMCPY_H2D);
    } else {
        for (size_t r = 0; r < slot.rows; ++r) {
            rt.api()->memcpy_sync(dst + r * slot.ld * elem, src + r * slot.cols * elem, slot.cols * elem, LLAISYS_MEMCPY_H2D);
        }
    }
    slot.loaded = true;
    return true;
}

std::vector<std::string> StreamDecoder::missingTensors() const {
    std::vector<std::string> names;
    for (const auto &[name, slot] : _slots) {
        if (!slot.loaded) {
            names.push_back(name);
        }
    }
    return names;
}

void StreamDecoder::recordLayer(const float *stream, size_t n) {
    if (_record) {
        const size_t at = _recorded.size();
        _recorded.resize(at + n);
        copyToHost(_recorded.data() + at, stream, n * sizeof(float));
    }
}

size_t StreamDecoder::layerStream(float *out_host, size_t capacity_floats) {
    if (_recorded.empty()) {
        failModel(LLAISYS_E_INVALID, "no step has been recorded");
    }
    if (out_host != nullptr) {
        if (capacity_floats < _recorded.size()) {
            failModel(LLAISYS_E_INVALID, "stream buffer too small");
        }
        std::copy(_recorded.begin(), _recorded.end(), out_host);
    }
    return _recorded.size();
}

} // namespace llaisys::models
