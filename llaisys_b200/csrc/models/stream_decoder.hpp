// What decoders with an f32 residual stream share: weights that are loaded by their checkpoint names into packed matrices
// (several tensors side by side in one allocation, so that one product serves all their readers), and the development aid that
// keeps the stream after every layer. NVIDIA devices only.
#pragma once

#include "decoder.hpp"

#include <map>
#include <string>
#include <vector>

namespace llaisys::models {

class StreamDecoder : public Decoder {
public:
    StreamDecoder(const char *name, llaisysDeviceType_t device, int device_id, llaisysDataType_t dtype);

    bool loadTensor(const std::string &name, llaisysDataType_t dtype, const std::vector<size_t> &shape, const void *data) override;
    std::vector<std::string> missingTensors() const override;
    void recordStream(bool enable) override { _record = enable; }
    size_t layerStream(float *out_host, size_t capacity_floats) override;

protected:
    bool graphable() const override { return !_record; }

    std::byte *matrix(size_t rows, size_t cols); // zeroed, owned by the model
    // The named tensor goes to `rows` x `cols` elements at (row, col) of a packed matrix with `ld` columns; ndim of the
    // checkpoint tensor (1: a vector of `rows`, cols == 1).
    void place(const std::string &name, std::byte *base, size_t row, size_t col, size_t rows, size_t cols, size_t ld, size_t ndim = 2);
    std::byte *vector(const std::string &name, size_t n);
    // n numbers kept in f32 whatever the model's dtype; n == 0: one number, a tensor without dimensions
    float *floats(const std::string &name, size_t n);

    void beginRecord() { _recorded.clear(); }
    void recordLayer(const float *stream, size_t n); // n floats on the device; nothing unless recording is on

private:
    struct Slot {
        std::byte *base;
        size_t row, col, rows, cols, ld;
        size_t ndim;
        llaisysDataType_t dtype;
        bool loaded = false;
    };
    std::map<std::string, Slot> _slots;
    std::vector<core::storage_t> _weight_blocks;
    bool _record = false;
    std::vector<float> _recorded;
};

// Sizes are rounded up to whole 16-byte pieces of 16-bit elements wherever parts of a packed row follow one another.
inline size_t pad8(size_t n) { return (n + 7) / 8 * 8; }

} // namespace llaisys::models
