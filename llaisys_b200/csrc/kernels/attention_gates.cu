// Attention without a softmax, any dtype and sizes (GateArgs): the correctness baseline of attention_gates_tiles.cu and the kernel
// behind the shapes that one does not cover.
//
// One CTA of eight warps per query row and range of up to 4096 output elements, because the weights of ALL heads meet in every
// output. Blocks of 32 keys: a warp takes a head at a time, a lane scores a key; the weights are mixed over the heads in shared
// memory; every thread adds up to 16 outputs. f32 arithmetic with exact expf and tanhf.
#include "device_utils.cuh"
#include "kernels.hpp"

namespace llaisys::kernels {

namespace {

constexpr int kThreads = 256, kKeys = 32, kOutPerThread = 16;

template <typename T>
__global__ void __launch_bounds__(kThreads)
    attention_gates_kernel(KVView kv, AttnBatch batch, const T *__restrict__ q, float scale, GateArgs gates, T *__restrict__ out,
                           int64_t out_stride, int32_t *error_flag) {
    extern __shared__ float smem[];
    const int d = kv.d, dv = kv.vDim(), nh = batch.nh, share = nh / kv.nkvh;
    float *q_s = smem;                                                  // [nh][d], times scale
    float *w_s = q_s + nh * d;                                          // [nh][32]
    float *m_s = w_s + nh * kKeys;                                      // [nh][32], mixed over the heads
    int64_t *v_off_s = reinterpret_cast<int64_t *>(m_s + nh * kKeys + ((nh * d) & 1)); // [32], -1: unseen
    const int row = blockIdx.x, warp = int(threadIdx.x) >> 5, lane = int(threadIdx.x) & 31;

    int seq, t, q_len;
    if (batch.q_starts != nullptr) {
        int lo = 0, hi = batch.n_seqs - 1;
        while (lo < hi) { // last seq with q_starts[seq] <= row
            const int mid = (lo + hi + 1) >> 1;
            if (batch.q_starts[mid] <= row) {
                lo = mid;
            } else {
                hi = mid - 1;
            }
        }
        seq = lo;
        t = row - batch.q_starts[seq];
        q_len = batch.q_starts[seq + 1] - batch.q_starts[seq];
    } else {
        seq = row / batch.const_q_len;
        t = row - seq * batch.const_q_len;
        q_len = batch.const_q_len;
    }
    const int kv_len = batch.kv_lens ? batch.kv_lens[seq] : batch.const_kv_len;
    int visible = kv_len - q_len + t + 1; // the query sits at position visible - 1
    visible = visible < 0 ? 0 : (visible > kv_len ? kv_len : visible);
    const int first = batch.window > 0 ? max(0, visible - batch.window) : 0;
    const int seq_row = batch.seq_ids ? batch.seq_ids[seq] : seq;

    for (int i = threadIdx.x; i < nh * d; i += kThreads) {
        q_s[i] = to_f32(q[int64_t(row) * nh * d + i]) * scale;
    }
    float acc[kOutPerThread];
#pragma unroll
    for (int i = 0; i < kOutPerThread; ++i) {
        acc[i] = 0.f;
    }
    const int out0 = int(blockIdx.y) * kThreads * kOutPerThread + int(threadIdx.x), n_out = nh * dv;
    const T *talk = static_cast<const T *>(gates.talk), *bias = static_cast<const T *>(gates.bias);

    for (int base = first; base < visible; base += kKeys) {
        const int j = base + lane;
        int64_t k_off = -1, v_off = -1;
        if (j < visible) {
            const int blk = j / kv.page_size;
            const int page = kv.block_table != nullptr ? kv.block_table[int64_t(seq_row) * kv.table_stride + blk] : blk;
            if (page < 0 || page >= kv.num_pages) {
                atomicOr(error_flag, kErrBadPage);
            } else {
                k_off = int64_t(page) * kv.page_stride + int64_t(j - blk * kv.page_size) * kv.token_stride;
                v_off = int64_t(page) * kv.page_stride + int64_t(j - blk * kv.page_size) * kv.vTokenStride();
            }
        }
        __syncthreads(); // q_s is complete; the block before this one has been read
        if (warp == 0) {
            v_off_s[lane] = v_off;
        }
        for (int h = warp; h < nh; h += kThreads / 32) {
            float w = 0.f;
            if (k_off >= 0) {
                const T *k_row = static_cast<const T *>(kv.k_base) + int64_t(h / share) * kv.head_stride + k_off;
                const float *q_row = q_s + h * d;
                float s = 0.f;
                for (int i = 0; i < d; ++i) {
                    s = fmaf(q_row[i], to_f32(k_row[i]), s);
                }
                if (gates.softcap > 0.f) {
                    s = gates.softcap * tanhf(s / gates.softcap);
                }
                if (gates.slopes != nullptr) {
                    s -= gates.slopes[h] * float(visible - 1 - j);
                }
                if (bias != nullptr) {
                    s += to_f32(bias[h]);
                }
                w = 1.f / (1.f + expf(-s));
            }
            w_s[h * kKeys + lane] = w;
        }
        __syncthreads();
        if (talk != nullptr) {
            for (int i = threadIdx.x; i < nh * kKeys; i += kThreads) {
                const T *t_row = talk + int64_t(i / kKeys) * nh;
                float m = 0.f;
                for (int g = 0; g < nh; ++g) {
                    m = fmaf(to_f32(t_row[g]), w_s[g * kKeys + (i & 31)], m);
                }
                m_s[i] = m;
            }
            __syncthreads();
        }
        const float *mixed = talk != nullptr ? m_s : w_s;
#pragma unroll
        for (int r = 0; r < kOutPerThread; ++r) {
            const int o = out0 + r * kThreads;
            if (o < n_out) {
                const int h = o / dv;
                const T *v_col = static_cast<const T *>(kv.v_base) + int64_t(h / share) * kv.vHeadStride() + (o - h * dv);
                for (int jj = 0; jj < kKeys; ++jj) {
                    const int64_t at = v_off_s[jj];
                    if (at >= 0) {
                        acc[r] = fmaf(mixed[h * kKeys + jj], to_f32(v_col[at]), acc[r]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < kOutPerThread; ++r) {
        const int o = out0 + r * kThreads;
        if (o < n_out) {
            out[int64_t(row) * out_stride + o] = from_f32<T>(acc[r]);
        }
    }
}

template <typename T>
void launch(cudaStream_t s, const KVView &kv, const AttnBatch &batch, const void *q, float scale, const GateArgs &gates, const AttnOut &out,
            int32_t *error_flag) {
    const int64_t n_out = int64_t(batch.nh) * kv.vDim();
    const dim3 grid(unsigned(batch.total_q), unsigned((n_out + kThreads * kOutPerThread - 1) / (kThreads * kOutPerThread)));
    const size_t smem = (size_t(batch.nh) * size_t(kv.d + 2 * kKeys) + 1) * sizeof(float) + kKeys * sizeof(int64_t);
    CHECK_ARGUMENT(smem <= 227 * 1024 && grid.y <= 65535, "gated attention: the heads of a query row do not fit");
    if (smem > 48 * 1024) {
        LLAISYS_CUDA_CHECK(cudaFuncSetAttribute(attention_gates_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    }
    attention_gates_kernel<T><<<grid, kThreads, smem, s>>>(kv, batch, static_cast<const T *>(q), scale, gates, static_cast<T *>(out.out),
                                                           out.row_stride ? out.row_stride : n_out, error_flag);
}

} // namespace

void attention_gates(stream_t stream, llaisysDataType_t dtype, const KVView &kv, const AttnBatch &batch, const void *q, float scale,
                     const GateArgs &gates, const AttnOut &out, int32_t *error_flag) {
    if (batch.total_q <= 0 || batch.nh <= 0) {
        return;
    }
    CHECK_ARGUMENT(kv.d > 0 && kv.vDim() > 0 && kv.nkvh > 0 && batch.nh % kv.nkvh == 0, "gated attention: nh must be a multiple of nkvh");
    CHECK_ARGUMENT(batch.keep_first == 0 && out.out != nullptr && out.part == nullptr && out.row_scale == nullptr,
                   "gated attention: neither kept tokens, partial results nor output factors");
    auto s = static_cast<cudaStream_t>(stream);
    switch (dtype) {
    case LLAISYS_DTYPE_F32:
        launch<float>(s, kv, batch, q, scale, gates, out, error_flag);
        break;
    case LLAISYS_DTYPE_F16:
        launch<__half>(s, kv, batch, q, scale, gates, out, error_flag);
        break;
    case LLAISYS_DTYPE_BF16:
        launch<__nv_bfloat16>(s, kv, batch, q, scale, gates, out, error_flag);
        break;
    default:
        EXCEPTION_UNSUPPORTED_DATATYPE(dtype);
    }
    check_launch("attention_gates");
}

} // namespace llaisys::kernels
