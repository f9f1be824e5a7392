"""llaisys_b200 -- B200-native implementation of the LLAISYS KV-cache / self-attention path.

The public names are the reference frontend's (python/llaisys/__init__.py:1-20): RuntimeAPI, DeviceType,
DataType, MemcpyKind, Stream, Tensor, Ops. `PagedKVCache`, `lse_merge` and `LlaisysError` are new: the
reference has no KV cache. A program written against the reference package can switch with
`import llaisys_b200 as llaisys`.
"""
from .libllaisys import DataType, DeviceType, MemcpyKind, Status
from .libllaisys import llaisysStream_t as Stream
from .runtime import RuntimeAPI, context_stream, set_context_runtime
from .tensor import Tensor
from .ops import Ops
from .paged_kv import (Kernel, LlaisysError, PagedKVCache, decode_no_alloc, decode_no_alloc_status, experts_dev, gated_delta_dev,
                       gated_delta_sizes, gated_linear_dev, gated_linear_segment_floats, last_attention_kernel, lse_merge, min_gru_dev,
                       min_gru_scratch_floats, rotary_table_dev, rotary_table_wide_dev, rotate_pairs_dev, state_space_dev,
                       state_space_sizes)
from . import models
from .serving import Engine

__all__ = [
    "RuntimeAPI", "DeviceType", "DataType", "MemcpyKind", "Stream", "Tensor", "Ops", "models", "Engine",
    "PagedKVCache", "lse_merge", "decode_no_alloc", "decode_no_alloc_status", "LlaisysError", "Status", "Kernel",
    "gated_delta_dev", "gated_delta_sizes", "gated_linear_dev", "gated_linear_segment_floats", "min_gru_dev", "min_gru_scratch_floats", "rotary_table_dev", "rotary_table_wide_dev",
    "rotate_pairs_dev", "state_space_dev", "state_space_sizes", "experts_dev", "last_attention_kernel", "context_stream", "set_context_runtime",
]
