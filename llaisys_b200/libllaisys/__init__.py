"""ctypes binding of libllaisys.so: enums, handle types and the prototype of every exported symbol.

Mirrors the reference's binding package (python/llaisys/libllaisys/__init__.py:17-40 and its tensor.py,
ops.py, runtime.py, llaisys_types.py): the library sits next to this file and is loaded at import time, and
every prototype is declared immediately, so a missing symbol fails the import rather than a later call.
There is no pure-Python or CPU stand-in: without the compiled library the import raises.
"""
from __future__ import annotations

import ctypes
import sys
from ctypes import (CFUNCTYPE, POINTER, Structure, c_char_p, c_double, c_float, c_int, c_int32, c_int64, c_size_t,
                    c_ssize_t, c_uint8, c_void_p)
from enum import IntEnum
from pathlib import Path


class DeviceType(IntEnum):
    CPU = 0
    NVIDIA = 1
    COUNT = 2


class DataType(IntEnum):
    INVALID = 0
    BYTE = 1
    BOOL = 2
    I8 = 3
    I16 = 4
    I32 = 5
    I64 = 6
    U8 = 7
    U16 = 8
    U32 = 9
    U64 = 10
    F8 = 11
    F16 = 12
    F32 = 13
    F64 = 14
    C16 = 15
    C32 = 16
    C64 = 17
    C128 = 18
    BF16 = 19


class MemcpyKind(IntEnum):
    H2H = 0
    H2D = 1
    D2H = 2
    D2D = 3


class Status(IntEnum):
    """Return codes of the paged-KV entry points (include/llaisys/paged_kv.h)."""
    OK = 0
    INVALID = 1
    NO_PAGES = 2
    NO_SEQ = 3
    DEVICE = 4
    UNSUPPORTED = 5
    KERNEL = 6


llaisysDeviceType_t = c_int
llaisysDataType_t = c_int
llaisysMemcpyKind_t = c_int
llaisysStream_t = c_void_p
llaisysTensor_t = c_void_p
llaisysPagedKV_t = c_void_p


class LlaisysRuntimeAPI(Structure):
    """The twelve function pointers of include/llaisys/runtime.h, in order."""
    _fields_ = [
        ("get_device_count", CFUNCTYPE(c_int)),
        ("set_device", CFUNCTYPE(None, c_int)),
        ("device_synchronize", CFUNCTYPE(None)),
        ("create_stream", CFUNCTYPE(llaisysStream_t)),
        ("destroy_stream", CFUNCTYPE(None, llaisysStream_t)),
        ("stream_synchronize", CFUNCTYPE(None, llaisysStream_t)),
        ("malloc_device", CFUNCTYPE(c_void_p, c_size_t)),
        ("free_device", CFUNCTYPE(None, c_void_p)),
        ("malloc_host", CFUNCTYPE(c_void_p, c_size_t)),
        ("free_host", CFUNCTYPE(None, c_void_p)),
        ("memcpy_sync", CFUNCTYPE(None, c_void_p, c_void_p, c_size_t, llaisysMemcpyKind_t)),
        ("memcpy_async", CFUNCTYPE(None, c_void_p, c_void_p, c_size_t, llaisysMemcpyKind_t, llaisysStream_t)),
    ]


_T = llaisysTensor_t
_KV = llaisysPagedKV_t
_I32P = POINTER(c_int32)

# name -> (restype, argtypes). Every symbol declared in include/llaisys/*.h appears here exactly once.


class LlaisysQwen2Meta(Structure):
    """struct LlaisysQwen2Meta (reference: include/llaisys/models/qwen2.h:7-13)."""
    _fields_ = [("dtype", llaisysDataType_t), ("nlayer", c_size_t), ("hs", c_size_t), ("nh", c_size_t),
                ("nkvh", c_size_t), ("dh", c_size_t), ("di", c_size_t), ("maxseq", c_size_t), ("voc", c_size_t),
                ("epsilon", c_float), ("theta", c_float), ("end_token", c_int64)]


class LlaisysQwen2Weights(Structure):
    """struct LlaisysQwen2Weights (reference: include/llaisys/models/qwen2.h:15-31)."""
    _fields_ = [("in_embed", llaisysTensor_t), ("out_embed", llaisysTensor_t), ("out_norm_w", llaisysTensor_t)] + [
        (name, POINTER(llaisysTensor_t)) for name in (
            "attn_norm_w", "attn_q_w", "attn_q_b", "attn_k_w", "attn_k_b", "attn_v_w", "attn_v_b", "attn_o_w",
            "mlp_norm_w", "mlp_gate_w", "mlp_up_w", "mlp_down_w")]


class LlaisysWindowAttentionMeta(Structure):
    """struct LlaisysWindowAttentionMeta (include/llaisys/models/vozozen.h)."""
    _fields_ = [("heads", c_size_t), ("kv_heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("window", c_size_t),
                ("scale", c_float)]


class LlaisysGatedLinearMeta(Structure):
    """struct LlaisysGatedLinearMeta (include/llaisys/models/vozozen.h)."""
    _fields_ = [("heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("rank", c_size_t), ("tau", c_float)]


class LlaisysVozozenLayerMeta(Structure):
    """struct LlaisysVozozenLayerMeta (include/llaisys/models/vozozen.h)."""
    _fields_ = [("left", LlaisysWindowAttentionMeta), ("right", LlaisysGatedLinearMeta), ("left_scale", c_float),
                ("right_scale", c_float), ("ff", c_size_t)]


class LlaisysVozozenMeta(Structure):
    """struct LlaisysVozozenMeta (include/llaisys/models/vozozen.h)."""
    _fields_ = [("dtype", llaisysDataType_t), ("nlayer", c_size_t), ("layers", POINTER(LlaisysVozozenLayerMeta)),
                ("width", c_size_t), ("voc", c_size_t), ("maxseq", c_size_t), ("embed_scale", c_float), ("eps", c_float),
                ("logit_softcap", c_float), ("loop_start", c_size_t), ("loop_stop", c_size_t), ("loop_times", c_size_t),
                ("end_token", c_int64)]


class LlaisysDeltaMixerMeta(Structure):
    """struct LlaisysDeltaMixerMeta (include/llaisys/models/doderax.h)."""
    _fields_ = [("heads", c_size_t), ("kv_heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("taps", c_size_t),
                ("decay_rank", c_size_t), ("gate_rank", c_size_t)]


class LlaisysSinkAttentionMeta(Structure):
    """struct LlaisysSinkAttentionMeta (include/llaisys/models/doderax.h)."""
    _fields_ = [("heads", c_size_t), ("kv_heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("window", c_size_t),
                ("keep_first", c_size_t), ("rot_dims", c_size_t), ("rot_base", c_double), ("scale", c_float)]


class LlaisysDoderaxLayerMeta(Structure):
    """struct LlaisysDoderaxLayerMeta (include/llaisys/models/doderax.h)."""
    _fields_ = [("parallel", c_int), ("attn", LlaisysSinkAttentionMeta), ("delta", LlaisysDeltaMixerMeta), ("ff", c_size_t)]


class LlaisysDoderaxMeta(Structure):
    """struct LlaisysDoderaxMeta (include/llaisys/models/doderax.h)."""
    _fields_ = [("dtype", llaisysDataType_t), ("nlayer", c_size_t), ("layers", POINTER(LlaisysDoderaxLayerMeta)),
                ("width", c_size_t), ("voc", c_size_t), ("maxseq", c_size_t), ("pair_buckets", c_size_t), ("pair_mul_prev", c_int64),
                ("pair_mul_cur", c_int64), ("eps", c_float), ("logit_scale", c_float), ("end_token", c_int64)]


class LlaisysGatesAttentionMeta(Structure):
    """struct LlaisysGatesAttentionMeta (include/llaisys/models/lilovik.h)."""
    _fields_ = [("heads", c_size_t), ("kv_heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("scale", c_float),
                ("softcap", c_float), ("temp_coef", c_float), ("temp_every", c_float)]


class LlaisysLilovikLayerMeta(Structure):
    """struct LlaisysLilovikLayerMeta (include/llaisys/models/lilovik.h)."""
    _fields_ = [("recurrent", c_int), ("attn", LlaisysGatesAttentionMeta), ("gru_width", c_size_t), ("ff", c_size_t)]


class LlaisysLilovikMeta(Structure):
    """struct LlaisysLilovikMeta (include/llaisys/models/lilovik.h)."""
    _fields_ = [("dtype", llaisysDataType_t), ("nlayer", c_size_t), ("layers", POINTER(LlaisysLilovikLayerMeta)),
                ("width", c_size_t), ("voc", c_size_t), ("maxseq", c_size_t), ("eps", c_float), ("logit_scale", c_float),
                ("end_token", c_int64)]


class LlaisysLatentAttentionMeta(Structure):
    """struct LlaisysLatentAttentionMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("heads", c_size_t), ("dim", c_size_t), ("rot_dim", c_size_t), ("vdim", c_size_t), ("q_rank", c_size_t),
                ("kv_rank", c_size_t), ("rot_base", c_double), ("scale", c_float)]


class LlaisysFadingAttentionMeta(Structure):
    """struct LlaisysFadingAttentionMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("heads", c_size_t), ("kv_heads", c_size_t), ("dim", c_size_t), ("vdim", c_size_t), ("window", c_size_t),
                ("scale", c_float)]


class LlaisysStateSpaceMixerMeta(Structure):
    """struct LlaisysStateSpaceMixerMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("heads", c_size_t), ("groups", c_size_t), ("state", c_size_t), ("vdim", c_size_t), ("taps", c_size_t),
                ("norm_groups", c_size_t)]


class LlaisysExpertLayerMeta(Structure):
    """struct LlaisysExpertLayerMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("experts", c_size_t), ("identity", c_size_t), ("top", c_size_t), ("groups", c_size_t), ("keep", c_size_t),
                ("ff", c_size_t), ("shared_ff", c_size_t), ("scale", c_float)]


class LlaisysFolivikLayerMeta(Structure):
    """struct LlaisysFolivikLayerMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("mixer", c_int), ("latent", LlaisysLatentAttentionMeta), ("attn", LlaisysFadingAttentionMeta),
                ("ssm", LlaisysStateSpaceMixerMeta), ("mlp", LlaisysExpertLayerMeta)]


class LlaisysFolivikMeta(Structure):
    """struct LlaisysFolivikMeta (include/llaisys/models/folivik.h)."""
    _fields_ = [("dtype", llaisysDataType_t), ("nlayer", c_size_t), ("layers", POINTER(LlaisysFolivikLayerMeta)),
                ("width", c_size_t), ("voc", c_size_t), ("maxseq", c_size_t), ("eps", c_float), ("end_token", c_int64)]


class LlaisysNormAppend(Structure):
    """struct LlaisysNormAppend (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("q_at", c_int64), ("k_at", c_int64), ("v_at", c_int64),
                ("gate_at", c_int64), ("q_norm", c_void_p), ("k_norm", c_void_p), ("eps", c_float), ("gate_scale", c_float),
                ("q_out", c_void_p), ("row_scale", c_void_p), ("seq_ids_dev", c_void_p), ("positions_dev", c_void_p),
                ("n_rows", c_size_t), ("nh", c_size_t), ("rot_dims", c_size_t), ("rot_table", c_void_p), ("row_norm", c_int),
                ("bias", c_void_p), ("temp_coef", c_float), ("temp_every", c_float), ("head_scale", c_void_p)]


class LlaisysLatentAppend(Structure):
    """struct LlaisysLatentAppend (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("q_at", c_int64), ("kv_at", c_int64), ("gate_at", c_int64),
                ("q_rank", c_size_t), ("rank", c_size_t), ("rot_dims", c_size_t), ("nh", c_size_t), ("q_norm", c_void_p),
                ("kv_norm", c_void_p), ("eps", c_float), ("rot_table", c_void_p), ("q_latent", c_void_p), ("q_latent_stride", c_int64),
                ("row_scale", c_void_p), ("seq_ids_dev", c_void_p), ("positions_dev", c_void_p), ("n_rows", c_size_t)]


class LlaisysExpandedAttention(Structure):
    """struct LlaisysExpandedAttention (include/llaisys/mixers.h)."""
    _fields_ = [("q", c_void_p), ("k", c_void_p), ("k_shared", c_void_p), ("v", c_void_p), ("shared_stride", c_int64), ("tokens", c_size_t),
                ("nh", c_size_t), ("dim", c_size_t), ("rot_dim", c_size_t), ("vdim", c_size_t), ("page_starts_dev", c_void_p),
                ("q_starts_dev", c_void_p), ("kv_lens_dev", c_void_p), ("n_seqs", c_size_t), ("scale", c_float), ("out", c_void_p),
                ("out_stride", c_int64), ("row_scale", c_void_p)]


class LlaisysStateSpace(Structure):
    """struct LlaisysStateSpace (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("z_at", c_int64), ("x_at", c_int64), ("dt_at", c_int64),
                ("conv_w", c_void_p), ("conv_b", c_void_p), ("norm_w", c_void_p), ("a_log", c_void_p), ("dt_bias", c_void_p),
                ("d_skip", c_void_p), ("taps", c_size_t), ("heads", c_size_t), ("groups", c_size_t), ("dk", c_size_t), ("dv", c_size_t),
                ("norm_groups", c_size_t), ("eps", c_float), ("state", c_void_p), ("slot_stride", c_int64), ("seq_ids_dev", c_void_p),
                ("q_starts_dev", c_void_p), ("kv_lens_dev", c_void_p), ("n_seqs", c_size_t), ("n_rows", c_size_t),
                ("max_q_len", c_size_t), ("out", c_void_p), ("out_stride", c_int64), ("scratch", c_void_p), ("scratch_floats", c_size_t),
                ("scratch_segments", c_void_p), ("scratch_segment_floats", c_size_t)]


class LlaisysExperts(Structure):
    """struct LlaisysExperts (include/llaisys/mixers.h)."""
    _fields_ = [("experts", c_size_t), ("identity", c_size_t), ("top", c_size_t), ("groups", c_size_t), ("keep", c_size_t),
                ("width", c_size_t), ("ff", c_size_t), ("n_rows", c_size_t), ("scale", c_float), ("eps", c_float), ("gate_up", c_void_p),
                ("down", c_void_p), ("correction", c_void_p), ("logits", c_void_p), ("gain", c_void_p), ("h", c_void_p),
                ("chosen", c_void_p), ("weights", c_void_p), ("place", c_void_p), ("counts", c_void_p), ("line", c_void_p),
                ("rows", c_void_p), ("act", c_void_p), ("out", c_void_p), ("x", c_void_p), ("next", c_void_p)]


class LlaisysGates(Structure):
    """struct LlaisysGates (include/llaisys/mixers.h)."""
    _fields_ = [("softcap", c_float), ("slopes", c_void_p), ("bias", c_void_p), ("talk", c_void_p)]


class LlaisysMinGru(Structure):
    """struct LlaisysMinGru (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("z_at", c_int64), ("x_at", c_int64), ("g_at", c_int64),
                ("bias_z", c_void_p), ("bias_x", c_void_p), ("width", c_size_t), ("state", c_void_p), ("slot_stride", c_int64),
                ("seq_ids_dev", c_void_p), ("q_starts_dev", c_void_p), ("kv_lens_dev", c_void_p), ("n_seqs", c_size_t),
                ("n_rows", c_size_t), ("max_q_len", c_size_t), ("out", c_void_p), ("out_stride", c_int64), ("scratch", c_void_p),
                ("scratch_floats", c_size_t)]


class LlaisysGatedDelta(Structure):
    """struct LlaisysGatedDelta (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("q_at", c_int64), ("k_at", c_int64), ("v_at", c_int64),
                ("b_at", c_int64), ("a_at", c_int64), ("conv_q", c_void_p), ("conv_k", c_void_p), ("conv_v", c_void_p),
                ("decay_w", c_void_p), ("decay_ld", c_int64), ("a_log", c_void_p), ("dt_bias", c_void_p), ("norm_w", c_void_p),
                ("gate", c_void_p), ("gate_stride", c_int64), ("gate_silu", c_int), ("q_scale", c_float), ("eps", c_float),
                ("unit_eps", c_float), ("taps", c_size_t), ("heads", c_size_t), ("kv_heads", c_size_t), ("dk", c_size_t),
                ("dv", c_size_t), ("rank", c_size_t), ("state", c_void_p), ("slot_stride", c_int64), ("seq_ids_dev", c_void_p),
                ("q_starts_dev", c_void_p), ("kv_lens_dev", c_void_p), ("n_seqs", c_size_t), ("n_rows", c_size_t),
                ("max_q_len", c_size_t), ("out", c_void_p), ("out_stride", c_int64), ("scratch", c_void_p),
                ("scratch_floats", c_size_t), ("scratch_segments", c_void_p), ("scratch_segment_floats", c_size_t)]


class LlaisysGatedLinear(Structure):
    """struct LlaisysGatedLinear (include/llaisys/mixers.h)."""
    _fields_ = [("proj", c_void_p), ("row_stride", c_int64), ("q_at", c_int64), ("k_at", c_int64), ("v_at", c_int64),
                ("g_at", c_int64), ("z_at", c_int64), ("decay_w", c_void_p), ("decay_b", c_void_p), ("norm_w", c_void_p),
                ("tau", c_float), ("q_scale", c_float), ("eps", c_float), ("out_scale", c_float), ("heads", c_size_t),
                ("dk", c_size_t), ("dv", c_size_t), ("rank", c_size_t), ("state", c_void_p), ("slot_stride", c_int64),
                ("seq_ids_dev", c_void_p), ("q_starts_dev", c_void_p), ("kv_lens_dev", c_void_p), ("n_seqs", c_size_t),
                ("n_rows", c_size_t), ("max_q_len", c_size_t), ("out", c_void_p), ("out_stride", c_int64),
                ("scratch_raw", c_void_p), ("scratch_decay", c_void_p), ("scratch_segments", c_void_p),
                ("scratch_segment_floats", c_size_t)]


class LlaisysEngineEvent(Structure):
    """struct LlaisysEngineEvent (include/llaisys/serving.h)."""
    _fields_ = [("request", c_int64), ("token", c_int64), ("finished", c_int32), ("reserved", c_int32)]


_MODEL = c_void_p
ALL_REDUCE_FN = CFUNCTYPE(c_int, c_void_p, c_size_t, c_int, c_void_p)  # llaisysAllReduceFn

PROTOTYPES: dict[str, tuple] = {
    # runtime.h
    "llaisysGetRuntimeAPI": (POINTER(LlaisysRuntimeAPI), [llaisysDeviceType_t]),
    "llaisysSetContextRuntime": (None, [llaisysDeviceType_t, c_int]),
    "llaisysGetContextStream": (llaisysStream_t, []),
    # tensor.h
    "tensorCreate": (_T, [POINTER(c_size_t), c_size_t, llaisysDataType_t, llaisysDeviceType_t, c_int]),
    "tensorDestroy": (None, [_T]),
    "tensorGetData": (c_void_p, [_T]),
    "tensorGetNdim": (c_size_t, [_T]),
    "tensorGetShape": (None, [_T, POINTER(c_size_t)]),
    "tensorGetStrides": (None, [_T, POINTER(c_ssize_t)]),
    "tensorGetDataType": (llaisysDataType_t, [_T]),
    "tensorGetDeviceType": (llaisysDeviceType_t, [_T]),
    "tensorGetDeviceId": (c_int, [_T]),
    "tensorDebug": (None, [_T]),
    "tensorIsContiguous": (c_uint8, [_T]),
    "tensorLoad": (None, [_T, c_void_p]),
    "tensorView": (_T, [_T, POINTER(c_size_t), c_size_t]),
    "tensorPermute": (_T, [_T, POINTER(c_size_t)]),
    "tensorSlice": (_T, [_T, c_size_t, c_size_t, c_size_t]),
    # ops.h
    "llaisysAdd": (None, [_T, _T, _T]),
    "llaisysArgmax": (None, [_T, _T, _T]),
    "llaisysEmbedding": (None, [_T, _T, _T]),
    "llaisysLinear": (None, [_T, _T, _T, _T]),
    "llaisysLinearAccumulate": (None, [_T, _T, _T]),
    "llaisysRearrange": (None, [_T, _T]),
    "llaisysRmsNorm": (None, [_T, _T, _T, c_float]),
    "llaisysROPE": (None, [_T, _T, _T, c_float]),
    "llaisysSelfAttention": (None, [_T, _T, _T, _T, c_float]),
    "llaisysSwiGLU": (None, [_T, _T, _T]),
    # paged_kv.h
    "llaisysGetLastError": (c_char_p, []),
    "llaisysPagedKVCreate": (c_int, [POINTER(_KV), llaisysDeviceType_t, c_int, llaisysDataType_t, c_size_t, c_size_t,
                                     c_size_t, c_size_t, c_size_t, c_size_t, c_size_t]),
    "llaisysPagedKVDestroy": (c_int, [_KV]),
    "llaisysPagedKVSeqAdd": (c_int, [_KV, _I32P]),
    "llaisysPagedKVSeqReserve": (c_int, [_KV, c_int32, c_size_t]),
    "llaisysPagedKVSeqAssignPages": (c_int, [_KV, c_int32, _I32P, c_size_t]),
    "llaisysPagedKVSeqFree": (c_int, [_KV, c_int32]),
    "llaisysPagedKVNumFreePages": (c_size_t, [_KV]),
    "llaisysPagedKVNumSeqs": (c_size_t, [_KV]),
    "llaisysPagedKVSeqNumPages": (c_int64, [_KV, c_int32]),
    "llaisysPagedKVSeqPages": (c_int, [_KV, c_int32, _I32P, c_size_t]),
    "llaisysPagedKVPoolData": (c_void_p, [_KV, c_size_t]),
    "llaisysPagedKVLayerBytes": (c_size_t, [_KV]),
    "llaisysPagedKVBlockTableData": (c_void_p, [_KV]),
    "llaisysPagedKVFlush": (c_int, [_KV]),
    "llaisysPagedKVSetLaunchOverlap": (c_int, [_KV, c_int]),
    "llaisysPagedKVCheck": (c_int, [_KV]),
    "llaisysPagedKVAppend": (c_int, [_KV, c_size_t, c_void_p, c_void_p, _I32P, _I32P, c_size_t]),
    "llaisysPagedKVGather": (c_int, [_KV, c_size_t, c_int32, c_size_t, c_void_p, c_void_p]),
    "llaisysPagedAttentionDecode": (c_int, [_KV, c_size_t, c_void_p, c_void_p, _I32P, _I32P, c_size_t, c_size_t,
                                            c_float]),
    "llaisysPagedAttentionPrefill": (c_int, [_KV, c_size_t, c_void_p, c_void_p, _I32P, _I32P, _I32P, c_size_t,
                                             c_size_t, c_float]),
    "llaisysPagedAttentionDecodePartial": (c_int, [_KV, c_size_t, c_void_p, c_void_p, _I32P, _I32P, c_size_t,
                                                   c_size_t, c_float]),
    "llaisysLseMerge": (c_int, [llaisysDeviceType_t, c_int, c_void_p, llaisysDataType_t, c_void_p, c_size_t,
                                c_size_t, c_size_t]),
    "llaisysPagedKVAppendDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                        llaisysStream_t]),
    "llaisysPagedDecodeStepHost": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                           c_size_t, c_float]),
    "llaisysPagedKVSeqPublish": (c_int, [_KV, c_int32, POINTER(c_int64), c_size_t]),
    "llaisysPagedKVSeqMatchPrefix": (c_int, [_KV, c_int32, POINTER(c_int64), c_size_t, POINTER(c_size_t)]),
    "llaisysPagedKVSeqFork": (c_int, [_KV, c_int32, c_size_t, _I32P]),
    "llaisysPagedKVPageRefCount": (c_int, [_KV, c_int32]),
    "llaisysPagedKVNumCachedPages": (c_size_t, [_KV]),
    "llaisysPagedKVRopeAppendDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                            c_size_t, c_float, llaisysStream_t]),
    "llaisysPagedAttentionDecodeDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                               c_size_t, c_size_t, c_float, llaisysStream_t]),
    "llaisysPagedAttentionDecodePartialDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p,
                                                      c_size_t, c_size_t, c_size_t, c_float, llaisysStream_t]),
    "llaisysPagedAttentionPrefillDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                                c_size_t, c_size_t, c_size_t, c_size_t, c_size_t, c_float,
                                                llaisysStream_t]),
    "llaisysPagedAttentionDecodeNoAlloc": (c_int, [c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t, c_size_t,
                                                   c_void_p, c_void_p, c_size_t, c_size_t, c_size_t, c_size_t,
                                                   llaisysDataType_t, c_float, c_void_p, llaisysStream_t]),
    "llaisysPeerExchangeCreate": (c_int, [POINTER(c_void_p), c_int, c_int, c_int, c_size_t]),
    "llaisysPeerExchangeDestroy": (None, [c_void_p]),
    "llaisysPeerExchangeHandle": (c_int, [c_void_p, c_void_p]),
    "llaisysPeerExchangeConnect": (c_int, [c_void_p, c_void_p]),
    "llaisysPagedAttentionDecodeSplitDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                                    c_size_t, c_size_t, c_float, c_void_p, llaisysStream_t]),
    "llaisysPeerExchangeStatus": (c_int, [c_void_p, llaisysStream_t]),
    "llaisysPeerExchangeSetWaitLimit": (c_int, [c_void_p, ctypes.c_uint32]),
    "llaisysPeerExchangeDisconnect": (c_int, [c_void_p]),
    "llaisysPagedDecodeStepDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                          c_size_t, c_size_t, c_size_t, c_float, llaisysStream_t]),
    "llaisysPagedKVLastKernel": (c_int, [_KV]),
    "llaisysLastAttentionKernel": (c_int, []),
    "llaisysPagedAttentionDecodeNoAllocStatus": (c_int, [c_int, llaisysStream_t, _I32P]),
    "llaisysSetLinearPolicy": (c_int, [c_int]),
    # include/llaisys/models/qwen2.h
    "llaisysQwen2ModelCreate": (_MODEL, [POINTER(LlaisysQwen2Meta), llaisysDeviceType_t, POINTER(c_int), c_int]),
    "llaisysQwen2ModelDestroy": (None, [_MODEL]),
    "llaisysQwen2ModelWeights": (POINTER(LlaisysQwen2Weights), [_MODEL]),
    "llaisysQwen2ModelInfer": (c_int64, [_MODEL, POINTER(c_int64), c_size_t]),
    "llaisysQwen2ModelConfigureCache": (c_int, [_MODEL, c_size_t, c_size_t]),
    "llaisysQwen2ModelSeqAdd": (c_int, [_MODEL, _I32P]),
    "llaisysQwen2ModelSeqAddWithPrefix": (c_int, [_MODEL, POINTER(c_int64), c_size_t, _I32P, POINTER(c_size_t)]),
    "llaisysQwen2ModelSeqFree": (c_int, [_MODEL, c_int32]),
    "llaisysQwen2ModelReset": (c_int, [_MODEL]),
    "llaisysQwen2ModelStep": (c_int, [_MODEL, _I32P, _I32P, c_size_t, POINTER(c_int64), POINTER(c_int64)]),
    "llaisysQwen2ModelDecodeLoop": (c_int, [_MODEL, _I32P, c_size_t, POINTER(c_int64), c_size_t, POINTER(c_int64)]),
    "llaisysQwen2ModelLastLogits": (c_int, [_MODEL, POINTER(c_float), c_size_t]),
    "llaisysQwen2ModelLastLoopMs": (c_double, [_MODEL]),
    "llaisysQwen2ModelCreateTP": (_MODEL, [POINTER(LlaisysQwen2Meta), llaisysDeviceType_t, c_int, c_int, c_int]),
    "llaisysNcclUniqueId": (c_int, [c_void_p]),
    "llaisysQwen2ModelSetAllReduceNccl": (c_int, [_MODEL, c_void_p]),
    "llaisysQwen2ModelSetAllReduceCallback": (c_int, [_MODEL, ALL_REDUCE_FN, c_void_p]),
    # include/llaisys/mixers.h
    "llaisysPagedKVCreateLayers": (c_int, [POINTER(_KV), llaisysDeviceType_t, c_int, llaisysDataType_t, c_size_t,
                                           POINTER(c_size_t), POINTER(c_size_t), POINTER(c_size_t), c_size_t, c_size_t,
                                           c_size_t, c_size_t]),
    "llaisysPagedKVNormAppendDev": (c_int, [_KV, c_size_t, POINTER(LlaisysNormAppend), llaisysStream_t]),
    "llaisysPagedAttentionOptDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                            c_size_t, c_size_t, c_size_t, c_size_t, c_float, c_size_t, c_size_t, c_void_p,
                                            c_size_t, llaisysStream_t]),
    "llaisysPagedAttentionGatesDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t,
                                              c_size_t, c_size_t, c_size_t, c_size_t, c_float, c_size_t, POINTER(LlaisysGates),
                                              c_size_t, llaisysStream_t]),
    "llaisysMinGruScratchFloats": (c_size_t, [c_size_t, c_size_t]),
    "llaisysRotaryTableWideDev": (c_int, [llaisysDeviceType_t, c_int, c_void_p, c_void_p, c_void_p, c_size_t, c_size_t, llaisysStream_t]),
    "llaisysPagedAttentionFadeDev": (c_int, [_KV, c_size_t, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_size_t, c_size_t, c_size_t,
                                             c_size_t, c_size_t, c_float, c_size_t, c_void_p, c_void_p, c_size_t, llaisysStream_t]),
    "llaisysPagedKVCreateLatents": (c_int, [POINTER(_KV), llaisysDeviceType_t, c_int, llaisysDataType_t, c_size_t, POINTER(c_size_t),
                                            POINTER(c_size_t), c_size_t, c_size_t, c_size_t, c_size_t]),
    "llaisysPagedKVLatentAppendDev": (c_int, [_KV, c_size_t, POINTER(LlaisysLatentAppend), llaisysStream_t]),
    "llaisysRotatePairsDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, c_void_p, c_size_t, c_size_t, c_void_p, c_size_t, c_size_t,
                                      c_void_p, c_size_t, c_size_t, llaisysStream_t]),
    "llaisysPagedKVLatentGatherDev": (c_int, [_KV, c_size_t, c_void_p, c_int64, c_void_p, c_void_p, c_void_p, c_size_t, c_size_t,
                                              llaisysStream_t]),
    "llaisysPagedAttentionExpandedDev": (c_int, [_KV, POINTER(LlaisysExpandedAttention), llaisysStream_t]),
    "llaisysStateSpaceDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, POINTER(LlaisysStateSpace), c_int, llaisysStream_t]),
    "llaisysStateSpaceSizes": (None, [llaisysDataType_t, c_size_t, c_size_t, c_size_t, c_size_t, c_size_t, c_size_t, POINTER(c_size_t),
                                      POINTER(c_size_t), POINTER(c_size_t)]),
    "llaisysExpertsDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, POINTER(LlaisysExperts), llaisysStream_t]),
    "llaisysMinGruDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, POINTER(LlaisysMinGru), c_int, llaisysStream_t]),
    "llaisysRotaryTableDev": (c_int, [llaisysDeviceType_t, c_int, c_void_p, c_void_p, c_void_p, c_size_t, c_size_t,
                                      llaisysStream_t]),
    "llaisysGatedDeltaDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, POINTER(LlaisysGatedDelta), c_int,
                                     llaisysStream_t]),
    "llaisysGatedDeltaSizes": (None, [llaisysDataType_t] + [c_size_t] * 6 + [POINTER(c_size_t)] * 3),
    "llaisysGatedLinearDev": (c_int, [llaisysDeviceType_t, c_int, llaisysDataType_t, POINTER(LlaisysGatedLinear), c_int,
                                      llaisysStream_t]),
    "llaisysGatedLinearSegmentFloats": (c_size_t, [llaisysDataType_t, c_size_t, c_size_t, c_size_t]),
    # include/llaisys/models/model.h
    "llaisysModelDestroy": (None, [_MODEL]),
    "llaisysModelVocab": (c_size_t, [_MODEL]),
    "llaisysModelLoadTensor": (c_int, [_MODEL, c_char_p, llaisysDataType_t, POINTER(c_size_t), c_size_t, c_void_p,
                                       POINTER(c_int)]),
    "llaisysModelMissingTensors": (c_size_t, [_MODEL, c_char_p, c_size_t]),
    "llaisysModelConfigureCache": (c_int, [_MODEL, c_size_t, c_size_t, c_size_t]),
    "llaisysModelSeqAdd": (c_int, [_MODEL, _I32P]),
    "llaisysModelSeqAddWithPrefix": (c_int, [_MODEL, POINTER(c_int64), c_size_t, _I32P, POINTER(c_size_t)]),
    "llaisysModelSeqFree": (c_int, [_MODEL, c_int32]),
    "llaisysModelFreePages": (c_size_t, [_MODEL]),
    "llaisysModelInfer": (c_int, [_MODEL, POINTER(c_int64), c_size_t, POINTER(c_int64)]),
    "llaisysModelReset": (c_int, [_MODEL]),
    "llaisysModelStep": (c_int, [_MODEL, _I32P, _I32P, c_size_t, POINTER(c_int64), POINTER(c_int64)]),
    "llaisysModelStepRows": (c_int, [_MODEL, _I32P, _I32P, c_size_t, POINTER(c_int64), _I32P, c_size_t, POINTER(c_int64)]),
    "llaisysModelDecodeLoop": (c_int, [_MODEL, _I32P, c_size_t, POINTER(c_int64), c_size_t, POINTER(c_int64)]),
    "llaisysModelLastLogits": (c_int, [_MODEL, POINTER(c_float), c_size_t]),
    "llaisysModelLastLoopMs": (c_double, [_MODEL]),
    "llaisysModelRecordStream": (c_int, [_MODEL, c_int]),
    "llaisysModelLayerStream": (c_int, [_MODEL, POINTER(c_float), c_size_t, POINTER(c_size_t)]),
    # include/llaisys/models/vozozen.h
    # include/llaisys/models/lilovik.h
    "llaisysLilovikModelCreate": (_MODEL, [POINTER(LlaisysLilovikMeta), llaisysDeviceType_t, c_int]),
    # include/llaisys/models/folivik.h
    "llaisysFolivikModelCreate": (_MODEL, [POINTER(LlaisysFolivikMeta), llaisysDeviceType_t, c_int]),
    # include/llaisys/models/doderax.h
    "llaisysDoderaxModelCreate": (_MODEL, [POINTER(LlaisysDoderaxMeta), llaisysDeviceType_t, c_int]),
    "llaisysVozozenModelCreate": (_MODEL, [POINTER(LlaisysVozozenMeta), llaisysDeviceType_t, c_int]),
    # include/llaisys/serving.h
    "llaisysEngineCreate": (c_int, [POINTER(c_void_p), _MODEL, c_size_t, c_size_t, c_size_t]),
    "llaisysEngineDestroy": (None, [c_void_p]),
    "llaisysEngineSubmit": (c_int, [c_void_p, POINTER(c_int64), c_size_t, c_size_t, c_int64, POINTER(c_int64)]),
    "llaisysEngineStep": (c_int, [c_void_p, POINTER(LlaisysEngineEvent), c_size_t, POINTER(c_size_t)]),
    "llaisysEngineCancel": (c_int, [c_void_p, c_int64]),
    "llaisysEngineNumWaiting": (c_size_t, [c_void_p]),
    "llaisysEngineNumRunning": (c_size_t, [c_void_p]),
    "llaisysEngineCounter": (c_size_t, [c_void_p, c_int]),
}


def library_path() -> Path:
    if sys.platform.startswith("linux"):
        name = "libllaisys.so"
    elif sys.platform == "win32":
        name = "llaisys.dll"
    elif sys.platform == "darwin":
        name = "llaisys.dylib"
    else:
        raise RuntimeError("Unsupported platform")
    return Path(__file__).parent / name


def load_shared_library() -> ctypes.CDLL:
    path = library_path()
    if not path.is_file():
        raise FileNotFoundError(
            f"Shared library not found: {path}. Build it with `python llaisys_b200/build.py`; "
            "there is no Python fallback for the compiled kernels.")
    lib = ctypes.CDLL(str(path))
    for name, (restype, argtypes) in PROTOTYPES.items():
        fn = getattr(lib, name)  # AttributeError here = the library is older than this binding
        fn.restype = restype
        fn.argtypes = argtypes
    return lib


LIB_LLAISYS = load_shared_library()

__all__ = [
    "LIB_LLAISYS", "PROTOTYPES", "LlaisysRuntimeAPI", "llaisysStream_t", "llaisysTensor_t", "llaisysPagedKV_t",
    "llaisysDataType_t", "DataType", "llaisysDeviceType_t", "DeviceType", "llaisysMemcpyKind_t", "MemcpyKind",
    "Status", "library_path", "LlaisysQwen2Meta", "LlaisysQwen2Weights", "LlaisysEngineEvent",
    "LlaisysNormAppend", "LlaisysGatedLinear", "LlaisysGatedDelta", "LlaisysDoderaxMeta", "LlaisysDoderaxLayerMeta",
    "LlaisysLatentAppend", "LlaisysExpandedAttention", "LlaisysStateSpace", "LlaisysExperts",
    "LlaisysGates", "LlaisysMinGru", "LlaisysLilovikMeta", "LlaisysLilovikLayerMeta", "LlaisysGatesAttentionMeta",
    "LlaisysFolivikMeta", "LlaisysFolivikLayerMeta", "LlaisysLatentAttentionMeta", "LlaisysFadingAttentionMeta",
    "LlaisysStateSpaceMixerMeta", "LlaisysExpertLayerMeta",
    "LlaisysSinkAttentionMeta", "LlaisysDeltaMixerMeta", "LlaisysVozozenMeta", "LlaisysVozozenLayerMeta", "LlaisysWindowAttentionMeta", "LlaisysGatedLinearMeta", "ALL_REDUCE_FN",
]
