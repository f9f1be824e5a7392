"""Vozozen on the C model API (include/llaisys/models/vozozen.h): layers of sliding-window attention and gated linear
attention side by side, with a range of layers run several times over. Runs on NVIDIA devices, in bfloat16 or float32.
"""
from __future__ import annotations

import ctypes
import json
from ctypes import c_int, c_size_t
from pathlib import Path
from typing import Mapping

import numpy as np

from ..libllaisys import (LIB_LLAISYS, DataType, DeviceType, LlaisysGatedLinearMeta, LlaisysVozozenLayerMeta,
                          LlaisysVozozenMeta, LlaisysWindowAttentionMeta)
from ..paged_kv import LlaisysError, _check
from .base import DTYPE_NAMES, CausalLM
from .weights import LIBRARY_DTYPE, checkpoint_files


def _layer_meta(index: int, entry: Mapping, decay_rank: int) -> LlaisysVozozenLayerMeta:
    if entry.get("type") != "parallel":
        raise ValueError(f"layer {index}: unknown layer type {entry.get('type')!r}")
    mixer, mlp = entry["mixer"], entry.get("mlp")
    left, right = mixer["left"], mixer["right"]
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
    return LlaisysVozozenLayerMeta(
        left=LlaisysWindowAttentionMeta(heads=int(left["heads"]), kv_heads=int(left["kv_heads"]), dim=int(left["dim"]),
                                        vdim=int(left["vdim"]), window=int(left["mask"]["size"]), scale=float(left["scale"])),
        right=LlaisysGatedLinearMeta(heads=int(right["heads"]), dim=int(right["dim"]), vdim=int(right["vdim"]),
                                     rank=decay_rank, tau=float(right["tau"])),
        left_scale=float(mixer["left_scale"]), right_scale=float(mixer["right_scale"]), ff=int(mlp["ff"]) if mlp else 0)


def build_meta(config: Mapping, decay_ranks: list[int], dtype: DataType, max_seq_len: int | None = None) -> LlaisysVozozenMeta:
    """The C description of a model. decay_ranks: rows of every layer's `mix.right.a1` (a size only the weights hold)."""
    entries = config["layers"]
    layers = (LlaisysVozozenLayerMeta * len(entries))(*[_layer_meta(i, e, decay_ranks[i]) for i, e in enumerate(entries)])
    loop = config.get("loop")
    eos = config.get("eos_token_id")
    meta = LlaisysVozozenMeta(
        dtype=int(dtype), nlayer=len(entries), layers=layers, width=int(config["width"]), voc=int(config["vocab"]),
        maxseq=int(max_seq_len or config.get("max_position_embeddings", 4096)),
        embed_scale=float(config["embedding"]["scale"]), eps=float(config["norm"]["eps"]),
        logit_softcap=float(config.get("logit_softcap") or 0.0),
        loop_start=int(loop["start"]) if loop else 0, loop_stop=int(loop["stop"]) if loop else 0,
        loop_times=int(loop["times"]) if loop else 0, end_token=-1 if eos is None else int(eos))
    meta._layers = layers  # keeps the array alive as long as the struct
    return meta


def weight_shapes(config: Mapping, decay_ranks: list[int]) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a model's weights."""
    width, vocab = int(config["width"]), int(config["vocab"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (vocab, width)}
    if config.get("loop"):
        shapes["loop.in"] = (width, 2 * width)
    for i, entry in enumerate(config["layers"]):
        left, right, rank = entry["mixer"]["left"], entry["mixer"]["right"], decay_ranks[i]
        h, g, d, dv = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
        rh, rd, rv = right["heads"], right["dim"], right["vdim"]
        ml, mr = f"l{i}.mix.left.", f"l{i}.mix.right."
        shapes |= {f"l{i}.norm1": (width,), ml + "q": (h * d, width), ml + "k": (g * d, width), ml + "v": (g * dv, width),
                   ml + "q.norm": (d,), ml + "k.norm": (d,), ml + "g": (h, width), ml + "o": (width, h * dv),
                   mr + "q": (rh * rd, width), mr + "k": (rh * rd, width), mr + "v": (rh * rv, width),
                   mr + "g": (rh * rv, width), mr + "o": (width, rh * rv), mr + "norm": (rv,), mr + "a1": (rank, width),
                   mr + "a2": (rh * rd, rank), mr + "a2.b": (rh * rd,)}
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            shapes |= {f"l{i}.norm2": (width,), f"l{i}.mlp.up": (ff, width), f"l{i}.mlp.down": (width, ff)}
    return shapes | {"final.norm": (width,), "head": (vocab, width)}


class Vozozen(CausalLM):
    def __init__(self, model_path=None, device: DeviceType = DeviceType.NVIDIA, *, device_id: int = 0,
                 config: Mapping | None = None, state_dict: Mapping | None = None, dtype: DataType | None = None,
                 max_seq_len: int | None = None):
        """From a checkpoint directory, or from a config and a state dict of numpy arrays (float32, or bfloat16 as its
        16-bit words) or torch tensors. dtype: of matrix products and activations; bfloat16 when neither this argument nor
        the config names one."""
        files = []
        if model_path is not None:
            config = json.loads((Path(model_path) / "config.json").read_text())
            files = list(checkpoint_files(model_path))
        if config is None:
            raise ValueError("Vozozen needs a checkpoint directory or a config")
        if dtype is None:
            dtype = DTYPE_NAMES.get(str(config.get("torch_dtype", "bfloat16")), DataType.BF16)
        shapes = {name: f.shape(name) for f in files for name in f.names()}
        if state_dict is not None:
            shapes |= {name: tuple(value.shape) for name, value in state_dict.items()}
        missing = [n for n in (f"l{i}.mix.right.a1" for i in range(len(config["layers"]))) if n not in shapes]
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors, e.g. {missing[:3]}")
        ranks = [int(shapes[f"l{i}.mix.right.a1"][0]) for i in range(len(config["layers"]))]
        self.config = dict(config)
        self.meta = build_meta(config, ranks, dtype, max_seq_len)
        self.vocab, self.max_seq, self.end_token = int(self.meta.voc), int(self.meta.maxseq), int(self.meta.end_token)
        self.dtype, self.device, self.device_id = dtype, device, device_id
        self._model = LIB_LLAISYS.llaisysVozozenModelCreate(ctypes.byref(self.meta), int(device), device_id)
        if not self._model:
            raise RuntimeError("llaisysVozozenModelCreate failed: " + (LIB_LLAISYS.llaisysGetLastError() or b"").decode())
        for f in files:
            for name in f.names():
                if f.dtype(name) in LIBRARY_DTYPE:
                    self._load(name, f.array(name), LIBRARY_DTYPE[f.dtype(name)])
        for name, value in (state_dict or {}).items():
            self.load_tensor(name, value)
        first = ctypes.create_string_buffer(256)
        n_missing = int(LIB_LLAISYS.llaisysModelMissingTensors(self._model, first, len(first)))
        if n_missing:
            raise ValueError(f"checkpoint lacks {n_missing} tensors, e.g. {first.value.decode()}")

    def load_tensor(self, name: str, value) -> None:
        """Copies one weight: a numpy array (float32 / float16, or uint16 holding bfloat16) or a torch tensor."""
        if not isinstance(value, np.ndarray):
            import torch
            host = value.detach().to("cpu").contiguous()
            if host.dtype == torch.bfloat16:
                value = host.view(torch.int16).numpy().view(np.uint16)
            else:
                value = host.float().numpy()
        kind = {np.dtype(np.float32): DataType.F32, np.dtype(np.float16): DataType.F16,
                np.dtype(np.uint16): DataType.BF16}.get(value.dtype)
        if kind is None:
            raise ValueError(f"{name}: unsupported array type {value.dtype}")
        self._load(name, value, kind)

    def _load(self, name: str, array: np.ndarray, kind: DataType) -> None:
        array = np.ascontiguousarray(array)
        shape = (c_size_t * array.ndim)(*array.shape)
        known = c_int(0)
        try:
            _check(LIB_LLAISYS.llaisysModelLoadTensor(self._model, name.encode(), int(kind), shape, array.ndim,
                                                      array.ctypes.data, ctypes.byref(known)))
        except LlaisysError as err:
            raise ValueError(str(err)) from err

    # ---- development aid ------------------------------------------------------------------------------------------------

    def record_stream(self, enable: bool = True) -> None:
        """Keep the residual stream after every layer run of the steps that follow (slow)."""
        _check(LIB_LLAISYS.llaisysVozozenModelRecordStream(self._model, int(enable)))

    def layer_stream(self) -> np.ndarray:
        """float32 [layer runs, rows, width] of the last step."""
        n = c_size_t(0)
        _check(LIB_LLAISYS.llaisysVozozenModelLayerStream(self._model, None, 0, ctypes.byref(n)))
        out = np.zeros(n.value, dtype=np.float32)
        _check(LIB_LLAISYS.llaisysVozozenModelLayerStream(
            self._model, out.ctypes.data_as(ctypes.POINTER(ctypes.c_float)), out.size, ctypes.byref(n)))
        loop = self.config.get("loop")
        runs = len(self.config["layers"]) + ((loop["stop"] - loop["start"]) * (loop["times"] - 1) if loop else 0)
        return out.reshape(runs, -1, int(self.meta.width))
