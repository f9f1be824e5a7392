"""What every decoder-only model of the package can do, on the generic C model API (include/llaisys/models/model.h):
batched sequences, mixed steps, generation, sampling. A family's class derives from CausalLM, creates its handle and loads
its weights; everything here works on the handle alone.
"""
from __future__ import annotations

import ctypes
import itertools
import json
from ctypes import c_float, c_int, c_int32, c_int64, c_size_t
from pathlib import Path
from typing import Mapping, Sequence

import numpy as np

from ..libllaisys import LIB_LLAISYS, DataType, DeviceType
from ..paged_kv import LlaisysError, _check
from .weights import LIBRARY_DTYPE, checkpoint_files

DTYPE_NAMES = {"bfloat16": DataType.BF16, "float16": DataType.F16, "float32": DataType.F32}

_I32P = ctypes.POINTER(c_int32)
_I64P = ctypes.POINTER(c_int64)


class CausalLM:
    _model = None   # the C handle
    vocab: int      # vocabulary size
    max_seq: int    # default bound of a sequence
    end_token: int  # < 0: none

    @classmethod
    def from_pretrained(cls, model_path, device, **kwargs):
        """A model from a checkpoint directory (config.json + *.safetensors)."""
        return cls(model_path, device, **kwargs)

    def close(self) -> None:
        if getattr(self, "_model", None):
            LIB_LLAISYS.llaisysModelDestroy(self._model)
            self._model = None

    def __del__(self):
        self.close()

    # ---- one prompt in, prompt + completion out (the call of the reference's test, test/test_infer.py:57-80) ----------------------------------------------------

    def generate(self, inputs: Sequence[int], max_new_tokens: int | None = None, top_k: int = 1, top_p: float = 0.8,
                 temperature: float = 0.8, seed: int | None = None) -> list[int]:
        """Greedy when top_k == 1 (the argmax is taken on the device); otherwise temperature / top-k / top-p sampling
        on the host from the step's logits. Stops after max_new_tokens or at the model's end token (kept in the
        output, as Hugging Face's generate does)."""
        inputs = [int(t) for t in inputs]
        if not inputs:
            return []
        if max_new_tokens is None:
            max_new_tokens = max(0, self.max_seq - len(inputs))
        _check(LIB_LLAISYS.llaisysModelReset(self._model))
        rng = np.random.default_rng(seed)
        out = list(inputs)
        feed = inputs
        for _ in range(max_new_tokens):
            arr, nxt = (c_int64 * len(feed))(*feed), c_int64(0)
            _check(LIB_LLAISYS.llaisysModelInfer(self._model, arr, len(feed), ctypes.byref(nxt)))
            token = nxt.value
            if top_k != 1:
                token = self._sample(self.last_logits()[0], top_k, top_p, temperature, rng)
            out.append(token)
            if token == self.end_token:
                break
            feed = [token]
        return out

    @staticmethod
    def _sample(logits: np.ndarray, top_k: int, top_p: float, temperature: float, rng) -> int:
        scores = logits.astype(np.float64) / max(float(temperature), 1e-6)
        order = np.argsort(-scores, kind="stable")
        if top_k and top_k > 0:
            order = order[:top_k]
        probs = np.exp(scores[order] - scores[order[0]])
        probs /= probs.sum()
        if 0.0 < top_p < 1.0:
            keep = int(np.searchsorted(np.cumsum(probs), top_p, side="left")) + 1
            order, probs = order[:keep], probs[:keep] / probs[:keep].sum()
        return int(order[rng.choice(len(order), p=probs)])

    # ---- batched sequences ----------------------------------------------------------------------------------------------

    def configure_cache(self, max_seqs: int, max_tokens: int, pool_tokens: int = 0) -> None:
        """At most max_seqs live sequences of at most max_tokens tokens; pool_tokens bounds the tokens all of them together
        can hold (0: max_seqs * max_tokens)."""
        _check(LIB_LLAISYS.llaisysModelConfigureCache(self._model, max_seqs, max_tokens, pool_tokens))

    @property
    def free_pages(self) -> int:
        return int(LIB_LLAISYS.llaisysModelFreePages(self._model))

    def add_seq(self) -> int:
        seq = c_int32(-1)
        _check(LIB_LLAISYS.llaisysModelSeqAdd(self._model, ctypes.byref(seq)))
        return seq.value

    def add_seq_with_prefix(self, tokens: Sequence[int]) -> tuple[int, int]:
        """New sequence that reuses cached K/V of earlier sequences starting with the same tokens (whole pages, leaving
        at least one token to run). -> (sequence id, tokens already covered); feed tokens[covered:] to step()."""
        arr = np.ascontiguousarray(tokens, dtype=np.int64)
        seq, matched = c_int32(-1), ctypes.c_size_t(0)
        _check(LIB_LLAISYS.llaisysModelSeqAddWithPrefix(self._model, arr.ctypes.data_as(_I64P),
                                                             arr.size, ctypes.byref(seq), ctypes.byref(matched)))
        return seq.value, int(matched.value)

    def free_seq(self, seq: int) -> None:
        _check(LIB_LLAISYS.llaisysModelSeqFree(self._model, seq))

    def step(self, seq_ids: Sequence[int], tokens: Sequence[Sequence[int]]) -> list[int]:
        """Appends tokens[i] to sequence seq_ids[i] (any mix of prefill chunks and single decode tokens) and returns
        the greedy next token of every sequence."""
        n = len(seq_ids)
        if len(tokens) != n:
            raise ValueError("one token list per sequence")
        ids = np.ascontiguousarray(seq_ids, dtype=np.int32)
        # (one pass over the token lists: building an array per sequence and concatenating them cost more than the
        # library call's own host work in a 64-sequence decode step)
        counts = np.fromiter(map(len, tokens), dtype=np.int32, count=n)
        flat = np.fromiter(itertools.chain.from_iterable(tokens), dtype=np.int64, count=int(counts.sum()))
        nxt = np.zeros(n, dtype=np.int64)
        _check(LIB_LLAISYS.llaisysModelStep(
            self._model, ids.ctypes.data_as(_I32P), counts.ctypes.data_as(_I32P), n,
            flat.ctypes.data_as(_I64P), nxt.ctypes.data_as(_I64P)))
        return nxt.tolist()

    def step_rows(self, seq_ids: Sequence[int], tokens: Sequence[Sequence[int]], rows: Sequence[int]) -> np.ndarray:
        """The same step with logits at chosen rows of the packed tokens (tokens[0] + tokens[1] + ...) instead of at each
        sequence's last token; no rows skip the vocabulary projection. -> float32 [len(rows), vocab]"""
        ids = np.ascontiguousarray(seq_ids, dtype=np.int32)
        counts = np.fromiter(map(len, tokens), dtype=np.int32, count=len(tokens))
        flat = np.fromiter(itertools.chain.from_iterable(tokens), dtype=np.int64, count=int(counts.sum()))
        want = np.ascontiguousarray(rows, dtype=np.int32)
        nxt = np.zeros(max(want.size, 1), dtype=np.int64)
        _check(LIB_LLAISYS.llaisysModelStepRows(
            self._model, ids.ctypes.data_as(_I32P), counts.ctypes.data_as(_I32P), ids.size, flat.ctypes.data_as(_I64P),
            want.ctypes.data_as(_I32P), want.size, nxt.ctypes.data_as(_I64P)))
        return self.last_logits(want.size) if want.size else np.zeros((0, self.vocab), dtype=np.float32)

    def decode_loop(self, seq_ids: Sequence[int], first_tokens: Sequence[int], n_steps: int) -> np.ndarray:
        """n_steps greedy steps with the loop state kept on the device; returns int64 [n_steps, n_seqs]."""
        n = len(seq_ids)
        ids = np.ascontiguousarray(seq_ids, dtype=np.int32)
        first = np.ascontiguousarray(first_tokens, dtype=np.int64)
        if first.shape != (n,):
            raise ValueError("one first token per sequence")
        out = np.zeros((n_steps, n), dtype=np.int64)
        _check(LIB_LLAISYS.llaisysModelDecodeLoop(
            self._model, ids.ctypes.data_as(_I32P), n, first.ctypes.data_as(_I64P),
            n_steps, out.ctypes.data_as(_I64P)))
        return out

    def last_logits(self, n_seqs: int = 1) -> np.ndarray:
        """float32 [n_seqs, voc] logits of the most recent step (n_seqs = that step's sequence count)."""
        out = np.zeros((n_seqs, self.vocab), dtype=np.float32)
        _check(LIB_LLAISYS.llaisysModelLastLogits(self._model, out.ctypes.data_as(ctypes.POINTER(c_float)), out.size))
        return out

    @property
    def last_loop_ms(self) -> float:
        """Device milliseconds per decode step of the last decode_loop()."""
        return float(LIB_LLAISYS.llaisysModelLastLoopMs(self._model))


class NamedWeightsLM(CausalLM):
    """A family whose weights are loaded by their checkpoint names (llaisysModelLoadTensor) and whose residual stream is f32. It
    supplies meta_of() and the library's constructor."""
    create: str          # C function: (meta *, device, device id) -> handle

    def meta_of(self, config: Mapping, shapes: Mapping[str, tuple[int, ...]], dtype: DataType, max_seq_len: int | None):
        """The C description of a model: `shapes` holds the shapes of the checkpoint's tensors."""
        raise NotImplementedError

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
            raise ValueError(f"{type(self).__name__} needs a checkpoint directory or a config")
        if dtype is None:
            dtype = DTYPE_NAMES.get(str(config.get("torch_dtype", "bfloat16")), DataType.BF16)
        shapes = {name: f.shape(name) for f in files for name in f.names()}
        if state_dict is not None:
            shapes |= {name: tuple(value.shape) for name, value in state_dict.items()}
        self.config = dict(config)
        self.meta = self.meta_of(config, shapes, dtype, max_seq_len)
        self.vocab, self.max_seq, self.end_token = int(self.meta.voc), int(self.meta.maxseq), int(self.meta.end_token)
        self.dtype, self.device, self.device_id = dtype, device, device_id
        self._model = getattr(LIB_LLAISYS, self.create)(ctypes.byref(self.meta), int(device), device_id)
        if not self._model:
            raise RuntimeError(f"{self.create} failed: " + (LIB_LLAISYS.llaisysGetLastError() or b"").decode())
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
        ndim, shape = array.ndim, (c_size_t * array.ndim)(*array.shape)
        array = np.ascontiguousarray(array)  # (gives a single number a dimension)
        known = c_int(0)
        try:
            _check(LIB_LLAISYS.llaisysModelLoadTensor(self._model, name.encode(), int(kind), shape, ndim,
                                                      array.ctypes.data, ctypes.byref(known)))
        except LlaisysError as err:
            raise ValueError(str(err)) from err

    # ---- development aid ------------------------------------------------------------------------------------------------

    def record_stream(self, enable: bool = True) -> None:
        """Keep the residual stream after every layer run of the steps that follow (slow)."""
        _check(LIB_LLAISYS.llaisysModelRecordStream(self._model, int(enable)))

    def layer_runs(self) -> int:
        return len(self.config["layers"])

    def layer_stream(self) -> np.ndarray:
        """float32 [layer runs, rows, width] of the last step."""
        n = c_size_t(0)
        _check(LIB_LLAISYS.llaisysModelLayerStream(self._model, None, 0, ctypes.byref(n)))
        out = np.zeros(n.value, dtype=np.float32)
        _check(LIB_LLAISYS.llaisysModelLayerStream(self._model, out.ctypes.data_as(ctypes.POINTER(c_float)), out.size,
                                                   ctypes.byref(n)))
        return out.reshape(self.layer_runs(), -1, int(self.meta.width))


def tensor_rows(shapes: Mapping[str, tuple[int, ...]], names: Sequence[str]) -> list[int]:
    """First dimension of each named tensor: sizes that only a checkpoint's weights hold."""
    missing = [n for n in names if n not in shapes]
    if missing:
        raise ValueError(f"checkpoint lacks {len(missing)} tensors, e.g. {missing[:3]}")
    return [int(shapes[n][0]) for n in names]
