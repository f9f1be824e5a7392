"""Reading safetensors files without a tensor library: an 8-byte little-endian header length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data. Arrays are views of the mapped file; bfloat16 comes as its 16-bit
words."""
from __future__ import annotations

import json
import mmap
from pathlib import Path
from typing import Iterator

import numpy as np

from ..libllaisys import DataType

_NUMPY = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I64": np.int64, "I32": np.int32,
          "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}
LIBRARY_DTYPE = {"BF16": DataType.BF16, "F16": DataType.F16, "F32": DataType.F32}


class SafetensorsFile:
    def __init__(self, path):
        self.path = Path(path)
        with open(self.path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError(f"{self.path}: too short for a safetensors file")
        n = int.from_bytes(self._map[:8], "little")
        if n > len(self._map) - 8:
            raise ValueError(f"{self.path}: the header is longer than the file")
        self._entries = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}
        self._data = 8 + n

    def names(self) -> list[str]:
        return list(self._entries)

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self._entries[name]["shape"])

    def dtype(self, name: str) -> str:
        return self._entries[name]["dtype"]

    def array(self, name: str) -> np.ndarray:
        e = self._entries[name]
        lo, hi = e["data_offsets"]
        kind = np.dtype(_NUMPY[e["dtype"]])
        count = int(np.prod(e["shape"], dtype=np.int64))
        if hi - lo != count * kind.itemsize or self._data + hi > len(self._map):
            raise ValueError(f"{self.path}: {name} has {hi - lo} bytes for shape {e['shape']} of {e['dtype']}")
        return np.frombuffer(self._map, dtype=kind, count=count, offset=self._data + lo).reshape(e["shape"])


def checkpoint_files(model_path) -> Iterator[SafetensorsFile]:
    files = sorted(Path(model_path).glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"no *.safetensors in {model_path}")
    for f in files:
        yield SafetensorsFile(f)
