"""Reader of safetensors files: an 8-byte little-endian header length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data.  Tensors are views of the mapped file."""
from __future__ import annotations

import json
import struct

import numpy as np

# bf16 has no numpy type: its bit patterns come back as uint16
DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8,
          "I16": np.int16, "U16": np.uint16, "I32": np.int32, "U32": np.uint32, "I64": np.int64, "U64": np.uint64, "BOOL": np.bool_}


class SafeTensors:
    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError(f"{path}: not a safetensors file")
            n = struct.unpack("<Q", head)[0]
            text = f.read(n)
        if len(text) != n:
            raise ValueError(f"{path}: header of {n} bytes is cut off")
        self._index = {k: v for k, v in json.loads(text).items() if k != "__metadata__"}
        self._data = np.memmap(path, dtype=np.uint8, mode="r", offset=8 + n)

    def names(self) -> list[str]:
        return list(self._index)

    def __contains__(self, name: str) -> bool:
        return name in self._index

    def dtype(self, name: str) -> str:
        return self._index[name]["dtype"]

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self._index[name]["shape"])

    def __getitem__(self, name: str) -> np.ndarray:
        if name not in self._index:
            raise KeyError(f"{self.path} holds no tensor {name!r}")
        d = self._index[name]
        a, b = d["data_offsets"]
        return np.frombuffer(self._data[a:b].tobytes(), dtype=DTYPES[d["dtype"]]).reshape(d["shape"])

    def bf16_bits(self, name: str) -> np.ndarray:
        """The tensor as bf16 bit patterns; fp32 and fp16 tensors are rounded to nearest even."""
        a = self[name]
        if self.dtype(name) == "BF16":
            return a
        return to_bf16_bits(a)


def to_bf16_bits(a) -> np.ndarray:
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16_bits(bits) -> np.ndarray:
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)
