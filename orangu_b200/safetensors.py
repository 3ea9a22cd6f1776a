"""Reader of .safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets), data.
The file is mapped; tensors are views into the mapping until something needs another type."""
from __future__ import annotations

import json
import mmap
import struct

import numpy as np

DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "I32": np.int32, "I64": np.int64, "U8": np.uint8}  # BF16: the bits


class SafetensorsFile:
    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError(f"{path}: too short for a safetensors file")
        n = struct.unpack_from("<Q", self._map, 0)[0]
        if 8 + n > len(self._map):
            raise ValueError(f"{path}: the header runs past the end of the file")
        self.header = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}
        self.path, self._data = path, 8 + n

    def __contains__(self, name: str) -> bool:
        return name in self.header

    def names(self):
        return list(self.header)

    def dtype(self, name: str) -> str:
        return self.header[name]["dtype"]

    def raw(self, name: str, shape=None) -> np.ndarray:
        """The tensor as stored (bfloat16: uint16 bits); ValueError when it is missing or its shape is not the expected one."""
        if name not in self.header:
            raise ValueError(f"{self.path}: no tensor {name}")
        h = self.header[name]
        if h["dtype"] not in DTYPES:
            raise ValueError(f"{self.path}: {name} has unsupported type {h['dtype']}")
        dt = np.dtype(DTYPES[h["dtype"]])
        lo, hi = h["data_offsets"]
        count = int(np.prod(h["shape"], dtype=np.int64))
        if hi - lo != count * dt.itemsize or self._data + hi > len(self._map):
            raise ValueError(f"{self.path}: {name} does not fit its offsets")
        if shape is not None and tuple(h["shape"]) != tuple(shape):
            raise ValueError(f"{self.path}: {name} is {h['shape']}, expected {list(shape)}")
        return np.frombuffer(self._map, dt, count, self._data + lo).reshape(h["shape"])

    def bf16(self, name: str, shape=None) -> np.ndarray:
        """The tensor's bfloat16 bits; wider float types are rounded to nearest even."""
        a = self.raw(name, shape)
        if self.dtype(name) == "BF16":
            return a
        return to_bf16(a)

    def f32(self, name: str, shape=None) -> np.ndarray:
        a = self.raw(name, shape)
        return from_bf16(a) if self.dtype(name) == "BF16" else np.array(a, np.float32, order="C")


def from_bf16(bits: np.ndarray) -> np.ndarray:
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def to_bf16(x: np.ndarray) -> np.ndarray:
    u = np.array(x, np.float32, order="C").view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def save(path: str, tensors: dict) -> None:
    """Writes arrays; uint16 arrays are stored as bfloat16 bits."""
    back = {np.dtype(v): k for k, v in DTYPES.items()}
    header, at = {}, 0
    for k, a in tensors.items():
        header[k] = {"dtype": back[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())
