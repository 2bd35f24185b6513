"""Model folders: config.json and model.safetensors.

A safetensors file is an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets) and the tensor data; tensors are handed out as views of the mapped file.
"""
from __future__ import annotations

import json
import mmap
import os

import numpy as np

_NUMPY = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class SafeTensors:
    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._map)
        length = int.from_bytes(self._map[:8], "little") if size >= 8 else 0
        if length < 2 or 8 + length > size:
            raise ValueError(f"{path}: not a safetensors file")
        self.entries = json.loads(self._map[8:8 + length])
        self.entries.pop("__metadata__", None)
        self._base = 8 + length
        self.path = path
        for name, e in self.entries.items():
            begin, end = e["data_offsets"]
            if e["dtype"] not in _NUMPY:
                raise ValueError(f"{path}: tensor '{name}' has the unknown dtype {e['dtype']}")
            count = int(np.prod(e["shape"], dtype=np.int64))
            if not 0 <= begin <= end <= size - self._base or end - begin != count * np.dtype(_NUMPY[e["dtype"]]).itemsize:
                raise ValueError(f"{path}: tensor '{name}' does not fit its data")

    def __contains__(self, name: str) -> bool:
        return name in self.entries

    def shape(self, name: str):
        if name not in self.entries:
            raise KeyError(f"{self.path} has no tensor '{name}'")
        return tuple(self.entries[name]["shape"])

    def dtype(self, name: str) -> str:
        return self.entries[name]["dtype"]

    def raw(self, name: str) -> np.ndarray:
        """The tensor as stored (bf16 as uint16)."""
        shape = self.shape(name)
        e = self.entries[name]
        begin, end = e["data_offsets"]
        return np.frombuffer(self._map, dtype=_NUMPY[e["dtype"]], count=int(np.prod(shape, dtype=np.int64)), offset=self._base + begin).reshape(shape)

    def f32(self, name: str) -> np.ndarray:
        a = self.raw(name)
        if self.dtype(name) == "BF16":
            return (a.astype(np.uint32) << 16).view(np.float32)
        return a.astype(np.float32)


def write_safetensors(path: str, tensors) -> None:
    """tensors: name -> (dtype name, numpy array as stored)."""
    header, at = {}, 0
    for name, (dtype, a) in tensors.items():
        header[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    blob = json.dumps(header).encode()
    blob += b" " * (-len(blob) % 8)
    with open(path, "wb") as f:
        f.write(len(blob).to_bytes(8, "little") + blob)
        for _, a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())


def to_bf16(a: np.ndarray) -> np.ndarray:
    """f32 -> bf16 bit patterns, round to nearest even (finite values)."""
    b = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
