"""Reader of safetensors files: an 8-byte little-endian header length, a JSON table of names, then the data."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

from . import cabi

_NUMPY = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "F64": np.float64, "I32": np.int32, "I64": np.int64}


class Checkpoint:
    """Tensors of one file, memory-mapped.  bf16 values come as their 16-bit patterns with `raw`, widened with `f32`."""

    def __init__(self, path: str):
        if os.path.isdir(path):
            path = os.path.join(path, "model.safetensors")
        self.path = path
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError("%s: not a safetensors file" % path)
            n = struct.unpack("<Q", head)[0]
            if n > os.path.getsize(path) - 8:
                raise ValueError("%s: the header says %d bytes, the file is shorter" % (path, n))
            table = json.loads(f.read(n))
        table.pop("__metadata__", None)
        self.table = table
        self._data = np.memmap(path, np.uint8, "r", offset=8 + n) if os.path.getsize(path) > 8 + n else np.zeros(0, np.uint8)

    def __contains__(self, name: str) -> bool:
        return name in self.table

    def shape(self, name: str) -> tuple:
        return tuple(self._entry(name)["shape"])

    def _entry(self, name: str):
        if name not in self.table:
            raise KeyError("%s has no tensor '%s'" % (self.path, name))
        return self.table[name]

    def raw(self, name: str, shape=None):
        """(array, dtype code for cabi.Matrix.put); float types other than bf16 and float32 are widened."""
        e = self._entry(name)
        if e["dtype"] not in _NUMPY:
            raise ValueError("tensor '%s' has unsupported type %s" % (name, e["dtype"]))
        lo, hi = e["data_offsets"]
        a = np.frombuffer(self._data[lo:hi].tobytes(), _NUMPY[e["dtype"]]).reshape(e["shape"])
        if shape is not None and tuple(a.shape) != tuple(shape):
            raise ValueError("tensor '%s' is %s, expected %s" % (name, list(a.shape), list(shape)))
        if e["dtype"] == "BF16":
            return a, cabi.DTYPE_BF16
        return a.astype(np.float32, copy=False), cabi.DTYPE_F32

    def f32(self, name: str, shape=None) -> np.ndarray:
        a, code = self.raw(name, shape)
        return (a.astype(np.uint32) << 16).view(np.float32).reshape(a.shape) if code == cabi.DTYPE_BF16 else a

    def scalar(self, name: str) -> float:
        return float(self.f32(name).reshape(-1)[0])
