"""Reader of safetensors files: an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape,
data_offsets relative to the end of the header), then the data.  Tensors are views of the mapped file; bfloat16 has no numpy
type and is handed out as its uint16 bit patterns."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import numpy as np

_DTYPES = {"BF16": np.uint16, "F32": np.float32, "F16": np.float16, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class SafetensorsError(RuntimeError):
    pass


class SafetensorsFile:
    def __init__(self, path):
        self.path = Path(path)
        self._f = open(self.path, "rb")
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._map)
        n = struct.unpack("<Q", self._map[:8])[0] if size >= 8 else size
        if 8 + n > size:
            raise SafetensorsError("%s: the header is longer than the file" % self.path)
        self._base = 8 + n
        head = json.loads(self._map[8:8 + n])
        head.pop("__metadata__", None)
        self.info = head
        for name, t in head.items():
            a, b = t["data_offsets"]
            if t["dtype"] not in _DTYPES:
                raise SafetensorsError("%s: tensor %s has an unknown dtype %s" % (self.path, name, t["dtype"]))
            want = int(np.prod(t["shape"], dtype=np.int64)) * np.dtype(_DTYPES[t["dtype"]]).itemsize
            if b - a != want or self._base + b > size or a < 0:
                raise SafetensorsError("%s: tensor %s does not fit its shape or the file" % (self.path, name))

    def __contains__(self, name: str) -> bool:
        return name in self.info

    def dtype(self, name: str) -> str:
        return self._entry(name)["dtype"]

    def shape(self, name: str):
        return tuple(self._entry(name)["shape"])

    def _entry(self, name: str):
        try:
            return self.info[name]
        except KeyError:
            raise SafetensorsError("%s: no tensor %s" % (self.path, name)) from None

    def tensor(self, name: str) -> np.ndarray:
        """The tensor as stored (bfloat16: uint16 bit patterns)."""
        t = self._entry(name)
        a, b = t["data_offsets"]
        return np.frombuffer(self._map, _DTYPES[t["dtype"]], count=(b - a) // np.dtype(_DTYPES[t["dtype"]]).itemsize,
                             offset=self._base + a).reshape(t["shape"])

    def f32(self, name: str) -> np.ndarray:
        """The tensor as float32 values."""
        x = self.tensor(name)
        return bf16_to_f32(x) if self.dtype(name) == "BF16" else x.astype(np.float32)

    def bf16(self, name: str) -> np.ndarray:
        """The tensor as bfloat16 bit patterns (rounded to nearest even from other float types)."""
        x = self.tensor(name)
        return x if self.dtype(name) == "BF16" else f32_to_bf16(x.astype(np.float32))


def bf16_to_f32(u: np.ndarray) -> np.ndarray:
    return (np.asarray(u, np.uint16).astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    b = np.array(x, np.float32, order="C", ndmin=1).view(np.uint32)
    return ((b + np.uint32(0x7FFF) + ((b >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint16).reshape(np.shape(x))
