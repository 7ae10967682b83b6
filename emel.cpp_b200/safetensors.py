"""safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets) and the
tensors' bytes.  Tensors are views of a read-only mapping; bf16 comes as uint16 bit patterns."""
from __future__ import annotations

import json
import mmap
import struct

import numpy as np

_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8, "I16": np.int16,
           "I32": np.int32, "I64": np.int64}


class File:
    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError(f"{path}: no safetensors header")
        (n,) = struct.unpack("<Q", self._map[:8])
        if 8 + n > len(self._map):
            raise ValueError(f"{path}: the header does not fit the file")
        self._base = 8 + n
        self.entries = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}

    def __contains__(self, name: str) -> bool:
        return name in self.entries

    def names(self):
        return list(self.entries)

    def dtype(self, name: str) -> str:
        return self.entries[name]["dtype"]

    def shape(self, name: str):
        return tuple(self.entries[name]["shape"])

    def array(self, name: str) -> np.ndarray:
        e = self.entries[name]
        begin, end = e["data_offsets"]
        dt = np.dtype(_DTYPES[e["dtype"]])
        count = int(np.prod(e["shape"], dtype=np.int64)) if e["shape"] else 1
        if end - begin != count * dt.itemsize or self._base + end > len(self._map):
            raise ValueError(f"tensor {name}: its bytes do not fit its shape")
        return np.frombuffer(self._map, dt, count, self._base + begin).reshape(e["shape"])

    def f32(self, name: str) -> np.ndarray:
        a = self.array(name)
        return bf16_to_f32(a) if self.dtype(name) == "BF16" else a.astype(np.float32)

    def bf16(self, name: str) -> np.ndarray:
        """Bit patterns; other float types are rounded to nearest even."""
        return self.array(name) if self.dtype(name) == "BF16" else f32_to_bf16(self.array(name).astype(np.float32))


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def write(path: str, tensors: dict) -> None:
    """name -> float32 (stored as bf16) or int32 array."""
    head, at, blobs = {}, 0, []
    for name, a in tensors.items():
        raw = a if a.dtype == np.int32 else f32_to_bf16(a)
        b = np.ascontiguousarray(raw).tobytes()
        head[name] = {"dtype": "I32" if a.dtype == np.int32 else "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
