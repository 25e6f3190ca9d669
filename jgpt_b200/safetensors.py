"""Reader and writer of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets into the rest), the data.  numpy has no bfloat16: such tensors are handed out as float32 (exact)."""
from __future__ import annotations

import json
import mmap

import numpy as np

_PLAIN = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "I64": np.int64, "I32": np.int32, "I16": np.int16,
          "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    """Bits of the nearest bfloat16, ties to even (finite inputs)."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class SafetensorsFile:
    """Tensors are read from the mapped file when asked for."""

    def __init__(self, path):
        self._f = open(path, "rb")
        self._m = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        n = int.from_bytes(self._m[:8], "little")
        if n <= 0 or 8 + n > len(self._m):
            raise ValueError(f"{path}: not a safetensors file")
        self._head = json.loads(self._m[8:8 + n])
        self._head.pop("__metadata__", None)
        self._base = 8 + n

    def names(self):
        return list(self._head)

    def __contains__(self, name):
        return name in self._head

    def shape(self, name):
        return tuple(self._head[name]["shape"])

    def get(self, name) -> np.ndarray:
        if name not in self._head:
            raise KeyError(f"tensor {name} is not in the file")
        t = self._head[name]
        lo, hi = t["data_offsets"]
        dt, shape = t["dtype"], tuple(t["shape"])
        kind = np.uint16 if dt == "BF16" else _PLAIN.get(dt)
        if kind is None:
            raise ValueError(f"tensor {name}: dtype {dt} is not supported")
        a = np.frombuffer(self._m, kind, count=(hi - lo) // np.dtype(kind).itemsize, offset=self._base + lo)
        if a.size != int(np.prod(shape, dtype=np.int64)):
            raise ValueError(f"tensor {name}: {a.size} elements for shape {shape}")
        return (bf16_to_f32(a) if dt == "BF16" else a).reshape(shape)

    def close(self):
        self._head = {}
        try:
            self._m.close()
        except BufferError:  # a tensor handed out still looks at the mapping; it goes with the last of them
            pass
        self._f.close()


def write_bf16(path, tensors: dict):
    """Writes float arrays as bfloat16 tensors."""
    head, blobs, at = {}, [], 0
    for name, x in tensors.items():
        b = f32_to_bf16(np.asarray(x, np.float32)).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(x)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h)
        for b in blobs:
            f.write(b)
