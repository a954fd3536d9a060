"""Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets relative to the end of the JSON), then the data."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import numpy as np

# bfloat16 comes out as its 16-bit patterns
DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class SafetensorsFile:
    def __init__(self, path):
        self._f = open(path, "rb")
        try:
            size = Path(path).stat().st_size
            head = self._f.read(8)
            n = struct.unpack("<Q", head)[0] if len(head) == 8 else size
            if n > size - 8:
                raise ValueError(f"{path}: not a safetensors file")
            self.tensors = json.loads(self._f.read(n))
            self.metadata = self.tensors.pop("__metadata__", {})
            self._base = 8 + n
            for name, t in self.tensors.items():
                lo, hi = t["data_offsets"]
                if t["dtype"] in DTYPES:
                    need = int(np.prod(t["shape"], dtype=np.int64)) * np.dtype(DTYPES[t["dtype"]]).itemsize
                    if need != hi - lo:
                        raise ValueError(f"{path}: tensor {name} of shape {t['shape']} needs {need} bytes, the file gives {hi - lo}")
                if lo < 0 or hi < lo or self._base + hi > size:
                    raise ValueError(f"{path}: tensor {name} lies outside the file")
            self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        except Exception:
            self._f.close()
            raise

    def names(self):
        return list(self.tensors)

    def dtype(self, name: str) -> str:
        return self.tensors[name]["dtype"]

    def shape(self, name: str) -> tuple:
        return tuple(self.tensors[name]["shape"])

    def data(self, name: str) -> np.ndarray:
        """The tensor's values, not copied (valid until close)."""
        t = self.tensors[name]
        dt = np.dtype(DTYPES[t["dtype"]])
        lo, hi = t["data_offsets"]
        return np.frombuffer(self._map, dt, (hi - lo) // dt.itemsize, self._base + lo).reshape(t["shape"])

    def close(self):
        self._f.close()  # the map goes when the last array does


def write_safetensors(path, tensors: dict) -> None:
    """tensors: name -> array; uint16 arrays are written as bfloat16 patterns."""
    names = {np.dtype(v): k for k, v in DTYPES.items()}
    head, at = {}, 0
    arrays = {k: np.ascontiguousarray(v) for k, v in tensors.items()}
    for k, a in arrays.items():
        head[k] = {"dtype": names[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    j = json.dumps(head).encode()
    j += b" " * (-len(j) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(j)) + j)
        for a in arrays.values():
            f.write(a.tobytes())


def to_bf16(x) -> np.ndarray:
    """f32 values to bfloat16 patterns, round to nearest even."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(u) -> np.ndarray:
    return (np.ascontiguousarray(u, np.uint16).astype(np.uint32) << 16).view(np.float32)
