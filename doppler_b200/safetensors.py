"""safetensors reader (and a writer for tests and exports): an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data.  bfloat16 tensors come back as their bits (uint16)."""
from __future__ import annotations

import json
import mmap
import os
from typing import Dict

import numpy as np

_NUMPY = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8, "I16": np.int16, "U16": np.uint16,
          "I32": np.int32, "U32": np.uint32, "I64": np.int64, "U64": np.uint64, "BOOL": np.bool_}


class SafetensorsError(Exception):
    pass


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        self._file = open(path, "rb")
        size = os.fstat(self._file.fileno()).st_size
        if size < 8:
            raise SafetensorsError(f"{path}: too short for a header")
        self._map = mmap.mmap(self._file.fileno(), 0, access=mmap.ACCESS_READ)
        n = int.from_bytes(self._map[:8], "little")
        if n > size - 8:
            raise SafetensorsError(f"{path}: header of {n} bytes in a file of {size}")
        header = json.loads(self._map[8:8 + n].decode("utf-8"))
        header.pop("__metadata__", None)
        self._base, self._size, self.header = 8 + n, size, header

    def names(self):
        return list(self.header)

    def __contains__(self, name: str) -> bool:
        return name in self.header

    def dtype(self, name: str) -> str:
        return self.header[name]["dtype"]

    def shape(self, name: str):
        """A tensor's shape, None if there is none of that name."""
        return tuple(self.header[name]["shape"]) if name in self.header else None

    def tensor(self, name: str) -> np.ndarray:
        if name not in self.header:
            raise SafetensorsError(f"{self.path}: no tensor '{name}'")
        e = self.header[name]
        if e["dtype"] not in _NUMPY:
            raise SafetensorsError(f"{self.path}: {name}: unknown dtype {e['dtype']}")
        dt = np.dtype(_NUMPY[e["dtype"]])
        lo, hi = e["data_offsets"]
        count = int(np.prod(e["shape"], dtype=np.int64))
        if lo < 0 or hi < lo or self._base + hi > self._size or hi - lo != count * dt.itemsize:
            raise SafetensorsError(f"{self.path}: {name}: bytes [{lo},{hi}) do not hold {e['dtype']}{e['shape']}")
        return np.frombuffer(self._map, dt, count, self._base + lo).reshape(e["shape"])

    def close(self):
        try:
            self._map.close()
        except BufferError:  # a tensor still looks into the map: it goes with the last of them
            pass
        self._file.close()


def bf16_bits(a: np.ndarray) -> np.ndarray:
    """Round finite f32 values to bfloat16 (nearest even), as bits."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_values(bits: np.ndarray) -> np.ndarray:
    return (np.ascontiguousarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def write_bf16(path: str, tensors: Dict[str, np.ndarray]):
    """Write tensors of bfloat16 bits (uint16)."""
    header, off = {}, 0
    for name, a in tensors.items():
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + 2 * a.size]}
        off += 2 * a.size
    raw = json.dumps(header).encode()
    raw += b" " * (-len(raw) % 8)
    with open(path, "wb") as f:
        f.write(len(raw).to_bytes(8, "little"))
        f.write(raw)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a, np.uint16).tobytes())
