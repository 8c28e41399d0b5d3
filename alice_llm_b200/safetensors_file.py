"""The safetensors container: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets),
then the data. Read as views of a memory map; bfloat16 tensors come as uint16 bit patterns."""
from __future__ import annotations

import json
import mmap
import os
import struct

import numpy as np

DTYPES = {"BF16": np.uint16, "F32": np.float32, "I32": np.int32}
MAX_HEADER = 100 << 20


class SafetensorsError(ValueError):
    pass


def bf16_to_f32(bits) -> np.ndarray:
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x) -> np.ndarray:
    """Round to nearest, ties to even (finite values)."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class SafetensorsFile:
    def __init__(self, path):
        with open(path, "rb") as f:
            size = os.fstat(f.fileno()).st_size
            if size < 8:
                raise SafetensorsError(f"{path}: {size} bytes are no safetensors file")
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        n = struct.unpack("<Q", self._map[:8])[0]
        if n > min(MAX_HEADER, size - 8):
            raise SafetensorsError(f"{path}: header of {n} bytes in a file of {size}")
        try:
            head = json.loads(self._map[8:8 + n].decode("utf-8"))
        except ValueError as e:
            raise SafetensorsError(f"{path}: header is not JSON ({e})") from None
        self.tensors = {}
        for name, info in head.items():
            if name == "__metadata__":
                continue
            if info["dtype"] not in DTYPES:
                raise SafetensorsError(f"{path}: {name} has dtype {info['dtype']}, known are {', '.join(DTYPES)}")
            dt, shape = np.dtype(DTYPES[info["dtype"]]), tuple(int(v) for v in info["shape"])
            lo, hi = info["data_offsets"]
            count = int(np.prod(shape, dtype=np.int64))
            if not 0 <= lo <= hi <= size - 8 - n or hi - lo != count * dt.itemsize:
                raise SafetensorsError(f"{path}: {name} {shape} does not fit its offsets {lo} .. {hi}")
            self.tensors[name] = np.frombuffer(self._map, dt, count, 8 + n + lo).reshape(shape)

    def names(self):
        return self.tensors.keys()

    def get(self, name) -> np.ndarray:
        if name not in self.tensors:
            raise SafetensorsError(f"tensor {name} missing")
        return self.tensors[name]


def write_safetensors(path, tensors: dict) -> None:
    """tensors: name -> array (uint16 = bfloat16 bits, float32 or int32)."""
    names = {np.dtype(v): k for k, v in DTYPES.items()}
    head, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.ascontiguousarray(a)
        head[name] = {"dtype": names[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        blobs.append(a.tobytes())
        at += a.nbytes
    raw = json.dumps(head).encode()
    raw += b" " * (-len(raw) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(raw)) + raw)
        for b in blobs:
            f.write(b)
