"""The safetensors container: 8-byte little-endian header length, JSON header (name -> dtype, shape, data_offsets), raw
little-endian data.  Written and parsed here, no third-party package.
"""
from __future__ import annotations

import json
import os
import struct
from typing import Dict, List, Tuple

import numpy as np

_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "U8": np.uint8, "I32": np.int32, "U32": np.uint32, "I64": np.int64}


def write_safetensors(path: str, tensors: Dict[str, Tuple[str, np.ndarray]], metadata: Dict[str, str]) -> None:
    """tensors: name -> (safetensors dtype tag, array whose bytes are stored as they are)."""
    header: Dict[str, object] = {"__metadata__": {k: str(v) for k, v in metadata.items()}}
    blobs: List[bytes] = []
    off = 0
    for name in sorted(tensors):
        tag, arr = tensors[name]
        raw = np.ascontiguousarray(arr).tobytes()
        header[name] = {"dtype": tag, "shape": list(arr.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(header, separators=(",", ":")).encode()
    hj += b" " * ((8 - len(hj) % 8) % 8)
    tmp = path + ".tmp"
    with open(tmp, "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
    os.replace(tmp, path)  # a reader never sees a half-written block


def read_safetensors(path: str) -> Tuple[Dict[str, np.ndarray], Dict[str, str]]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    meta = header.pop("__metadata__", {})
    out = {}
    for name, info in header.items():
        a, b = info["data_offsets"]
        out[name] = np.frombuffer(data[a:b], dtype=_DTYPES[info["dtype"]]).reshape(info["shape"])
    return out, meta


class SafetensorsFile:
    """Tensors of one file by name, read one at a time (a memory map; bf16 comes as its bits in uint16)."""

    def __init__(self, path: str):
        with open(path, "rb") as f:
            (n,) = struct.unpack("<Q", f.read(8))
            header = json.loads(f.read(n))
        header.pop("__metadata__", None)
        self._info, self._start = header, 8 + n
        self._data = np.memmap(path, np.uint8, "r")

    def names(self) -> List[str]:
        return list(self._info)

    def __contains__(self, name: str) -> bool:
        return name in self._info

    def dtype(self, name: str) -> str:
        return self._info[name]["dtype"]

    def shape(self, name: str) -> Tuple[int, ...]:
        return tuple(self._info[name]["shape"])

    def __getitem__(self, name: str) -> np.ndarray:
        info = self._info[name]
        a, b = info["data_offsets"]
        raw = self._data[self._start + a:self._start + b]
        return np.frombuffer(raw.tobytes(), _DTYPES[info["dtype"]]).reshape(info["shape"])

    def bf16(self, name: str) -> np.ndarray:
        """The tensor as bf16 bits (f32 and f16 tensors are rounded to nearest even)."""
        t = self[name]
        if self.dtype(name) == "BF16":
            return t
        if self.dtype(name) not in ("F32", "F16"):
            raise ValueError(f"{name}: {self.dtype(name)} is not a floating-point tensor")
        u = np.ascontiguousarray(t, np.float32).view(np.uint32)
        return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)
