"""Checkpoints: a folder with ``config.json`` and ``model.safetensors``.

Layout of the latter: the header's size as a 64-bit little-endian integer, the header (a JSON object that
gives dtype, shape and byte range of every tensor, counted from the header's end), then the raw tensors.
"""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Dict, Iterable, Tuple

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "U8": torch.uint8, "I8": torch.int8}


class CheckpointError(ValueError):
    """The folder does not hold what the model needs."""


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


class SafetensorsFile:
    """Read-only view of one file; tensors are copied out one at a time, on the CPU."""

    def __init__(self, path: str):
        self._file = open(path, "rb")
        size = os.fstat(self._file.fileno()).st_size
        if size < 8:
            raise CheckpointError(f"{path}: too short for a safetensors file")
        self._map = mmap.mmap(self._file.fileno(), 0, access=mmap.ACCESS_READ)
        (n,) = struct.unpack("<Q", self._map[:8])
        if 8 + n > size:
            raise CheckpointError(f"{path}: header of {n} bytes in a file of {size}")
        header = json.loads(self._map[8:8 + n])
        self._base, self._size, self.path = 8 + n, size, path
        self._entries = {k: v for k, v in header.items() if k != "__metadata__"}

    def names(self) -> Iterable[str]:
        return self._entries.keys()

    def shape(self, name: str) -> Tuple[int, ...]:
        """The shape of the tensor `name`, for sizes that the configuration does not give."""
        e = self._entries.get(name)
        if e is None:
            raise CheckpointError(f"{self.path}: tensor {name!r} is missing")
        return tuple(e["shape"])

    def get(self, name: str, shape: Tuple[int, ...]) -> torch.Tensor:
        """The tensor `name`, which must have the given shape."""
        e = self._entries.get(name)
        if e is None:
            raise CheckpointError(f"{self.path}: tensor {name!r} is missing")
        if tuple(e["shape"]) != tuple(shape):
            raise CheckpointError(f"{self.path}: tensor {name!r} has shape {e['shape']}, the configuration says {list(shape)}")
        dtype = _DTYPES.get(e["dtype"])
        if dtype is None:
            raise CheckpointError(f"{self.path}: tensor {name!r} has unsupported dtype {e['dtype']}")
        lo, hi = e["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if hi - lo != count * torch.empty(0, dtype=dtype).element_size() or self._base + hi > self._size:
            raise CheckpointError(f"{self.path}: tensor {name!r} has inconsistent offsets")
        raw = bytearray(self._map[self._base + lo:self._base + hi])
        if count == 0:
            return torch.empty(shape, dtype=dtype)
        return torch.frombuffer(raw, dtype=dtype).reshape(shape)

    def close(self) -> None:
        self._map.close()
        self._file.close()


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        blob = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    head = json.dumps(header, separators=(",", ":")).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for blob in blobs:
            f.write(blob)
