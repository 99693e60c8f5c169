"""safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets), the data."""
from __future__ import annotations

import json
import mmap
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "I32": torch.int32, "I64": torch.int64}
_NAMES = {v: k for k, v in _DTYPES.items()}


class SafetensorsFile:
    """Mapped file; `get(name)` is a CPU tensor over the mapping (read-only use)."""

    def __init__(self, path: str):
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError(f"{path}: too short for a safetensors file")
            (n,) = struct.unpack("<Q", head)
            size = os.fstat(f.fileno()).st_size
            if n > size - 8:
                raise ValueError(f"{path}: header length {n} past the end of the file")
            self.header = json.loads(f.read(n))
            self.header.pop("__metadata__", None)
            self._base, self._path = 8 + n, path
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
        for name, e in self.header.items():
            lo, hi = e["data_offsets"]
            if e["dtype"] not in _DTYPES:
                raise ValueError(f"{path}: {name} has element type {e['dtype']}")
            count = 1
            for d in e["shape"]:
                count *= d
            if lo < 0 or hi - lo != count * _DTYPES[e["dtype"]].itemsize or self._base + hi > size:
                raise ValueError(f"{path}: {name} does not fit its data range")

    def names(self):
        return list(self.header)

    def __contains__(self, name: str) -> bool:
        return name in self.header

    def get(self, name: str) -> torch.Tensor:
        if name not in self.header:
            raise KeyError(f"{self._path}: no tensor {name}")
        e = self.header[name]
        lo, hi = e["data_offsets"]
        if hi == lo:
            return torch.empty(e["shape"], dtype=_DTYPES[e["dtype"]])
        raw = torch.frombuffer(self._map, dtype=torch.uint8, count=hi - lo, offset=self._base + lo)
        return (raw if raw.data_ptr() % 8 == 0 else raw.clone()).view(_DTYPES[e["dtype"]]).reshape(e["shape"])


def write_safetensors(path: str, tensors: dict) -> None:
    header, off = {}, 0
    for name, t in tensors.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + n]}
        off += n
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for t in tensors.values():
            f.write(t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes())
