"""Reading and writing of ``model.safetensors`` files.

The format: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, byte range) and the raw tensor
data.  The reader maps the file and hands out tensors one at a time, so a model is filled without a second copy of
all its weights in host memory."""
from __future__ import annotations

import json
import mmap
import os
import struct

import torch

_TO_TORCH = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
             "I64": torch.int64, "U8": torch.uint8, "I8": torch.int8, "BOOL": torch.bool}
_FROM_TORCH = {v: k for k, v in _TO_TORCH.items()}


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            if size < 8:
                raise ValueError(f"{path}: not a safetensors file")
            (n,) = struct.unpack("<Q", f.read(8))
            if 8 + n > size:
                raise ValueError(f"{path}: header reaches past the end of the file")
            header = json.loads(f.read(n))
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        header.pop("__metadata__", None)
        self.header, self._base = header, 8 + n
        for name, h in header.items():
            a, b = h["data_offsets"]
            if not 0 <= a <= b <= size - self._base:
                raise ValueError(f"{path}: {name} lies outside the file")

    def keys(self):
        return self.header.keys()

    def shape(self, name: str) -> tuple:
        return tuple(self.header[name]["shape"])

    def tensor(self, name: str) -> torch.Tensor:
        h = self.header[name]
        a, b = h["data_offsets"]
        dtype = _TO_TORCH[h["dtype"]]
        if a == b:
            return torch.empty(h["shape"], dtype=dtype)
        raw = bytearray(self._map[self._base + a:self._base + b])   # a private, writable copy of this tensor only
        return torch.frombuffer(raw, dtype=dtype).reshape(h["shape"])


def save_safetensors(path: str, tensors: dict) -> None:
    header, offset = {}, 0
    host = {k: v.detach().cpu().contiguous() for k, v in tensors.items()}
    for name, t in host.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": _FROM_TORCH[t.dtype], "shape": list(t.shape), "data_offsets": [offset, offset + n]}
        offset += n
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for t in host.values():
            f.write(t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b"")
