"""Reader and writer of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets), then the tensors' bytes.  Tensors come back as torch CPU tensors over a memory map of the file."""
from __future__ import annotations

import json
import mmap
import struct

_DTYPES = {"BF16": "bfloat16", "F16": "float16", "F32": "float32", "I32": "int32", "U8": "uint8"}


class SafetensorsFile:
    """Mapping name -> torch tensor, read on access."""

    def __init__(self, path):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        (n,) = struct.unpack("<Q", self._map[:8])
        if n > len(self._map) - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {len(self._map)}")
        head = json.loads(self._map[8:8 + n])
        head.pop("__metadata__", None)
        self._head, self._base, self.path = head, 8 + n, path
        for name, t in head.items():
            lo, hi = t["data_offsets"]
            if t["dtype"] not in _DTYPES or lo < 0 or hi < lo or self._base + hi > len(self._map):
                raise ValueError(f"{path}: tensor {name} is {t['dtype']} at {lo}..{hi}")

    def __contains__(self, name):
        return name in self._head

    def keys(self):
        return self._head.keys()

    def __getitem__(self, name):
        import torch
        t = self._head[name]
        lo, hi = t["data_offsets"]
        # a writable copy: torch wants no read-only buffers, and offsets need not be aligned to the element size
        return torch.frombuffer(bytearray(self._map[self._base + lo:self._base + hi]), dtype=getattr(torch, _DTYPES[t["dtype"]])).reshape(t["shape"])


def save_file(tensors, path):
    import torch
    names = {getattr(torch, v): k for k, v in _DTYPES.items()}
    head, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    h = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)
