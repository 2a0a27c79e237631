"""Reader and writer of safetensors files: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the tensors' bytes."""
from __future__ import annotations

import json
import mmap
import struct

_DTYPES = {"F64": "float64", "F32": "float32", "F16": "float16", "BF16": "bfloat16", "I64": "int64", "I32": "int32",
           "I16": "int16", "I8": "int8", "U8": "uint8", "BOOL": "bool"}


class SafeTensors:
    """Shapes without reading data, tensors (copies on the CPU) by name."""

    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError(f"{path}: not a safetensors file")
        n, = struct.unpack("<Q", self._map[:8])
        if n > len(self._map) - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {len(self._map)}")
        self._base = 8 + n
        self._entries = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}
        self.shapes = {k: tuple(v["shape"]) for k, v in self._entries.items()}

    def __contains__(self, name):
        return name in self._entries

    def __iter__(self):
        return iter(self._entries)

    def __getitem__(self, name):
        import torch
        e = self._entries[name]
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{name}: dtype {e['dtype']} is not supported")
        a, b = e["data_offsets"]
        dtype = getattr(torch, _DTYPES[e["dtype"]])
        if a == b:
            return torch.empty(*e["shape"], dtype=dtype)
        raw = bytearray(self._map[self._base + a:self._base + b])
        return torch.frombuffer(raw, dtype=dtype).view(*e["shape"])


def save_safetensors(path: str, tensors) -> None:
    """Writes a dict of CPU tensors."""
    import torch
    names = {str(getattr(torch, v)): k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = dict(dtype=names[str(t.dtype)], shape=list(t.shape), data_offsets=[at, at + len(raw)])
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for b in blobs:
            f.write(b)
