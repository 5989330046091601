"""Reader and writer of .safetensors files (8-byte little-endian header length, JSON header name -> dtype, shape, data_offsets,
then the data). The file is memory-mapped; a tensor is copied out when it is asked for."""
from __future__ import annotations

import json
import mmap
import os

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64, "I32": torch.int32,
           "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


class SafeTensors:
    """Mapping name -> CPU tensor over one file."""

    def __init__(self, path: str):
        self.path = path
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            n = int.from_bytes(f.read(8), "little")
            if size < 8 or n > size - 8:
                raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
            header = json.loads(f.read(n))
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        self._base = 8 + n
        self._entries = {k: v for k, v in header.items() if k != "__metadata__"}
        for k, v in self._entries.items():
            lo, hi = v["data_offsets"]
            if v["dtype"] not in _DTYPES:
                raise ValueError(f"{path}: tensor {k}: dtype {v['dtype']} is not supported")
            want = torch.Size(v["shape"]).numel() * _DTYPES[v["dtype"]].itemsize
            if not (0 <= lo <= hi <= size - self._base) or hi - lo != want:
                raise ValueError(f"{path}: tensor {k}: offsets {lo}..{hi} do not hold shape {v['shape']}")

    def __contains__(self, name: str) -> bool:
        return name in self._entries

    def keys(self):
        return self._entries.keys()

    def shape(self, name: str):
        return tuple(self._entries[name]["shape"])

    def __getitem__(self, name: str) -> torch.Tensor:
        if name not in self._entries:
            raise KeyError(f"{self.path} has no tensor {name!r}")
        e = self._entries[name]
        lo, hi = e["data_offsets"]
        if hi == lo:
            return torch.empty(e["shape"], dtype=_DTYPES[e["dtype"]])
        buf = bytearray(self._map[self._base + lo:self._base + hi])
        return torch.frombuffer(buf, dtype=_DTYPES[e["dtype"]]).reshape(e["shape"])


def save(path: str, tensors: dict):
    header, chunks, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        chunks.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little"))
        f.write(head)
        for c in chunks:
            f.write(c)
