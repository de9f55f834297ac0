"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets), then the tensors' bytes.  The file is mapped, not read: a tensor's bytes are touched when it is copied."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path
from typing import Dict, List

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
           "I8": torch.int8, "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "U8": torch.uint8,
           "BOOL": torch.bool}


class Checkpoint:
    """Tensors of a safetensors file by name.  Names that were asked for are remembered, so that a loader can tell
    what it left unread."""

    def __init__(self, path):
        self.path = Path(path)
        with open(self.path, "rb") as f:
            raw = f.read(8)
            if len(raw) != 8:
                raise ValueError(f"{self.path}: not a safetensors file")
            n = struct.unpack("<Q", raw)[0]
            size = self.path.stat().st_size
            if n > size - 8:
                raise ValueError(f"{self.path}: header of {n} bytes in a file of {size}")
            self.header = json.loads(f.read(n))
            self._base = 8 + n
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
        self.header.pop("__metadata__", None)
        self.read = set()
        for name, t in self.header.items():
            lo, hi = t["data_offsets"]
            count = 1
            for d in t["shape"]:
                count *= d
            if t["dtype"] not in _DTYPES:
                raise ValueError(f"{self.path}: {name} has dtype {t['dtype']}")
            if lo < 0 or self._base + hi > size or hi - lo != count * _DTYPES[t["dtype"]].itemsize:
                raise ValueError(f"{self.path}: {name} has offsets {lo}..{hi} for shape {t['shape']}")

    def __contains__(self, name: str) -> bool:
        return name in self.header

    def names(self) -> List[str]:
        return list(self.header)

    def __getitem__(self, name: str) -> torch.Tensor:
        """A CPU tensor over the mapped bytes (copy-on-write: the file stays as it is)."""
        if name not in self.header:
            raise KeyError(f"{self.path} has no tensor {name!r}")
        t = self.header[name]
        self.read.add(name)
        dtype = _DTYPES[t["dtype"]]
        lo, hi = t["data_offsets"]
        if hi == lo:
            return torch.empty(t["shape"], dtype=dtype)
        if (self._base + lo) % dtype.itemsize:             # torch wants elements on their own boundary
            raw = torch.frombuffer(bytearray(self._map[self._base + lo:self._base + hi]), dtype=dtype)
        else:
            raw = torch.frombuffer(self._map, dtype=dtype, count=(hi - lo) // dtype.itemsize, offset=self._base + lo)
        return raw.view(t["shape"])

    def unread(self) -> List[str]:
        return sorted(set(self.header) - self.read)


def save(path, tensors: Dict[str, torch.Tensor]) -> None:
    """Write tensors as a safetensors file (random models for tests and benchmarks)."""
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for raw in blobs:
            f.write(raw)
