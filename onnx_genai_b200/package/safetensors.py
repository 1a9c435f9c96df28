"""Reader of safetensors files: eight bytes of header length, a JSON table (name -> dtype, shape, offsets), then the data.
The file is mapped; a tensor is copied when it is taken."""
from __future__ import annotations

import json
import mmap
import struct
from collections.abc import Mapping

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64, "I32": torch.int32,
           "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class SafetensorsFile(Mapping):
    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        (n,) = struct.unpack("<Q", self._map[:8])
        if n > len(self._map) - 8:
            raise ValueError(f"{path}: the header claims {n} bytes, more than the file holds")
        table = json.loads(self._map[8:8 + n])
        table.pop("__metadata__", None)
        self._base, self._table = 8 + n, table

    def __getitem__(self, name: str) -> torch.Tensor:
        e = self._table[name]
        dt = _DTYPES.get(e["dtype"])
        if dt is None:
            raise ValueError(f"{self.path}: tensor {name!r} has unsupported type {e['dtype']}")
        lo, hi = e["data_offsets"]
        count = 1
        for d in e["shape"]:
            count *= d
        size = torch.empty(0, dtype=dt).element_size()
        if hi - lo != count * size or self._base + hi > len(self._map):
            raise ValueError(f"{self.path}: tensor {name!r} does not fit its data range")
        if count == 0:
            return torch.empty(e["shape"], dtype=dt)
        raw = bytearray(self._map[self._base + lo:self._base + hi])
        return torch.frombuffer(raw, dtype=dt).reshape(e["shape"])

    def __iter__(self):
        return iter(self._table)

    def __len__(self):
        return len(self._table)


def save_file(tensors: dict, path: str) -> None:
    """Write name -> tensor (tests and exports)."""
    names = {v: k for k, v in _DTYPES.items()}
    table, blobs, off = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        table[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
