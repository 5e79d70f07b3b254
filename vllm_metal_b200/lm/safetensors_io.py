"""Reader / writer of the safetensors container: an 8-byte little-endian header length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the raw tensors.  The file is memory-mapped; a tensor is copied once, when
it is asked for."""

from __future__ import annotations

import json
import mmap
import os
from collections.abc import Iterator

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


class SafetensorsFile:
    def __init__(self, path: str) -> None:
        self.path = str(path)
        with open(self.path, "rb") as f:
            size = os.fstat(f.fileno()).st_size
            head = f.read(8)
            n = int.from_bytes(head, "little") if len(head) == 8 else size
            if 8 + n > size:
                raise ValueError(f"{self.path}: not a safetensors file (header of {n} bytes in {size})")
            table = json.loads(f.read(n))
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ) if size else b""
        self._base = 8 + n
        self._meta = {k: v for k, v in table.items() if k != "__metadata__"}
        for name, t in self._meta.items():
            lo, hi = t["data_offsets"]
            if t["dtype"] not in _DTYPES or not 0 <= lo <= hi <= size - self._base:
                raise ValueError(f"{self.path}: tensor '{name}' is {t['dtype']} at {lo}..{hi}")

    def __contains__(self, name: str) -> bool:
        return name in self._meta

    def keys(self) -> Iterator[str]:
        return iter(self._meta)

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self._meta[name]["shape"])

    def tensor(self, name: str) -> torch.Tensor:
        t = self._meta[name]
        lo, hi = t["data_offsets"]
        dtype = _DTYPES[t["dtype"]]
        out = torch.empty(tuple(t["shape"]), dtype=dtype)
        if out.numel() * out.element_size() != hi - lo:
            raise ValueError(f"{self.path}: tensor '{name}' has {hi - lo} bytes for shape {t['shape']}")
        if hi > lo:
            raw = torch.frombuffer(bytearray(self._map[self._base + lo:self._base + hi]), dtype=torch.uint8)
            out = raw.view(dtype).reshape(tuple(t["shape"]))
        return out


class SafetensorsFolder:
    """Every ``*.safetensors`` file of a model folder as one name space."""

    def __init__(self, folder: str) -> None:
        files = sorted(f for f in os.listdir(folder) if f.endswith(".safetensors"))
        if not files:
            raise FileNotFoundError(f"{folder}: no .safetensors file")
        self._where: dict[str, SafetensorsFile] = {}
        for f in files:
            part = SafetensorsFile(os.path.join(folder, f))
            for k in part.keys():
                if k in self._where:
                    raise ValueError(f"{folder}: tensor '{k}' is in two files")
                self._where[k] = part

    def __contains__(self, name: str) -> bool:
        return name in self._where

    def keys(self) -> Iterator[str]:
        return iter(self._where)

    def shape(self, name: str) -> tuple[int, ...]:
        return self._where[name].shape(name)

    def tensor(self, name: str) -> torch.Tensor:
        if name not in self._where:
            raise KeyError(f"tensor '{name}' is not in the checkpoint")
        return self._where[name].tensor(name)


def save_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> None:
    table, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        table[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(table).encode()
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little"))
        f.write(head)
        for b in blobs:
            f.write(b)
