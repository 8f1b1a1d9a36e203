"""Safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets), the data.

The file is memory-mapped; a tensor is a view of the mapping until it is copied to the device.
"""
from __future__ import annotations

import json
import os

import numpy as np

_TORCH = {"BF16": "bfloat16", "F32": "float32", "F16": "float16", "I32": "int32", "I64": "int64"}
_BYTES = {"BF16": 2, "F16": 2, "F32": 4, "I32": 4, "I64": 8}


class SafetensorsFile:
    def __init__(self, path: str):
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            n = int.from_bytes(f.read(8), "little")
            if n <= 0 or 8 + n > size:
                raise ValueError(f"{path}: not a safetensors file")
            header = json.loads(f.read(n))
        self.path = path
        self.tensors = {k: v for k, v in header.items() if k != "__metadata__"}
        self._data = np.memmap(path, np.uint8, "r", 8 + n) if size > 8 + n else np.empty(0, np.uint8)
        for name, t in self.tensors.items():
            lo, hi = t["data_offsets"]
            want = int(np.prod(t["shape"], dtype=np.int64)) * _BYTES.get(t["dtype"], 0)
            if t["dtype"] not in _BYTES or hi - lo != want or lo < 0 or hi > self._data.size:
                raise ValueError(f"{path}: tensor '{name}' ({t['dtype']} {t['shape']}) does not fit its {hi - lo} bytes")

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def __getitem__(self, name: str):
        """The tensor as a torch CPU tensor (a copy of its bytes)."""
        import torch

        if name not in self.tensors:
            raise KeyError(f"{self.path} has no tensor '{name}'")
        t = self.tensors[name]
        lo, hi = t["data_offsets"]
        raw = torch.from_numpy(np.array(self._data[lo:hi]))
        return raw.view(getattr(torch, _TORCH[t["dtype"]])).reshape(t["shape"])
