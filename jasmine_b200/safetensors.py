"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, offsets), data."""
from __future__ import annotations

import json
import mmap
from pathlib import Path

import numpy as np

# bf16 has no numpy type: its tensors come back as uint16 bit patterns
DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class SafeTensors:
    """Memory-mapped view of one file: iterate names, `get(name)` -> (dtype name, array)."""

    def __init__(self, path):
        self._f = open(Path(path), "rb")
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        n = int.from_bytes(self._map[:8], "little")
        if n > len(self._map) - 8:
            raise ValueError(f"{path}: not a safetensors file")
        header = json.loads(self._map[8:8 + n])
        self._base = 8 + n
        self._entries = {k: v for k, v in header.items() if k != "__metadata__"}

    def __iter__(self):
        return iter(self._entries)

    def __contains__(self, name):
        return name in self._entries

    def get(self, name):
        e = self._entries[name]
        if e["dtype"] not in DTYPES:
            raise ValueError(f"tensor {name}: dtype {e['dtype']}")
        lo, hi = e["data_offsets"]
        dt = np.dtype(DTYPES[e["dtype"]])
        a = np.frombuffer(self._map, dt, (hi - lo) // dt.itemsize, self._base + lo)
        return e["dtype"], a.reshape(e["shape"])
