"""Reader of safetensors files.  The JSON header follows its own length (u64, little-endian) and gives
each tensor's dtype, shape and place in the data behind it.  The file is mapped, not copied."""
from __future__ import annotations

import json
import mmap
from pathlib import Path


class SafetensorsFile:
    def __init__(self, path):
        path = Path(path)
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._map)
        n = int.from_bytes(self._map[:8], "little") if size >= 8 else -1
        if n < 0 or 8 + n > size:
            raise ValueError(f"{path}: not a safetensors file (header of {n} bytes in a file of {size})")
        header = json.loads(self._map[8:8 + n].decode("utf-8"))
        header.pop("__metadata__", None)
        self.tensors, view = {}, memoryview(self._map)
        for name, t in header.items():
            a, b = t["data_offsets"]
            if not 0 <= a <= b <= size - 8 - n:
                raise ValueError(f"{path}: tensor {name!r} lies outside the file")
            self.tensors[name] = (t["dtype"], tuple(t["shape"]), view[8 + n + a:8 + n + b])

    def items(self):
        return self.tensors.items()
