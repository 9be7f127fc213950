"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets relative to the end of the header), the data.  The file is mapped, tensors are read one by one."""
from __future__ import annotations

import json
import mmap
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "I32": torch.int32, "I64": torch.int64}


class SafetensorsFile:
    def __init__(self, path: str):
        self._f = open(path, "rb")
        head = self._f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", head)[0]
        self._f.seek(0, 2)
        size = self._f.tell()
        if n > size - 8:
            raise ValueError(f"{path}: header longer than the file")
        self._f.seek(8)
        self._header = {k: v for k, v in json.loads(self._f.read(n)).items() if k != "__metadata__"}
        self._base = 8 + n
        self._data_bytes = size - self._base
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)

    def keys(self):
        return self._header.keys()

    def __contains__(self, name) -> bool:
        return name in self._header

    def __getitem__(self, name: str) -> torch.Tensor:
        meta = self._header[name]
        dtype = _DTYPES.get(meta["dtype"])
        if dtype is None:
            raise ValueError(f"{name}: unsupported dtype {meta['dtype']}")
        lo, hi = meta["data_offsets"]
        shape = tuple(meta["shape"])
        count = 1
        for s in shape:
            count *= s
        if not 0 <= lo <= hi <= self._data_bytes or hi - lo != count * torch.empty((), dtype=dtype).element_size():
            raise ValueError(f"{name}: data_offsets do not fit shape and file")
        if count == 0:
            return torch.empty(shape, dtype=dtype)
        raw = bytearray(self._map[self._base + lo:self._base + hi])
        return torch.frombuffer(raw, dtype=dtype).view(shape)

    def close(self) -> None:
        self._map.close()
        self._f.close()

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()
