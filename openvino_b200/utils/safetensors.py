"""Reader of the safetensors format: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the data. The file is mapped; a tensor is copied only when it is asked for."""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Dict, Iterator, List, Tuple

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64, "I32": torch.int32,
           "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = os.fspath(path)
        with open(self.path, "rb") as f:
            size = os.fstat(f.fileno()).st_size
            if size < 8:
                raise ValueError("%s: not a safetensors file" % self.path)
            (n,) = struct.unpack("<Q", f.read(8))
            if n > size - 8:
                raise ValueError("%s: header of %d bytes in a file of %d" % (self.path, n, size))
            header = json.loads(f.read(n))
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        self._base, self._size = 8 + n, size
        self._entries: Dict[str, dict] = {k: v for k, v in header.items() if k != "__metadata__"}

    def keys(self) -> List[str]:
        return list(self._entries)

    def __contains__(self, name: str) -> bool:
        return name in self._entries

    def __iter__(self) -> Iterator[str]:
        return iter(self._entries)

    def shape(self, name: str) -> Tuple[int, ...]:
        return tuple(self._entries[name]["shape"])

    def __getitem__(self, name: str) -> torch.Tensor:
        e = self._entries[name]
        if e["dtype"] not in _DTYPES:
            raise ValueError("%s: %s has the unsupported type %s" % (self.path, name, e["dtype"]))
        dtype, shape = _DTYPES[e["dtype"]], tuple(e["shape"])
        lo, hi = e["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        itemsize = torch.empty((), dtype=dtype).element_size()
        if hi - lo != count * itemsize or lo < 0 or self._base + hi > self._size:
            raise ValueError("%s: %s does not fit its shape" % (self.path, name))
        if count == 0:
            return torch.empty(shape, dtype=dtype)
        return torch.frombuffer(bytearray(self._map[self._base + lo:self._base + hi]), dtype=dtype).reshape(shape)
