"""The safetensors container: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the data.  Host bookkeeping only; tensors are views into the mapped file."""
from __future__ import annotations

import json
import struct
from typing import Dict, Iterator, Tuple

import numpy as np

# bfloat16 has no numpy type: its bit patterns are returned as uint16
DTYPES = {"BF16": np.uint16, "F32": np.float32, "F16": np.float16, "I32": np.int32, "I64": np.int64, "U8": np.uint8, "I8": np.int8}


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        self.data = np.memmap(path, np.uint8, mode="r")
        if self.data.size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        (n,) = struct.unpack("<Q", self.data[:8].tobytes())
        if n > self.data.size - 8:
            raise ValueError(f"{path}: the header is longer than the file")
        header = json.loads(self.data[8:8 + n].tobytes())
        header.pop("__metadata__", None)
        self.base = 8 + n
        self.entries: Dict[str, Tuple[str, Tuple[int, ...], int, int]] = {}
        for name, e in header.items():
            lo, hi = e["data_offsets"]
            shape = tuple(int(d) for d in e["shape"])
            if e["dtype"] not in DTYPES:
                raise ValueError(f"{path}: {name} has type {e['dtype']}")
            if hi - lo != int(np.prod(shape, dtype=np.int64)) * np.dtype(DTYPES[e["dtype"]]).itemsize or self.base + hi > self.data.size or lo < 0:
                raise ValueError(f"{path}: the extent of {name} does not fit its shape or the file")
            self.entries[name] = (e["dtype"], shape, lo, hi)

    def __contains__(self, name: str) -> bool:
        return name in self.entries

    def __iter__(self) -> Iterator[str]:
        return iter(self.entries)

    def dtype(self, name: str) -> str:
        return self.entries[name][0]

    def shape(self, name: str) -> Tuple[int, ...]:
        return self.entries[name][1]

    def __getitem__(self, name: str) -> np.ndarray:
        dtype, shape, lo, hi = self.entries[name]
        return np.frombuffer(self.data[self.base + lo:self.base + hi].tobytes(), DTYPES[dtype]).reshape(shape)


def write(path: str, tensors: Dict[str, np.ndarray], bf16=()) -> None:
    """tensors: name -> array; the uint16 arrays named in `bf16` (or all of them if it is True) hold bfloat16 bits."""
    names = {np.dtype(v): k for k, v in DTYPES.items() if k != "BF16"}
    header, at = {}, 0
    for name, a in tensors.items():
        is_bf16 = a.dtype == np.uint16 and (bf16 is True or name in bf16)
        header[name] = {"dtype": "BF16" if is_bf16 else names[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())
