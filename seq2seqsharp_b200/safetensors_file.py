"""Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets), the data.

bfloat16 tensors come back as their bit patterns (uint16 arrays), which the engine takes as they are; `to_float32` widens them.
Only the Python standard library and NumPy are used.
"""
import json
import os
import struct
from typing import Dict, Iterator, Tuple

import numpy as np

_DTYPES = {"BF16": np.dtype("<u2"), "F32": np.dtype("<f4"), "I32": np.dtype("<i4"), "F16": np.dtype("<f2")}


def to_float32(a: np.ndarray) -> np.ndarray:
    """float32 values of a tensor as the reader returns it (uint16 arrays are bfloat16 bit patterns)."""
    if a.dtype == np.uint16:
        return (a.astype(np.uint32) << 16).view(np.float32)
    return a.astype(np.float32)


def to_bfloat16(a: np.ndarray) -> np.ndarray:
    """bfloat16 bit patterns (uint16) of float32 values, rounded to nearest even."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        size = os.path.getsize(path)
        with open(path, "rb") as fh:
            head = fh.read(8)
            if len(head) < 8:
                raise ValueError("%s: too short for a safetensors file" % path)
            n = struct.unpack("<Q", head)[0]
            if n > size - 8:
                raise ValueError("%s: the header is longer than the file" % path)
            self.header = json.loads(fh.read(n).decode("utf-8"))
        self.header.pop("__metadata__", None)
        self._base = 8 + n
        for name, t in self.header.items():
            if t["dtype"] not in _DTYPES:
                raise ValueError("%s: tensor %s has unsupported type %s" % (path, name, t["dtype"]))
            a, e = t["data_offsets"]
            count = int(np.prod(t["shape"], dtype=np.int64)) if t["shape"] else 1
            if a < 0 or e - a != count * _DTYPES[t["dtype"]].itemsize or self._base + e > size:
                raise ValueError("%s: tensor %s does not fit its place in the file" % (path, name))

    def __contains__(self, name):
        return name in self.header

    def names(self):
        return list(self.header)

    def shape(self, name: str) -> Tuple[int, ...]:
        return tuple(self.header[name]["shape"])

    def get(self, name: str) -> np.ndarray:
        t = self.header[name]
        a, e = t["data_offsets"]
        dt = _DTYPES[t["dtype"]]
        return np.fromfile(self.path, dtype=dt, count=(e - a) // dt.itemsize, offset=self._base + a).reshape(t["shape"])

    def items(self) -> Iterator[Tuple[str, np.ndarray]]:
        for name in self.header:
            yield name, self.get(name)


def write_safetensors(path: str, tensors: Dict[str, np.ndarray]):
    """Writes arrays (float32, int32, or uint16 = bfloat16 bit patterns)."""
    kinds = {np.dtype("uint16"): "BF16", np.dtype("float32"): "F32", np.dtype("int32"): "I32"}
    header, at = {}, 0
    arrays = {k: np.ascontiguousarray(v) for k, v in tensors.items()}
    for name, a in arrays.items():
        header[name] = {"dtype": kinds[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    head = json.dumps(header).encode("utf-8")
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as fh:
        fh.write(struct.pack("<Q", len(head)))
        fh.write(head)
        for a in arrays.values():
            fh.write(a.tobytes())
