"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets) and the tensor data, memory-mapped.  The counterpart of gguf.py for dense checkpoints."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

# bf16 has no numpy type: its bit patterns are handed out as uint16
DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8, "I16": np.int16,
          "U16": np.uint16, "I32": np.int32, "U32": np.uint32, "I64": np.int64, "U64": np.uint64, "BOOL": np.bool_}


class SafetensorsFile:
    """tensors[name] = (dtype name, shape); get(name) = array (BF16: uint16 bit patterns) over the mapping."""

    def __init__(self, path: str):
        self.path = path
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError(f"{path}: not a safetensors file")
            n = struct.unpack("<Q", head)[0]
            if n > size - 8:
                raise ValueError(f"{path}: the header length passes the end of the file")
            header = json.loads(f.read(n))
        header.pop("__metadata__", None)
        self._base, self._size = 8 + n, size
        self._map = np.memmap(path, dtype=np.uint8, mode="r") if size else np.empty(0, np.uint8)
        self.tensors, self._span = {}, {}
        for name, t in header.items():
            dtype, shape, (lo, hi) = t["dtype"], tuple(int(d) for d in t["shape"]), t["data_offsets"]
            if dtype not in DTYPES:
                raise ValueError(f"{name}: unknown element type {dtype}")
            want = int(np.prod(shape, dtype=np.int64)) * np.dtype(DTYPES[dtype]).itemsize
            if lo < 0 or hi - lo != want or self._base + hi > size:
                raise ValueError(f"{name}: {hi - lo} bytes do not hold {shape} {dtype}")
            self.tensors[name] = (dtype, shape)
            self._span[name] = (self._base + lo, self._base + hi)

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def get(self, name: str) -> np.ndarray:
        if name not in self.tensors:
            raise KeyError(f"{self.path} has no tensor {name!r}")
        dtype, shape = self.tensors[name]
        lo, hi = self._span[name]
        return np.frombuffer(self._map[lo:hi].tobytes(), dtype=DTYPES[dtype]).reshape(shape)

    def bf16_bits(self, name: str, shape) -> np.ndarray:
        """A weight as bf16 bit patterns; its stored type must be BF16 and its shape the expected one."""
        dtype, have = self.tensors.get(name, (None, None))
        if dtype is None:
            raise KeyError(f"{self.path} has no tensor {name!r}")
        if have != tuple(shape):
            raise ValueError(f"{name} is {list(have)}, expected {list(shape)}")
        if dtype != "BF16":
            raise ValueError(f"{name} is {dtype}, expected BF16")
        return self.get(name)


def write_safetensors(path: str, tensors: dict) -> None:
    """tensors: name -> array; uint16 arrays are written as BF16 bit patterns."""
    names = {np.dtype(v): k for k, v in DTYPES.items() if k not in ("BF16", "U16")}
    header, at = {}, 0
    for name, a in tensors.items():
        dtype = "BF16" if a.dtype == np.uint16 else names[a.dtype]
        header[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    raw = json.dumps(header).encode()
    raw += b" " * (-len(raw) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(raw)) + raw)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())
