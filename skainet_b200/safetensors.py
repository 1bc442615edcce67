"""Tensors of a safetensors file, memory-mapped: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets relative to the end of the header), then the data. The counterpart of gguf.py for checkpoints in that format."""
from __future__ import annotations

import json
import mmap
import struct
from dataclasses import dataclass
from typing import Dict

import numpy as np

_ITEM = {"BF16": 2, "F16": 2, "F32": 4, "I32": 4, "I64": 8, "U8": 1, "I8": 1}
_NUMPY = {"F16": np.float16, "F32": np.float32, "I32": np.int32, "I64": np.int64, "U8": np.uint8, "I8": np.int8}


@dataclass
class TensorInfo:
    name: str
    dtype: str
    shape: tuple
    offset: int      # absolute, in the file
    nbytes: int


class SafetensorsReader:
    def __init__(self, path: str):
        self.path = path
        self._f = open(path, "rb")
        self._mm = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._mm)
        n = struct.unpack_from("<Q", self._mm, 0)[0] if size >= 8 else size
        if 8 + n > size:
            raise ValueError(f"{path}: not a safetensors file")
        header = json.loads(self._mm[8:8 + n].decode("utf-8"))
        self.metadata = header.pop("__metadata__", {})
        self.tensors: Dict[str, TensorInfo] = {}
        for name, t in header.items():
            if t["dtype"] not in _ITEM:
                raise ValueError(f"{path}: {name}: data type {t['dtype']} not supported")
            begin, end = t["data_offsets"]
            shape = tuple(int(d) for d in t["shape"])
            need = int(np.prod(shape, dtype=np.int64)) * _ITEM[t["dtype"]]
            if end - begin != need or 8 + n + end > size or begin < 0:
                raise ValueError(f"{path}: {name}: {end - begin} bytes for {t['dtype']} {list(shape)}")
            self.tensors[name] = TensorInfo(name, t["dtype"], shape, 8 + n + begin, need)

    def tensor(self, name: str) -> TensorInfo:
        if name not in self.tensors:
            raise ValueError(f"{self.path}: tensor {name} not found")
        return self.tensors[name]

    def raw(self, name: str) -> np.ndarray:
        """The tensor's bytes, a view of the mapped file."""
        t = self.tensor(name)
        return np.frombuffer(self._mm, dtype=np.uint8, count=t.nbytes, offset=t.offset)

    def floats(self, name: str) -> np.ndarray:
        """A floating-point tensor as fp32 (exact for BF16 and F16)."""
        t = self.tensor(name)
        raw = self.raw(name)
        if t.dtype == "BF16":
            return (raw.view(np.uint16).astype(np.uint32) << 16).view(np.float32).reshape(t.shape)
        if t.dtype not in ("F16", "F32"):
            raise ValueError(f"{name}: {t.dtype} is not a floating-point type")
        return raw.view(_NUMPY[t.dtype]).astype(np.float32).reshape(t.shape)

    def weight(self, name: str, rows: int, cols: int):
        """A BF16 matrix as a resident weight."""
        from .device import Weight
        t = self.tensor(name)
        if t.dtype != "BF16" or t.shape != (rows, cols):
            raise ValueError(f"{name}: {t.dtype} {list(t.shape)}, expected BF16 [{rows}, {cols}]")
        return Weight.upload(self.raw(name), "BF16", rows, cols)

    def close(self) -> None:
        self._mm.close()
        self._f.close()


def write(path: str, tensors: Dict[str, tuple]) -> None:
    """Writes name -> (dtype, shape, array whose bytes are the data)."""
    header, at, blobs = {}, 0, []
    for name, (dtype, shape, a) in tensors.items():
        b = np.ascontiguousarray(a).tobytes()
        header[name] = {"dtype": dtype, "shape": list(shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode("utf-8")
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
