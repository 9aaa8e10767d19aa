"""safetensors files: a u64 header size, a JSON header (per tensor: dtype, shape, byte range in the data section),
the data section. The file is mapped; a tensor is a view of it."""
from __future__ import annotations

import json
import mmap
import struct
from dataclasses import dataclass
from typing import Dict, Sequence, Tuple

import numpy as np

_NUMPY = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "BF16": np.uint16, "I64": np.int64, "I32": np.int32,
          "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}


class SafetensorsError(Exception):
    pass


@dataclass
class TensorInfo:
    dtype: str
    shape: Tuple[int, ...]
    begin: int
    end: int


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (np.ascontiguousarray(bits).astype(np.uint32) << np.uint32(16)).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    """Bit patterns (uint16) of the nearest bf16 values, ties to even."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + ((u >> np.uint32(16)) & np.uint32(1)) + np.uint32(0x7FFF)) >> np.uint32(16)).astype(np.uint16)


class SafetensorsFile:
    def __init__(self, path: str):
        self._f = open(path, "rb")
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise SafetensorsError("file is shorter than its header length")
        n = struct.unpack("<Q", self._map[:8])[0]
        if 8 + n > len(self._map):
            raise SafetensorsError(f"header of {n} bytes does not fit the file")
        self._base = 8 + n
        self.tensors: Dict[str, TensorInfo] = {}
        self.metadata: Dict[str, str] = {}
        for name, t in json.loads(self._map[8:8 + n]).items():
            if name == "__metadata__":
                self.metadata = t
                continue
            if t["dtype"] not in _NUMPY:
                raise SafetensorsError(f"{name}: unknown dtype {t['dtype']}")
            b, e = t["data_offsets"]
            count = int(np.prod(t["shape"], dtype=np.int64))
            if b < 0 or e < b or self._base + e > len(self._map) or e - b != count * np.dtype(_NUMPY[t["dtype"]]).itemsize:
                raise SafetensorsError(f"{name}: data range [{b}, {e}) does not fit shape {t['shape']} of {t['dtype']}")
            self.tensors[name] = TensorInfo(t["dtype"], tuple(t["shape"]), b, e)

    def info(self, name: str) -> TensorInfo:
        if name not in self.tensors:
            raise SafetensorsError(f"tensor {name} is missing")
        return self.tensors[name]

    def raw(self, name: str) -> np.ndarray:
        """The stored values (bf16 as uint16 bit patterns)."""
        t = self.info(name)
        dt = np.dtype(_NUMPY[t.dtype])
        return np.frombuffer(self._map, dt, (t.end - t.begin) // dt.itemsize, self._base + t.begin).reshape(t.shape)

    def f32(self, name: str) -> np.ndarray:
        v = self.raw(name)
        return bf16_to_f32(v).reshape(v.shape) if self.tensors[name].dtype == "BF16" else v.astype(np.float32)

    def bf16(self, name: str) -> np.ndarray:
        """Bit patterns (uint16) of the tensor in bf16."""
        v = self.raw(name)
        return v if self.tensors[name].dtype == "BF16" else f32_to_bf16(v.astype(np.float32)).reshape(v.shape)


def write_safetensors(path: str, tensors: Dict[str, Tuple[str, Sequence[int], np.ndarray]]) -> None:
    """tensors: name -> (dtype, shape, array of that dtype; BF16 as uint16 bit patterns)."""
    head, at, blobs = {}, 0, []
    for name, (dtype, shape, a) in tensors.items():
        b = np.ascontiguousarray(a, dtype=_NUMPY[dtype]).tobytes()
        head[name] = {"dtype": dtype, "shape": list(shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    js = json.dumps(head).encode()
    js += b" " * (-len(js) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(js)) + js + b"".join(blobs))
