"""Reader (and a small writer) of the safetensors container: an 8-byte little-endian header length, that many bytes of
JSON (name -> dtype, shape, data_offsets), then the data. bfloat16 tensors are handled as uint16 bit patterns."""
from __future__ import annotations

import json
import mmap
import struct

import numpy as np

_NUMPY_OF = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I64": np.int64, "I32": np.int32,
             "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}


class SafetensorsError(ValueError):
    pass


class SafetensorsFile:
    """`name in f`, f.names(), f.dtype(name), f.shape(name), f[name] (a read-only numpy view of the mapped file)."""

    def __init__(self, path):
        self._f = open(path, "rb")
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise SafetensorsError(f"{path}: too short")
        n = struct.unpack("<Q", self._map[:8])[0]
        if n > len(self._map) - 8:
            raise SafetensorsError(f"{path}: header of {n} bytes in a file of {len(self._map)}")
        header = json.loads(self._map[8:8 + n].decode("utf-8"))
        header.pop("__metadata__", None)
        self._base = 8 + n
        self._entries = header
        for name, e in header.items():
            if e["dtype"] not in _NUMPY_OF:
                raise SafetensorsError(f"{name}: unsupported dtype {e['dtype']}")
            a, b = e["data_offsets"]
            size = int(np.prod(e["shape"], dtype=np.int64)) * np.dtype(_NUMPY_OF[e["dtype"]]).itemsize
            if b - a != size or a < 0 or self._base + b > len(self._map):
                raise SafetensorsError(f"{name}: data offsets {a} .. {b} do not fit its shape or the file")

    def names(self):
        return list(self._entries)

    def __contains__(self, name):
        return name in self._entries

    def dtype(self, name) -> str:
        return self._entries[name]["dtype"]

    def shape(self, name):
        return tuple(self._entries[name]["shape"])

    def __getitem__(self, name) -> np.ndarray:
        if name not in self._entries:
            raise SafetensorsError(f"tensor '{name}' is missing")
        e = self._entries[name]
        count = int(np.prod(e["shape"], dtype=np.int64))
        return np.frombuffer(self._map, dtype=_NUMPY_OF[e["dtype"]], count=count,
                             offset=self._base + e["data_offsets"][0]).reshape(e["shape"])


def write_safetensors(path, tensors: dict) -> None:
    """name -> numpy array; uint16 arrays are stored as BF16."""
    code = {np.dtype(v): k for k, v in _NUMPY_OF.items()}
    header, at, blobs = {}, 0, []
    for name, a in tensors.items():
        a = np.asarray(a)
        data = a.tobytes()
        header[name] = {"dtype": code[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + len(data)]}
        at += len(data)
        blobs.append(data)
    h = json.dumps(header).encode("utf-8")
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)
