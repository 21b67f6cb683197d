"""Streaming reader of the safetensors layout: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets), then the raw bytes.  Used for stand-alone files and for the member inside a `.vn` archive."""

from __future__ import annotations

import json
import struct
from typing import Dict, Iterator, Tuple

import numpy as np

_DTYPES = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "I64": np.int64, "I32": np.int32,
           "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_, "U16": np.uint16, "U32": np.uint32,
           "U64": np.uint64}


def _bf16_to_f32(raw: bytes, shape) -> np.ndarray:
    u = np.frombuffer(raw, dtype=np.uint16).astype(np.uint32) << np.uint32(16)
    return u.view(np.float32).reshape(shape)


def read_header(f) -> dict:
    """Header of an open stream, which is left at the first data byte."""
    (hlen,) = struct.unpack("<Q", f.read(8))
    if hlen > (100 << 20):
        raise ValueError("implausible safetensors header length")
    header = json.loads(f.read(hlen).decode("utf-8"))
    header.pop("__metadata__", None)
    return header


def iter_tensors(f, header: dict) -> Iterator[Tuple[str, np.ndarray]]:
    """(name, array) pairs in file order from a stream positioned at the first data byte; floating-point tensors come out
    as float32, integer tensors in their own dtype."""
    pos = 0
    for name, e in sorted(header.items(), key=lambda ne: ne[1]["data_offsets"][0]):
        lo, hi = e["data_offsets"]
        if lo < pos:
            raise ValueError(f"{name}: overlapping tensor data")
        if lo > pos:
            f.read(lo - pos)
        raw = f.read(hi - lo)
        pos = hi
        if len(raw) != hi - lo:
            raise ValueError(f"{name}: truncated tensor data")
        shape = tuple(e["shape"])
        if e["dtype"] == "BF16":
            yield name, _bf16_to_f32(raw, shape)
            continue
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{name}: unsupported dtype {e['dtype']}")
        arr = np.frombuffer(raw, dtype=_DTYPES[e["dtype"]]).reshape(shape)
        yield name, arr.astype(np.float32) if arr.dtype in (np.float64, np.float16) else arr


class SafetensorsFile:
    def __init__(self, path: str):
        self._f = open(path, "rb")
        self.header = read_header(self._f)
        self._data = self._f.tell()

    def shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {n: tuple(e["shape"]) for n, e in self.header.items()}

    def __iter__(self):
        self._f.seek(self._data)
        return iter_tensors(self._f, self.header)

    def close(self):
        self._f.close()

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()
        return False
