"""safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets) and the
tensors' bytes.  The file is memory-mapped; every range is checked against the file before it is used."""
from __future__ import annotations

import json
import mmap
from typing import Dict, Tuple

import numpy as np

from .capi import ERR_INVALID_ARG, RatchetCudaError, from_bf16

_NP = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "BF16": np.uint16, "I64": np.int64, "I32": np.int32, "I16": np.int16, "I8": np.int8,
       "U8": np.uint8, "BOOL": np.bool_}


class SafetensorsFile:
    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._map)
        n = int.from_bytes(self._map[:8], "little") if size >= 8 else size
        if 8 + n > size:
            raise RatchetCudaError(ERR_INVALID_ARG, f"{path}: the header reaches beyond the file")
        header = json.loads(self._map[8:8 + n].decode("utf-8"))
        header.pop("__metadata__", None)
        self.tensors: Dict[str, Tuple[str, Tuple[int, ...], int]] = {}
        for name, t in header.items():
            a, b = (int(v) for v in t["data_offsets"])
            shape = tuple(int(s) for s in t["shape"])
            if t["dtype"] not in _NP:
                raise RatchetCudaError(ERR_INVALID_ARG, f"{path}: {name} has dtype {t['dtype']}")
            want = int(np.prod(shape, dtype=np.int64)) * np.dtype(_NP[t["dtype"]]).itemsize
            if not 0 <= a <= b <= size - 8 - n or b - a != want:
                raise RatchetCudaError(ERR_INVALID_ARG, f"{path}: {name} does not fit its data range")
            self.tensors[name] = (t["dtype"], shape, 8 + n + a)

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def shape(self, name: str) -> Tuple[int, ...]:
        return self._entry(name)[1]

    def _entry(self, name: str):
        if name not in self.tensors:
            raise RatchetCudaError(ERR_INVALID_ARG, f"the file has no tensor {name}")
        return self.tensors[name]

    def raw(self, name: str) -> Tuple[str, np.ndarray]:
        """(dtype name, array over the mapped file); BF16 comes as uint16 bit patterns."""
        dt, shape, at = self._entry(name)
        count = int(np.prod(shape, dtype=np.int64))
        return dt, np.frombuffer(self._map, _NP[dt], count, at).reshape(shape)

    def f32(self, name: str) -> np.ndarray:
        dt, a = self.raw(name)
        return from_bf16(a) if dt == "BF16" else a.astype(np.float32)
