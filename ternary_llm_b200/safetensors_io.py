"""The safetensors container: an 8-byte little-endian header length, a JSON table
name -> {dtype, shape, data_offsets}, then the data.  Reader (memory-mapped) and writer.

numpy has no bfloat16: BF16 tensors are uint16 arrays of bit patterns here, marked by the
reader's `dtypes`; to_bf16 / from_bf16 convert.
"""
from __future__ import annotations

import json
import os

import numpy as np

_NP = {"BF16": "<u2", "F16": "<f2", "F32": "<f4", "I32": "<i4", "I64": "<i8", "U8": "u1"}


def to_bf16(a: np.ndarray) -> np.ndarray:
    """float array -> BF16 bit patterns (round to nearest even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(u: np.ndarray) -> np.ndarray:
    return (np.asarray(u).astype(np.uint32) << 16).view(np.float32)


class SafetensorsFile:
    """Mapping name -> array (a view into the mapped file)."""

    def __init__(self, path: str):
        self.path = path
        size = os.path.getsize(path)
        if size < 8:
            raise ValueError(f"{path}: too short for a safetensors file")
        buf = np.memmap(path, dtype=np.uint8, mode="r")
        n = int.from_bytes(bytes(buf[:8]), "little")
        if n > size - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        table = json.loads(bytes(buf[8:8 + n]).decode("utf-8"))
        table.pop("__metadata__", None)
        data = buf[8 + n:]
        self.dtypes, self._arrays = {}, {}
        for name, e in table.items():
            a, b = e["data_offsets"]
            if e["dtype"] not in _NP:
                raise ValueError(f"{path}: tensor {name} has dtype {e['dtype']}")
            dt = np.dtype(_NP[e["dtype"]])
            count = int(np.prod(e["shape"], dtype=np.int64))
            if not 0 <= a <= b <= data.size or b - a != count * dt.itemsize:
                raise ValueError(f"{path}: tensor {name} does not fit its byte range")
            # the format does not align its data: copy a tensor whose view would be misaligned
            raw = data[a:b]
            if (8 + n + a) % dt.itemsize:
                raw = np.array(raw)
            self._arrays[name] = raw.view(dt).reshape(e["shape"])
            self.dtypes[name] = e["dtype"]

    def __getitem__(self, name: str) -> np.ndarray:
        return self._arrays[name]

    def __contains__(self, name: str) -> bool:
        return name in self._arrays

    def keys(self):
        return self._arrays.keys()


def write_safetensors(path: str, tensors: dict) -> None:
    """tensors: name -> array; uint16 arrays are written as BF16."""
    names = {"uint16": "BF16", "float16": "F16", "float32": "F32", "int32": "I32", "int64": "I64", "uint8": "U8"}
    table, off, blobs = {}, 0, []
    for name, a in tensors.items():
        a = np.ascontiguousarray(a)
        raw = a.tobytes()
        table[name] = {"dtype": names[a.dtype.name], "shape": list(a.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little"))
        f.write(head)
        for b in blobs:
            f.write(b)
