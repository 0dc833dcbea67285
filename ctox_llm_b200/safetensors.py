"""safetensors files without a dependency: tensors are views over a read-only mapping. The header is a
JSON object behind its uint64 size; offsets count from the end of the header."""
from __future__ import annotations

import json
import mmap
import struct
from typing import Dict

import numpy as np

from ._native import CtoxError

INVALID_ARTIFACT, UNSUPPORTED_DTYPE = 2, 3
ITEM_BYTES = {"BF16": 2, "F16": 2, "F32": 4, "I32": 4}


class SafetensorsFile:
    def __init__(self, path: str):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise CtoxError(INVALID_ARTIFACT, f"{path}: shorter than its length field")
        n = struct.unpack_from("<Q", self._map)[0]
        if 8 + n > len(self._map):
            raise CtoxError(INVALID_ARTIFACT, f"{path}: header lies beyond the file")
        try:
            entries = json.loads(self._map[8:8 + n])
        except ValueError as e:
            raise CtoxError(INVALID_ARTIFACT, f"{path}: header is not JSON: {e}")
        entries.pop("__metadata__", None)
        self._data = 8 + n
        self.tensors: Dict[str, dict] = entries
        for name, t in entries.items():
            begin, end = t["data_offsets"]
            if t["dtype"] not in ITEM_BYTES:
                raise CtoxError(UNSUPPORTED_DTYPE, f"tensor {name} is {t['dtype']}")
            count = int(np.prod(t["shape"], dtype=np.int64))
            if begin < 0 or self._data + end > len(self._map) or end - begin != count * ITEM_BYTES[t["dtype"]]:
                raise CtoxError(INVALID_ARTIFACT, f"tensor {name}: data range does not match its shape")

    def _entry(self, name: str) -> dict:
        if name not in self.tensors:
            raise CtoxError(INVALID_ARTIFACT, f"tensor {name} is not in the file")
        return self.tensors[name]

    def shape(self, name: str) -> list:
        return list(self._entry(name)["shape"])

    def raw(self, name: str) -> np.ndarray:
        """The tensor's bytes (uint8 view)."""
        begin, end = self._entry(name)["data_offsets"]
        return np.frombuffer(self._map, dtype=np.uint8, count=end - begin, offset=self._data + begin)

    def bf16_matrix(self, name: str) -> tuple:
        """(bytes, rows, columns) of a bf16 matrix."""
        t = self._entry(name)
        if t["dtype"] != "BF16" or len(t["shape"]) != 2:
            raise CtoxError(UNSUPPORTED_DTYPE, f"tensor {name} is not a bf16 matrix")
        return self.raw(name), int(t["shape"][0]), int(t["shape"][1])

    def float_vector(self, name: str) -> np.ndarray:
        """The tensor as fp32 values."""
        t, raw = self._entry(name), self.raw(name)
        if t["dtype"] == "BF16":
            return (raw.view("<u2").astype(np.uint32) << 16).view(np.float32)
        if t["dtype"] == "F16":
            return raw.view("<f2").astype(np.float32)
        if t["dtype"] == "F32":
            return raw.view("<f4").copy()
        raise CtoxError(UNSUPPORTED_DTYPE, f"tensor {name} is {t['dtype']}, not a float tensor")


def write_safetensors(path: str, tensors: Dict[str, tuple]) -> None:
    """tensors: name -> (dtype string, shape, contiguous array whose bytes are the payload)."""
    head, offset = {}, 0
    for name, (dtype, shape, data) in tensors.items():
        head[name] = {"dtype": dtype, "shape": list(shape), "data_offsets": [offset, offset + data.nbytes]}
        offset += data.nbytes
    blob = json.dumps(head).encode()
    blob += b" " * (-len(blob) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(blob)))
        f.write(blob)
        for _, _, data in tensors.values():
            f.write(data.tobytes())
