"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, byte range
behind the header), the data.  The file is mapped; a tensor is a view of the map."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

ITEM_BYTES = {"BF16": 2, "F16": 2, "F32": 4, "I32": 4, "I64": 8, "U8": 1, "I8": 1, "F64": 8, "BOOL": 1}


class SafetensorsError(ValueError):
    pass


class SafetensorsFile:
    def __init__(self, path):
        self._map = np.memmap(path, np.uint8, mode="r") if os.path.getsize(path) else np.empty(0, np.uint8)
        if self._map.size < 8:
            raise SafetensorsError("truncated safetensors header")
        n, = struct.unpack("<Q", self._map[:8].tobytes())
        if n > self._map.size - 8:
            raise SafetensorsError("truncated safetensors header")
        try:
            head = json.loads(self._map[8:8 + n].tobytes())
        except ValueError as e:
            raise SafetensorsError(f"safetensors header: {e}") from None
        if not isinstance(head, dict):
            raise SafetensorsError("safetensors header is not an object")
        self._data = self._map[8 + n:]
        self._info = {}
        for name, t in head.items():
            if name == "__metadata__":
                continue
            try:
                dtype, shape, (a, b) = t["dtype"], tuple(t["shape"]), t["data_offsets"]
                size = ITEM_BYTES[dtype] * int(np.prod(shape, dtype=np.int64))
            except (KeyError, TypeError, ValueError):
                raise SafetensorsError(f"{name}: malformed entry") from None
            if not 0 <= a <= b <= self._data.size or b - a != size:
                raise SafetensorsError(f"{name}: byte range does not match its shape or the file")
            self._info[name] = (dtype, shape, a, b)

    def __contains__(self, name: str) -> bool:
        return name in self._info

    def names(self) -> list:
        return list(self._info)

    def shape(self, name: str) -> tuple:
        return self._info[name][1]

    def dtype(self, name: str) -> str:
        return self._info[name][0]

    def raw(self, name: str) -> np.ndarray:
        """The tensor's bytes."""
        if name not in self._info:
            raise SafetensorsError(f"the file has no tensor {name}")
        _, _, a, b = self._info[name]
        return self._data[a:b]

    def f32(self, name: str) -> np.ndarray:
        """A small tensor as float32 (norm weights, biases, tables)."""
        raw, dt = self.raw(name), self.dtype(name)
        if dt == "BF16":
            v = (np.frombuffer(raw.tobytes(), np.uint16).astype(np.uint32) << 16).view(np.float32)
        elif dt in ("F32", "F16"):
            v = np.frombuffer(raw.tobytes(), np.float32 if dt == "F32" else np.float16).astype(np.float32)
        else:
            raise SafetensorsError(f"{name}: {dt} is not a float tensor")
        return v.reshape(self.shape(name))
