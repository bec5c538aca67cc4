"""From the tensors of a safetensors file to the matrices and vectors a session is made of."""
from __future__ import annotations

import numpy as np

from ..executor import BF16
from ..safetensors import SafetensorsError, SafetensorsFile


class Weights:
    """Uploads tensors of one file, stacked by rows where the products of a layer share their input."""

    def __init__(self, ex, file: SafetensorsFile):
        self.ex, self.file = ex, file

    def stack(self, *parts):
        """parts: (name, rows, cols), or a number of rows of zeros; one resident BF16 matrix of all their rows."""
        cols = next(p[2] for p in parts if not isinstance(p, int))
        raw = [np.zeros(2 * p * cols, np.uint8) if isinstance(p, int) else self._raw(*p) for p in parts]
        return self.ex.upload(BF16, sum(p if isinstance(p, int) else p[1] for p in parts), cols, raw[0] if len(raw) == 1 else np.concatenate(raw))

    def beside(self, *parts):
        """parts: (name, rows, cols) of equal rows; one resident BF16 matrix of all their columns."""
        rows = parts[0][1]
        raw = [self._raw(name, r, c).reshape(rows, 2 * c) for name, r, c in parts]
        return self.ex.upload(BF16, rows, sum(c for _, _, c in parts), np.concatenate(raw, 1).reshape(-1))

    def blocks(self, n, rows, cols, *names):
        """Tensors of n blocks of rows x cols each; one resident BF16 matrix that stacks the first block of each, the second
        block of each, ..."""
        raw = [self._raw(name, n, rows, cols).reshape(n, 1, 2 * rows * cols) for name in names]
        return self.ex.upload(BF16, n * rows * len(names), cols, np.concatenate(raw, 1).reshape(-1))

    def vector(self, name, *shape):
        self.expect(name, *shape)
        return self.file.f32(name)

    def rows(self, name):
        """Rows of a matrix whose size the configuration leaves to the tensor."""
        if name not in self.file:
            raise SafetensorsError(f"the file has no tensor {name}")
        return self.file.shape(name)[0]

    def _raw(self, name, *shape):
        self.expect(name, *shape)
        if self.file.dtype(name) != "BF16":
            raise SafetensorsError(f"{name}: expected BF16, found {self.file.dtype(name)}")
        return self.file.raw(name)

    def expect(self, name, *shape):
        if name not in self.file:
            raise SafetensorsError(f"the file has no tensor {name}")
        if self.file.shape(name) != shape:
            raise SafetensorsError(f"{name}: shape {self.file.shape(name)}, the configuration says {shape}")
