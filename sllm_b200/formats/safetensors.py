"""Tensors of a safetensors file by name (header checks are those of the quantised-checkpoint reader)."""
from __future__ import annotations

import torch

from .quantized_model import QuantizedModelError, read_safetensors_header

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "I32": torch.int32, "I64": torch.int64,
           "U8": torch.uint8, "I8": torch.int8, "F64": torch.float64}


class SafetensorsError(RuntimeError):
    pass


class SafetensorsFile:
    """``with SafetensorsFile(path) as f: t = f.tensor(name)`` - reads one tensor at a time into host memory."""

    def __init__(self, path: str):
        self.path = path
        try:
            self.entries, self._start = read_safetensors_header(path)
        except QuantizedModelError as exc:
            raise SafetensorsError(str(exc)) from None
        self._f = open(path, "rb")

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def close(self) -> None:
        self._f.close()

    def names(self) -> list:
        return list(self.entries)

    def tensor(self, name: str) -> torch.Tensor:
        e = self.entries.get(name)
        if e is None:
            raise SafetensorsError(f"{name}: tensor is absent")
        if e.dtype not in _DTYPES:
            raise SafetensorsError(f"{name}: unsupported dtype {e.dtype}")
        self._f.seek(self._start + e.begin)
        raw = bytearray(self._f.read(e.end - e.begin))
        if len(raw) != e.end - e.begin:
            raise SafetensorsError(f"{name}: truncated file")
        if not raw:
            return torch.empty(e.shape, dtype=_DTYPES[e.dtype])
        return torch.frombuffer(raw, dtype=_DTYPES[e.dtype]).view(e.shape)
