"""Reading a model folder: ``config.json`` and ``model.safetensors`` (one file, or several ``*.safetensors``).

A safetensors file is an 8-byte little-endian header length, a JSON object of that many bytes (name -> dtype,
shape, data_offsets) and the raw data.  The file is memory-mapped; a tensor is copied out when it is asked for.
"""

from __future__ import annotations

import json
import math
import mmap
import struct
from pathlib import Path

import torch

_DTYPES = {
    "F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
    "F8_E4M3": torch.float8_e4m3fn, "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8,
    "U8": torch.uint8, "BOOL": torch.bool,
}
_NAMES = {dtype: name for name, dtype in _DTYPES.items()}


class CheckpointError(RuntimeError):
    """A model folder lacks something or holds it in another form."""


def load_config(folder: str | Path) -> dict:
    path = Path(folder) / "config.json"
    try:
        config = json.loads(path.read_text())
    except (OSError, ValueError) as error:
        raise CheckpointError(f"cannot read {path}: {error}") from error
    if not isinstance(config, dict):
        raise CheckpointError(f"{path} does not hold a JSON object")
    return config


class SafetensorsFile:
    """Name -> tensor access to one memory-mapped safetensors file."""

    def __init__(self, path: str | Path) -> None:
        self.path = Path(path)
        with open(self.path, "rb") as handle:
            self._map = mmap.mmap(handle.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise CheckpointError(f"{self.path} is too short for a safetensors file")
        (length,) = struct.unpack("<Q", self._map[:8])
        if 8 + length > len(self._map):
            raise CheckpointError(f"{self.path} is shorter than its header says")
        header = json.loads(self._map[8:8 + length])
        header.pop("__metadata__", None)
        self._entries, self._base = header, 8 + length

    def keys(self) -> list[str]:
        return list(self._entries)

    def get(self, name: str) -> torch.Tensor:
        entry = self._entries[name]
        dtype, shape = _DTYPES.get(entry["dtype"]), tuple(int(n) for n in entry["shape"])
        begin, end = (int(n) for n in entry["data_offsets"])
        if dtype is None:
            raise CheckpointError(f"{name} has the unknown dtype {entry['dtype']}")
        if end - begin != math.prod(shape) * dtype.itemsize or not 0 <= begin <= end <= len(self._map) - self._base:
            raise CheckpointError(f"{name}: data offsets do not fit its shape or the file")
        if begin == end:
            return torch.empty(shape, dtype=dtype)
        raw = bytearray(self._map[self._base + begin:self._base + end])
        return torch.frombuffer(raw, dtype=torch.uint8).view(dtype).view(shape)


class Checkpoint:
    """All tensors of a model folder.  ``take`` checks the shape; ``unused`` lists what nobody asked for."""

    def __init__(self, folder: str | Path) -> None:
        files = sorted(Path(folder).glob("*.safetensors"))
        if not files:
            raise CheckpointError(f"no *.safetensors file in {folder}")
        self._where: dict[str, SafetensorsFile] = {}
        for path in files:
            file = SafetensorsFile(path)
            for name in file.keys():
                self._where[name] = file
        self._taken: set[str] = set()

    def take(self, name: str, shape: tuple[int, ...] | None = None) -> torch.Tensor:
        if name not in self._where:
            raise CheckpointError(f"the checkpoint has no tensor {name!r}")
        tensor = self._where[name].get(name)
        if shape is not None and tuple(tensor.shape) != tuple(shape):
            raise CheckpointError(f"{name} has shape {tuple(tensor.shape)}, expected {tuple(shape)}")
        self._taken.add(name)
        return tensor

    def unused(self) -> list[str]:
        return sorted(set(self._where) - self._taken)


def save_safetensors(path: str | Path, tensors: dict[str, torch.Tensor]) -> None:
    """Write ``tensors`` (moved to the CPU) as one safetensors file."""

    header, offset, blobs = {}, 0, []
    for name, tensor in tensors.items():
        data = tensor.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[tensor.dtype], "shape": list(tensor.shape),
                        "data_offsets": [offset, offset + len(data)]}
        offset += len(data)
        blobs.append(data)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as handle:
        handle.write(struct.pack("<Q", len(text)) + text)
        for blob in blobs:
            handle.write(blob)


__all__ = ["Checkpoint", "CheckpointError", "SafetensorsFile", "load_config", "save_safetensors"]
