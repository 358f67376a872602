"""Reader and writer of safetensors files: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets) and the data.  Only what checkpoints here use; numpy keeps bf16 as uint16 bits."""
from __future__ import annotations

import json
import math
import struct

import numpy as np
import torch

DTYPES = {"BF16": (np.uint16, torch.bfloat16), "F32": (np.float32, torch.float32), "I32": (np.int32, torch.int32)}


class CheckpointError(ValueError):
    pass


class Checkpoint:
    """The tensors of one file, read when asked for."""

    def __init__(self, path: str):
        self.path = path
        try:
            self._data = np.memmap(path, dtype=np.uint8, mode="r")
            length = struct.unpack("<Q", self._data[:8].tobytes())[0]
            header = json.loads(self._data[8:8 + length].tobytes())
        except (OSError, ValueError, struct.error) as error:
            raise CheckpointError(f"{path}: not a safetensors file ({error})") from error
        self._base = 8 + length
        self._entries = {name: entry for name, entry in header.items() if name != "__metadata__"}

    def names(self) -> set[str]:
        return set(self._entries)

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self._entry(name)["shape"])

    def _entry(self, name: str) -> dict:
        if name not in self._entries:
            raise CheckpointError(f"{self.path}: tensor {name} is missing")
        return self._entries[name]

    def tensor(self, name: str, shape: tuple[int, ...] | None = None) -> torch.Tensor:
        """The tensor on the host; `shape`: what it has to be."""
        entry = self._entry(name)
        if entry["dtype"] not in DTYPES:
            raise CheckpointError(f"{self.path}: {name} has unsupported type {entry['dtype']}")
        stored, dtype = DTYPES[entry["dtype"]]
        if shape is not None and tuple(entry["shape"]) != tuple(shape):
            raise CheckpointError(f"{self.path}: {name} has shape {entry['shape']}, expected {list(shape)}")
        begin, end = entry["data_offsets"]
        count = math.prod(entry["shape"])
        if end - begin != count * np.dtype(stored).itemsize or self._base + end > self._data.size:
            raise CheckpointError(f"{self.path}: {name} has inconsistent data offsets")
        values = np.frombuffer(self._data[self._base + begin:self._base + end].tobytes(), dtype=stored).copy()
        tensor = torch.from_numpy(values.view(np.int16) if stored is np.uint16 else values)
        return (tensor.view(dtype) if stored is np.uint16 else tensor).reshape(entry["shape"])


def write(path: str, tensors: dict[str, torch.Tensor]) -> None:
    """Writes bf16 / f32 / i32 host tensors."""
    names = {dtype: name for name, (_, dtype) in DTYPES.items()}
    header, parts, offset = {}, [], 0
    for name, tensor in tensors.items():
        tensor = tensor.detach().cpu().contiguous()
        raw = (tensor.view(torch.int16) if tensor.dtype == torch.bfloat16 else tensor).numpy().tobytes()
        header[name] = {"dtype": names[tensor.dtype], "shape": list(tensor.shape),
                        "data_offsets": [offset, offset + len(raw)]}
        parts.append(raw)
        offset += len(raw)
    text = json.dumps(header).encode()
    with open(path, "wb") as handle:
        handle.write(struct.pack("<Q", len(text)))
        handle.write(text)
        for part in parts:
            handle.write(part)
