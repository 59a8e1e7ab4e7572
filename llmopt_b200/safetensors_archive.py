"""Reader of safetensors checkpoints: an 8-byte little-endian index length, the JSON index
(name -> dtype, shape, data_offsets) and the payloads.  The counterpart of ``weight_archive`` for
models that are not compiled packages; the same ``Tensor`` records, errors and lookups.

``array`` hands a tensor out as numpy memory mapped from the file; bfloat16 comes as its uint16 bit
pattern (numpy has no such type), see ``as_float32`` and ``as_bfloat16_bits``."""

from __future__ import annotations

import json
import os
import struct
from typing import Dict, Iterator, Mapping

import numpy as np

from .weight_archive import ArchiveError, Tensor

# safetensors dtype -> numpy dtype of the payload
DTYPES = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "F64": np.float64, "I64": np.int64, "I32": np.int32,
          "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.uint8}


def as_float32(array: np.ndarray) -> np.ndarray:
    """fp32 values of an array as ``Archive.array`` hands it out (uint16: bfloat16 bits)."""
    if array.dtype == np.uint16:
        return (array.astype(np.uint32) << 16).view(np.float32)
    return np.ascontiguousarray(array, np.float32)


def as_bfloat16_bits(array: np.ndarray) -> np.ndarray:
    """bfloat16 bit pattern of an array, rounded to nearest even where it is wider."""
    if array.dtype == np.uint16:
        return array
    bits = np.ascontiguousarray(array, np.float32).view(np.uint32)
    return ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16).astype(np.uint16)


class Archive(Mapping):
    """The index of one file; a mapping from tensor name to its array."""

    def __init__(self, path: str):
        self.path = path
        self.file_size = os.path.getsize(path)
        with open(path, "rb") as source:
            prefix = source.read(8)
            if len(prefix) < 8:
                raise ArchiveError("safetensors file is shorter than its prefix")
            index_bytes = struct.unpack("<Q", prefix)[0]
            if index_bytes > self.file_size - 8:
                raise ArchiveError("safetensors index exceeds the file")
            try:
                header = json.loads(source.read(index_bytes))
            except ValueError as error:
                raise ArchiveError(f"safetensors index is not JSON: {error}") from None
        self.data_start = 8 + index_bytes
        self.index: Dict[str, Tensor] = {}
        for name, entry in header.items():
            if name == "__metadata__":
                continue
            if entry["dtype"] not in DTYPES:
                raise ArchiveError(f"safetensors tensor {name} has unknown dtype {entry['dtype']}")
            begin, end = entry["data_offsets"]
            shape = tuple(int(v) for v in entry["shape"])
            elements = 1
            for dimension in shape:
                elements *= dimension
            if begin < 0 or end > self.file_size - self.data_start or begin > end:
                raise ArchiveError(f"safetensors tensor {name} exceeds the file")
            if end - begin != elements * np.dtype(DTYPES[entry["dtype"]]).itemsize:
                raise ArchiveError(f"safetensors tensor {name} byte length disagrees with its dtype and shape")
            self.index[name] = Tensor(name, entry["dtype"], shape, self.data_start + begin, end - begin)
        self._map = np.memmap(path, np.uint8, "r") if self.file_size else np.empty(0, np.uint8)

    def find(self, name: str):
        return self.index.get(name)

    def read(self, name: str) -> bytes:
        tensor = self.index[name]
        return self._map[tensor.offset:tensor.offset + tensor.byte_length].tobytes()

    def array(self, name: str) -> np.ndarray:
        tensor = self.index[name]
        raw = np.array(self._map[tensor.offset:tensor.offset + tensor.byte_length])  # own, aligned memory
        return raw.view(DTYPES[tensor.dtype]).reshape(tensor.shape)

    def __getitem__(self, name: str) -> np.ndarray:
        if name not in self.index:
            raise KeyError(name)
        return self.array(name)

    def __iter__(self) -> Iterator[str]:
        return iter(self.index)

    def __len__(self) -> int:
        return len(self.index)
