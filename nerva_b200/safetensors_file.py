"""Safetensors files as byte ranges: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data.  Tensors are not read here: a FileTensor names
the range, and the library streams it to the device through its pinned staging buffer."""
from __future__ import annotations

import json
import struct
from dataclasses import dataclass

import numpy as np

_ELEMENT_BYTES = {"BF16": 2, "F16": 2, "F32": 4, "I32": 4}


@dataclass(frozen=True)
class FileTensor:
    path: bytes
    offset: int     # from the start of the file
    dtype: str
    shape: tuple

    @property
    def size(self) -> int:
        return int(np.prod(self.shape, dtype=np.int64))

    def read(self) -> np.ndarray:
        """The raw elements (16-bit types as uint16)."""
        kind = {"BF16": np.uint16, "F16": np.uint16, "F32": np.float32, "I32": np.int32}[self.dtype]
        return np.fromfile(self.path.decode(), dtype=kind, count=self.size, offset=self.offset).reshape(self.shape)


def open_tensors(path: str) -> dict:
    """name -> FileTensor of one file, with every range checked against the shape and the file's size."""
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        (length,) = struct.unpack("<Q", head)
        f.seek(0, 2)
        end = f.tell()
        if 8 + length > end:
            raise ValueError(f"{path}: header longer than the file")
        f.seek(8)
        header = json.loads(f.read(length))
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        begin, stop = entry["data_offsets"]
        tensor = FileTensor(path.encode(), 8 + length + begin, entry["dtype"], tuple(entry["shape"]))
        width = _ELEMENT_BYTES.get(tensor.dtype)
        if width is None:
            raise ValueError(f"{path}: {name} has the unsupported type {tensor.dtype}")
        if stop - begin != tensor.size * width or begin < 0 or 8 + length + stop > end:
            raise ValueError(f"{path}: {name} has a range that does not fit its shape or the file")
        out[name] = tensor
    return out


def write_tensors(path: str, tensors: dict) -> None:
    """Writes bf16 tensors (uint16 arrays of their bits)."""
    header, at = {}, 0
    for name, t in tensors.items():
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + t.size * 2]}
        at += t.size * 2
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for t in tensors.values():
            f.write(np.ascontiguousarray(t, dtype=np.uint16).tobytes())
