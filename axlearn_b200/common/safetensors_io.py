"""Reading and writing safetensors files.

The format: an 8-byte little-endian header length, a JSON object ``name -> {dtype, shape, data_offsets}``
(offsets relative to the end of the header; an optional ``__metadata__`` entry), then the raw row-major
data.  Tensors are views of one private memory map, so a file is paged in as its tensors are copied to
where they are used.
"""

from __future__ import annotations

import json
import mmap
from typing import Mapping, Optional

import torch

_DTYPES = {
    "BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I8": torch.int8,
    "U8": torch.uint8, "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "BOOL": torch.bool,
}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_safetensors(path: str) -> dict:
    """``{name: tensor}`` on the CPU."""
    with open(path, "rb") as f:
        size = int.from_bytes(f.read(8), "little")
        header = json.loads(f.read(size))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    base, out = 8 + size, {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: {name} has unsupported dtype {entry['dtype']}")
        dtype, shape = _DTYPES[entry["dtype"]], tuple(entry["shape"])
        lo, hi = entry["data_offsets"]
        item = torch.empty((), dtype=dtype).element_size()
        count = 1
        for n in shape:
            count *= n
        if lo < 0 or hi - lo != count * item or base + hi > len(data):
            raise ValueError(f"{path}: {name} has offsets {lo}..{hi} for shape {shape} of {entry['dtype']}")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif (base + lo) % item:
            out[name] = torch.frombuffer(bytearray(data[base + lo:base + hi]), dtype=dtype).reshape(shape)
        else:
            out[name] = torch.frombuffer(data, dtype=dtype, count=count, offset=base + lo).reshape(shape)
    return out


def write_safetensors(path: str, tensors: Mapping[str, torch.Tensor], metadata: Optional[dict] = None) -> None:
    header, blobs, at = {}, [], 0
    if metadata:
        header["__metadata__"] = metadata
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for raw in blobs:
            f.write(raw)


class TreeLoader:
    """Fills a model's parameter tree from a checkpoint's tensors.

    ``tree`` starts as zeros: matrices in ``dtype``, parameters declared fp32 in fp32.  Every tensor is taken
    with its expected shape; ``finish`` refuses tensors that no part of the model took."""

    def __init__(self, model, tensors, *, dtype):
        self._tensors, self._used = tensors, set()

        def build(node):
            if isinstance(node, dict):
                return {name: build(child) for name, child in node.items()}
            return torch.zeros(tuple(node.shape), dtype=torch.float32 if node.dtype == torch.float32 else dtype)

        self.tree = build(model.create_parameter_specs_recursively())

    def take(self, name: str, shape) -> torch.Tensor:
        t = self._tensors[name]
        if tuple(t.shape) != tuple(shape):
            raise ValueError(f"{name} has shape {tuple(t.shape)}, expected {tuple(shape)}")
        self._used.add(name)
        return t

    @staticmethod
    def put(dst: torch.Tensor, src: torch.Tensor, row: int = 0) -> None:
        """``src`` into the top left corner of ``dst`` from ``row`` on (stored sizes may be larger)."""
        dst[row:row + src.shape[0], :src.shape[1]] = src.to(dst.dtype)

    def fill(self, dst: torch.Tensor, name: str, shape, row: int = 0) -> None:
        self.put(dst, self.take(name, shape), row)

    def copy(self, dst: torch.Tensor, name: str, shape) -> None:
        dst.copy_(self.take(name, shape))

    def finish(self, device=None) -> dict:
        unused = set(self._tensors) - self._used
        if unused:
            raise ValueError(f"tensors of no part of the model: {sorted(unused)[:5]} ({len(unused)} in all)")

        def place(node):
            return {k: place(v) if isinstance(v, dict) else v.to(device) for k, v in node.items()}

        return place(self.tree)
