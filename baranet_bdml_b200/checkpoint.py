"""Reading a model folder: config.json and model.safetensors.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and
the data.  The file is mapped, so a tensor's bytes are read when it is copied to the GPU."""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Dict

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    """name -> CPU tensor over the mapped file (copy-on-write, so writing to one never reaches the file)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in DTYPES:
            raise RuntimeError(f"{path}: tensor {name} has dtype {entry['dtype']}")
        dtype, shape = DTYPES[entry["dtype"]], entry["shape"]
        begin, end = entry["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if end - begin != count * dtype.itemsize or 8 + n + end > len(data):
            raise RuntimeError(f"{path}: tensor {name} does not fit its data")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        out[name] = torch.frombuffer(data, dtype=torch.uint8, count=end - begin, offset=8 + n + begin).clone() \
            .view(dtype).reshape(shape)
    return out


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in DTYPES.items()}
    header, at = {}, 0
    for name, t in tensors.items():
        size = t.numel() * t.element_size()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + size]}
        at += size
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for t in tensors.values():
            f.write(t.detach().cpu().contiguous().view(torch.uint8).numpy().tobytes() if t.dim() else
                    t.detach().cpu().reshape(1).view(torch.uint8).numpy().tobytes())


class Weights:
    """The tensors of a checkpoint, handed out by name; `leftover()` names those that nothing asked for."""

    def __init__(self, tensors: Dict[str, torch.Tensor]):
        self.tensors, self.used = tensors, set()

    def __call__(self, name: str, *shape: int) -> torch.Tensor:
        if name not in self.tensors:
            raise RuntimeError(f"the checkpoint has no tensor {name}")
        t = self.tensors[name]
        if shape and tuple(t.shape) != shape:
            raise RuntimeError(f"tensor {name} has shape {tuple(t.shape)}, expected {shape}")
        self.used.add(name)
        return t

    def leftover(self):
        return sorted(set(self.tensors) - self.used)
