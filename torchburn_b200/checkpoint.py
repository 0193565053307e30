"""Reading model folders: config.json and safetensors files, without torch.

A safetensors file is an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets) and the raw tensors; it is mapped, not read."""
from __future__ import annotations

import json
import os
import struct
from typing import Dict, List

import numpy as np

# bfloat16 has no numpy type: its raw 16 bits
_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I64": np.int64, "I32": np.int32,
           "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}


class Tensors(Dict[str, np.ndarray]):
    """name -> array; ``stored`` keeps the dtype names of the file."""

    def __init__(self):
        super().__init__()
        self.stored: Dict[str, str] = {}

    def bf16(self, name: str, shape) -> np.ndarray:
        """The raw bfloat16 bits of a tensor of the given shape."""
        if name not in self:
            raise KeyError(f"Required tensor '{name}' is missing from the checkpoint")
        a = self[name]
        if self.stored[name] != "BF16":
            raise ValueError(f"tensor '{name}' is stored as {self.stored[name]}, expected BF16")
        if tuple(a.shape) != tuple(shape):
            raise ValueError(f"tensor '{name}' has shape {tuple(a.shape)}, the configuration asks for {tuple(shape)}")
        return np.ascontiguousarray(a)


def read_safetensors(path: str) -> Tensors:
    size = os.path.getsize(path)
    raw = np.memmap(path, np.uint8, mode="r")
    (n,) = struct.unpack("<Q", raw[:8].tobytes())
    if 8 + n > size:
        raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
    header = json.loads(raw[8:8 + n].tobytes().decode("utf-8"))
    out = Tensors()
    for name, t in header.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        dt = np.dtype(_DTYPES[t["dtype"]])
        if lo < 0 or hi < lo or 8 + n + hi > size or hi - lo != dt.itemsize * int(np.prod(t["shape"], dtype=np.int64)):
            raise ValueError(f"{path}: tensor '{name}' has bad offsets")
        part = raw[8 + n + lo:8 + n + hi]
        if (8 + n + lo) % dt.itemsize:
            part = np.frombuffer(part.tobytes(), np.uint8)
        out[name] = part.view(dt).reshape(t["shape"])
        out.stored[name] = t["dtype"]
    return out


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def weight_files(model_dir: str) -> List[str]:
    """The safetensors files of a model folder, caches of this package left out."""
    names = sorted(f for f in os.listdir(model_dir) if f.endswith(".safetensors") and not f.startswith("torchburn_int4"))
    if not names:
        raise FileNotFoundError(f"{model_dir}: no .safetensors file")
    return [os.path.join(model_dir, f) for f in names]


def read_model_tensors(model_dir: str) -> Tensors:
    out = Tensors()
    for path in weight_files(model_dir):
        part = read_safetensors(path)
        out.update(part)
        out.stored.update(part.stored)
    return out
