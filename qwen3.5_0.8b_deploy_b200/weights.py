"""Reading model folders: config.json and model.safetensors (8-byte little-endian header length, JSON header, data)."""
from __future__ import annotations

import json
import mmap
import os
import struct

import numpy as np

_TYPES = {"BF16": np.uint16, "F32": np.float32, "F16": np.float16, "I32": np.int32, "I64": np.int64, "I8": np.int8, "U8": np.uint8}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path: str) -> dict[str, np.ndarray]:
    """Name -> array over a read-only mapping of the file; bf16 tensors come as uint16 bits."""
    with open(path, "rb") as f:
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
    (n,) = struct.unpack("<Q", data[:8])
    out = {}
    for name, e in json.loads(data[8:8 + n]).items():
        if name == "__metadata__":
            continue
        dt = np.dtype(_TYPES[e["dtype"]])
        lo, hi = e["data_offsets"]
        count = int(np.prod(e["shape"], dtype=np.int64))
        if (hi - lo) != count * dt.itemsize:
            raise ValueError(f"{path}: tensor {name} holds {hi - lo} bytes, its shape needs {count * dt.itemsize}")
        out[name] = np.frombuffer(data, dt, count, 8 + n + lo).reshape(e["shape"])
    return out


def bf16_bits(a: np.ndarray) -> np.ndarray:
    """float32 -> bf16 bits (round to nearest even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)
