"""Model folders: config.json and safetensors files.

A safetensors file is an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets) and the data.  Tensors come back as numpy views of the memory-mapped file; BF16 stays in its
bits (uint16), which is how the C ABI takes it, so nothing is converted on the way to the device.
"""
from __future__ import annotations

import json
import os

import numpy as np

_DTYPES = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class CheckpointError(ValueError):
    pass


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(a: np.ndarray) -> np.ndarray:
    """Round to nearest even; bfloat16 bits in uint16."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class Checkpoint:
    """All tensors of a folder's *.safetensors files by name."""

    def __init__(self, folder: str):
        self._tensors: dict[str, np.ndarray] = {}
        files = sorted(f for f in os.listdir(folder) if f.endswith(".safetensors"))
        if not files:
            raise CheckpointError(f"no .safetensors file in {folder}")
        for name in files:
            self._map(os.path.join(folder, name))

    def _map(self, path: str) -> None:
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            n = int.from_bytes(f.read(8), "little")
            if 8 + n > size:
                raise CheckpointError(f"{path}: truncated header")
            header = json.loads(f.read(n))
        data = np.memmap(path, np.uint8, "r", offset=8 + n) if size > 8 + n else np.empty(0, np.uint8)
        for name, h in header.items():
            if name == "__metadata__":
                continue
            dt = _DTYPES.get(h["dtype"])
            if dt is None:
                raise CheckpointError(f"{path}: {name} has dtype {h['dtype']}")
            lo, hi = h["data_offsets"]
            shape = tuple(h["shape"])
            if not 0 <= lo <= hi <= data.size or hi - lo != int(np.prod(shape, dtype=np.int64)) * np.dtype(dt).itemsize:
                raise CheckpointError(f"{path}: {name} lies outside the file")
            self._tensors[name] = np.frombuffer(data[lo:hi].tobytes(), dt).reshape(shape)

    def __contains__(self, name: str) -> bool:
        return name in self._tensors

    def names(self):
        return self._tensors.keys()

    def get(self, name: str, shape=None) -> np.ndarray:
        """The tensor as stored (BF16 as uint16 bits), its shape checked when one is given."""
        if name not in self._tensors:
            raise CheckpointError(f"tensor {name} is missing")
        a = self._tensors[name]
        if shape is not None and a.shape != tuple(shape):
            raise CheckpointError(f"tensor {name} has shape {a.shape}, expected {tuple(shape)}")
        if a.dtype == np.float16:
            a = a.astype(np.float32)
        return a

    def f32(self, name: str, shape=None) -> np.ndarray:
        a = self.get(name, shape)
        return bf16_to_f32(a) if a.dtype == np.uint16 else np.ascontiguousarray(a, np.float32)


def save(folder: str, config: dict, tensors: dict) -> None:
    """Write a folder that Checkpoint reads: float32 arrays, or uint16 arrays holding BF16 bits."""
    os.makedirs(folder, exist_ok=True)
    header, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.ascontiguousarray(a)
        header[name] = {"dtype": "BF16" if a.dtype == np.uint16 else "F32", "shape": list(a.shape),
                        "data_offsets": [at, at + a.nbytes]}
        blobs.append(a.tobytes())
        at += a.nbytes
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head)
        for b in blobs:
            f.write(b)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
