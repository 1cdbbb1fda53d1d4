"""Safetensors checkpoints, byte-compatible with the reference.

The reference saves every tensor as little-endian F32 with no metadata through the Rust
``safetensors`` crate (rumus/src/nn/io.rs:27-81) and refuses anything but F32 on load
(io.rs:102-107).  That crate's serializer orders entries by (dtype alignment descending, name
ascending), writes a compact JSON header ``{"name":{"dtype":..,"shape":..,"data_offsets":..}}``
padded with spaces to a multiple of 8 bytes, preceded by its length as a little-endian u64.
This module reproduces that byte stream directly (no dependency on the Python package; a test
compares both), writes atomically (tmp + rename), and loads F32 files.
"""
from __future__ import annotations

import json
import os
import struct
from collections import OrderedDict
from typing import Dict, Mapping

import numpy as np
import torch


def _to_f32_bytes(t: torch.Tensor) -> bytes:
    a = t.detach().to(device="cpu", dtype=torch.float32).contiguous().numpy()
    if a.dtype.byteorder == ">":  # pragma: no cover - big-endian hosts
        a = a.byteswap()
    return a.tobytes()


def serialize(state: Mapping[str, torch.Tensor]) -> bytes:
    names = sorted(state.keys())  # single dtype (F32): order is by name
    header = OrderedDict()
    blobs = []
    off = 0
    for name in names:
        t = state[name]
        b = _to_f32_bytes(t)
        header[name] = OrderedDict([("dtype", "F32"), ("shape", [int(s) for s in t.shape]),
                                    ("data_offsets", [off, off + len(b)])])
        blobs.append(b)
        off += len(b)
    hjson = json.dumps(header, separators=(",", ":"), ensure_ascii=False).encode("utf-8")
    pad = (8 - len(hjson) % 8) % 8
    hjson += b" " * pad
    return struct.pack("<Q", len(hjson)) + hjson + b"".join(blobs)


def save_safetensors(state: Mapping[str, torch.Tensor], path: str) -> None:
    """Atomic write of ``state`` (any dtype/device; stored as F32)."""
    data = serialize(state)
    tmp = f"{path}.tmp.{os.getpid()}"
    with open(tmp, "wb") as f:
        f.write(data)
        f.flush()
        os.fsync(f.fileno())
    os.replace(tmp, path)


def _entries(path: str):
    """Yields ``(name, dtype string, shape, numpy uint8 view of the data)`` of a safetensors file."""
    raw = np.memmap(path, dtype=np.uint8, mode="r") if os.path.getsize(path) else np.zeros(0, np.uint8)
    if raw.size < 8:
        raise ValueError("safetensors: file too short")
    (n,) = struct.unpack("<Q", raw[:8].tobytes())
    if 8 + n > raw.size:
        raise ValueError("safetensors: header length exceeds file size")
    header = json.loads(raw[8:8 + n].tobytes().decode("utf-8"))
    base = 8 + n
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        if not 0 <= b <= e <= raw.size - base:
            raise ValueError(f"safetensors: data of {name!r} lies outside the file")
        yield name, info["dtype"], [int(s) for s in info["shape"]], raw[base + b:base + e]


def load_safetensors(path: str, device="cpu") -> Dict[str, torch.Tensor]:
    """F32 files, as the reference reads them; any other dtype is an error."""
    out: Dict[str, torch.Tensor] = OrderedDict()
    for name, dtype, shape, data in _entries(path):
        if dtype != "F32":
            raise ValueError(f"safetensors: unsupported dtype {dtype} for {name!r}, expected F32")
        if data.size % 4 != 0:
            raise ValueError(f"safetensors: data length {data.size} of {name!r} is not a multiple of 4")
        arr = np.frombuffer(data.tobytes(), dtype="<f4")
        if int(np.prod(shape)) != arr.size:
            raise ValueError(f"safetensors: shape {shape} does not match data of {name!r}")
        out[name] = torch.from_numpy(arr.copy()).view(*shape).to(device)
    return out


_TORCH_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
                 "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
                 "BOOL": torch.bool}


def load_tensors(path: str) -> Dict[str, torch.Tensor]:
    """Every tensor of a safetensors file with the dtype it is stored in (model checkpoints for serving:
    16-bit weights, integer tables), on the CPU."""
    out: Dict[str, torch.Tensor] = OrderedDict()
    for name, dtype, shape, data in _entries(path):
        if dtype not in _TORCH_DTYPES:
            raise ValueError(f"safetensors: unsupported dtype {dtype} for {name!r}")
        dt = _TORCH_DTYPES[dtype]
        n = 1
        for s in shape:
            n *= s
        if n * torch.empty((), dtype=dt).element_size() != data.size:
            raise ValueError(f"safetensors: shape {shape} does not match data of {name!r}")
        buf = torch.from_numpy(np.array(data)) if n else torch.empty(0, dtype=torch.uint8)
        out[name] = buf.view(dt).view(shape)
    return out


def save_tensors(state: Mapping[str, torch.Tensor], path: str) -> None:
    """Writes every tensor in its own dtype (what ``load_tensors`` reads), larger element sizes first."""
    names = {v: k for k, v in _TORCH_DTYPES.items()}
    order = sorted(state, key=lambda k: (-state[k].element_size(), k))
    header, off = OrderedDict(), 0
    for k in order:
        n = state[k].numel() * state[k].element_size()
        header[k] = {"dtype": names[state[k].dtype], "shape": list(state[k].shape), "data_offsets": [off, off + n]}
        off += n
    hjson = json.dumps(header, separators=(",", ":")).encode("utf-8")
    hjson += b" " * ((8 - len(hjson) % 8) % 8)
    tmp = f"{path}.tmp.{os.getpid()}"
    with open(tmp, "wb") as f:
        f.write(struct.pack("<Q", len(hjson)) + hjson)
        for k in order:
            f.write(state[k].detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes())
    os.replace(tmp, path)


def load_into(module: torch.nn.Module, path: str, strict: bool = False) -> None:
    """Load a checkpoint into ``module``: missing keys are skipped, a shape mismatch is an error
    (rumus/src/nn/parameter.rs:72-100)."""
    sd = load_safetensors(path)
    target = module.state_dict()
    for k, v in sd.items():
        if k in target and tuple(target[k].shape) != tuple(v.shape):
            raise ValueError(f"shape mismatch for {k!r}: checkpoint {tuple(v.shape)} vs model {tuple(target[k].shape)}")
    conv = {k: v.to(target[k].dtype) if k in target else v for k, v in sd.items()}
    module.load_state_dict(conv, strict=strict)
