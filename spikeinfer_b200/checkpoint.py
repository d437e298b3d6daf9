"""Model folders: ``config.json`` plus ``model.safetensors`` (one file, or shards with ``model.safetensors.index.json``).

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and the
data.  Files are mapped, not read: a tensor's bytes are touched when it is copied to the device.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np
import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def load_config(folder) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def read_safetensors(path) -> dict[str, torch.Tensor]:
    path = Path(path)
    size = path.stat().st_size
    with path.open("rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        (n,) = struct.unpack("<Q", head)
        if 8 + n > size:
            raise ValueError(f"{path}: header longer than the file")
        header = json.loads(f.read(n))
    data = np.memmap(path, dtype=np.uint8, mode="c", offset=8 + n) if size > 8 + n else np.zeros(0, dtype=np.uint8)
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has unknown dtype {entry['dtype']}")
        dtype, shape = _DTYPES[entry["dtype"]], entry["shape"]
        lo, hi = entry["data_offsets"]
        count = int(np.prod(shape, dtype=np.int64))
        if not 0 <= lo <= hi <= data.size or hi - lo != count * dtype.itemsize:
            raise ValueError(f"{path}: tensor {name} does not fit its place in the file")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        raw = data[lo:hi]
        if lo + 8 + n & (dtype.itemsize - 1):  # the view below needs an aligned start
            raw = raw.copy()
        out[name] = torch.from_numpy(raw).view(dtype).reshape(shape)
    return out


def load_weights(folder) -> dict[str, torch.Tensor]:
    folder = Path(folder)
    index = folder / "model.safetensors.index.json"
    if index.exists():
        out = {}
        for shard in sorted(set(json.loads(index.read_text())["weight_map"].values())):
            out.update(read_safetensors(folder / shard))
        return out
    return read_safetensors(folder / "model.safetensors")


def save_safetensors(path, tensors: dict[str, torch.Tensor]) -> None:
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with Path(path).open("wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for b in blobs:
            f.write(b)
