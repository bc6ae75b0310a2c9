"""Model folders: config.json and model.safetensors (an 8-byte little-endian header length, a JSON header
name -> dtype / shape / data_offsets, then the raw data)."""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np
import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder) -> dict:
    with open(Path(folder) / "config.json") as f:
        return json.load(f)


def read_safetensors(path) -> dict[str, torch.Tensor]:
    """Tensors of one file as CPU tensors over a copy-on-write map of it (nothing is read before it is used)."""
    path = Path(path)
    with open(path, "rb") as f:
        (length,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(length))
    if path.stat().st_size == 8 + length:
        data = torch.empty(0, dtype=torch.uint8)
    else:
        data = torch.from_numpy(np.memmap(path, dtype=np.uint8, mode="c", offset=8 + length))
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        dtype, shape = _DTYPES[entry["dtype"]], entry["shape"]
        raw = data[lo:hi]
        if (lo + 8 + length) % dtype.itemsize or raw.data_ptr() % dtype.itemsize:
            raw = raw.clone()
        tensors[name] = raw.view(dtype).view(shape)
    return tensors


def write_safetensors(path, tensors: dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, tensor in tensors.items():
        blob = tensor.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[tensor.dtype], "shape": list(tensor.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
