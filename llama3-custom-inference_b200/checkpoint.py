"""Reading a model folder: config.json and model.safetensors (one file).

A safetensors file is an 8-byte little-endian header length, that many bytes of JSON (tensor name -> dtype, shape and
data_offsets relative to the end of the header; "__metadata__" is not a tensor), then the data.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def read_safetensors(path) -> dict:
    """All tensors of the file, on the CPU."""
    data = bytearray(Path(path).read_bytes())
    header_len = int.from_bytes(data[:8], "little")
    header = json.loads(bytes(data[8:8 + header_len]))
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        dtype, (lo, hi) = DTYPES[entry["dtype"]], entry["data_offsets"]
        count = math.prod(entry["shape"])
        if hi - lo != count * dtype.itemsize or 8 + header_len + hi > len(data):
            raise ValueError(f"{path}: tensor {name} has {hi - lo} bytes for shape {entry['shape']}")
        raw = data[8 + header_len + lo:8 + header_len + hi]   # a copy: data offsets need not be aligned
        t = torch.frombuffer(raw, dtype=dtype) if count else torch.empty(0, dtype=dtype)
        out[name] = t.reshape(entry["shape"])
    return out


def read_weights(folder) -> dict:
    return read_safetensors(Path(folder) / "model.safetensors")
