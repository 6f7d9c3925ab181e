"""Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, byte range),
then the data.  Tensors are views of a private memory map, so only what is used is read."""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, Tuple

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_header(path: str) -> Tuple[Dict[str, dict], int]:
    """``(name -> {dtype, shape, data_offsets}, file offset of the data)``."""
    size = os.path.getsize(path)
    with open(path, "rb") as f:
        head = f.read(8)
        n = struct.unpack("<Q", head)[0] if len(head) == 8 else -1
        if n < 2 or n > size - 8:
            raise ValueError(f"{path}: not a safetensors file")
        table = json.loads(f.read(n))
    table.pop("__metadata__", None)
    return table, 8 + n


def read_tensors(path: str) -> Dict[str, torch.Tensor]:
    table, base = read_header(path)
    size = os.path.getsize(path)
    raw = torch.from_file(path, shared=False, size=size, dtype=torch.uint8)
    out = {}
    for name, e in table.items():
        lo, hi = e["data_offsets"]
        dt = _DTYPES.get(e["dtype"])
        if dt is None:
            raise ValueError(f"{path}: {name} has the unsupported type {e['dtype']}")
        item = torch.empty(0, dtype=dt).element_size()
        if hi - lo != math.prod(e["shape"]) * item or lo < 0 or base + hi > size:
            raise ValueError(f"{path}: {name} does not fit its byte range")
        piece = raw[base + lo:base + hi]
        if (base + lo) % item:
            piece = piece.clone()                                    # a view of the wider type needs an aligned start
        out[name] = piece.view(dt).reshape(e["shape"])
    return out
