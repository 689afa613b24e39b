"""Reading safetensors files: an 8-byte little-endian header length, the JSON header (name -> dtype,
shape, data_offsets), then the data.  Tensors are views of a private mapping of the file."""
from __future__ import annotations

import json
import mmap
from pathlib import Path

import torch

_DTYPE = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
          "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
          "BOOL": torch.bool}


def read_safetensors(path):
    with open(path, "rb") as f:
        size = int.from_bytes(f.read(8), "little")
        header = json.loads(f.read(size))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        dtype, (lo, hi) = _DTYPE[e["dtype"]], e["data_offsets"]
        n = (hi - lo) // dtype.itemsize
        if n == 0:
            out[name] = torch.empty(e["shape"], dtype=dtype)
            continue
        start = 8 + size + lo
        if start % dtype.itemsize:      # an odd header length: torch wants element-aligned views
            out[name] = torch.frombuffer(bytearray(data[start:8 + size + hi]), dtype=dtype).view(e["shape"])
        else:
            out[name] = torch.frombuffer(data, dtype=dtype, count=n, offset=start).view(e["shape"])
    return out


def read_model_weights(model_dir):
    """All tensors of a folder's *.safetensors files."""
    files = sorted(Path(model_dir).glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"no *.safetensors in {model_dir}")
    out = {}
    for f in files:
        out.update(read_safetensors(f))
    return out
