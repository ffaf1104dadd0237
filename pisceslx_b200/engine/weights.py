"""Reader of safetensors checkpoints: an 8-byte little-endian header length, a JSON header ``name -> {dtype, shape,
data_offsets}`` and the raw data.  Files are memory-mapped; tensors are copied out only where they are used."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path
from typing import Any, Dict

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path: str | Path) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    (n,) = struct.unpack("<Q", buf[:8])
    if 8 + n > len(buf):
        raise ValueError(f"{path}: truncated header")
    header: Dict[str, Any] = json.loads(buf[8:8 + n])
    out: Dict[str, torch.Tensor] = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has unsupported dtype {e['dtype']}")
        dt, shape = _DTYPES[e["dtype"]], [int(x) for x in e["shape"]]
        lo, hi = e["data_offsets"]
        count = 1
        for x in shape:
            count *= x
        size = torch.empty(0, dtype=dt).element_size()
        if hi - lo != count * size or 8 + n + hi > len(buf):
            raise ValueError(f"{path}: tensor {name} does not fit its data")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dt)
        else:
            out[name] = torch.frombuffer(buf, dtype=torch.uint8, count=hi - lo, offset=8 + n + lo).clone().view(dt).view(shape)
    return out


def read_folder(directory: str | Path) -> Dict[str, torch.Tensor]:
    """``model.safetensors``, or every shard named by ``model.safetensors.index.json``."""
    d = Path(directory)
    index = d / "model.safetensors.index.json"
    if index.is_file():
        out: Dict[str, torch.Tensor] = {}
        for name in sorted(set(json.loads(index.read_text())["weight_map"].values())):
            out.update(read_safetensors(d / name))
        return out
    return read_safetensors(d / "model.safetensors")
