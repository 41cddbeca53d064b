"""Reader of safetensors files.  Their header is a u64 size and a JSON table that gives every
tensor's element type, shape and byte range in the payload behind it."""
from __future__ import annotations

import json
import mmap
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "I32": torch.int32, "I64": torch.int64,
           "I8": torch.int8, "U8": torch.uint8}


class CheckpointError(ValueError):
    pass


def read_safetensors(path: str) -> dict:
    """name -> CPU tensor.  The tensors are views of one private mapping of the file."""
    with open(path, "rb") as f:
        size = f.seek(0, 2)
        f.seek(0)
        head = f.read(8)
        if len(head) < 8:
            raise CheckpointError(f"{path} is too short for a safetensors header")
        n = struct.unpack("<Q", head)[0]
        if n > size - 8:
            raise CheckpointError(f"{path}: header of {n} bytes in a file of {size}")
        table = json.loads(f.read(n))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out = {}
    for name, t in table.items():
        if name == "__metadata__":
            continue
        if t["dtype"] not in _DTYPES:
            raise CheckpointError(f"{name}: unsupported element type {t['dtype']}")
        dtype, shape = _DTYPES[t["dtype"]], list(t["shape"])
        lo, hi = t["data_offsets"]
        count = 1
        for s in shape:
            count *= s
        if hi - lo != count * dtype.itemsize or 8 + n + hi > size:
            raise CheckpointError(f"{name}: {hi - lo} bytes at {lo} do not hold {shape} of {t['dtype']}")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        out[name] = torch.frombuffer(data, dtype=torch.uint8, count=hi - lo, offset=8 + n + lo).clone().view(dtype).view(shape)
    return out
