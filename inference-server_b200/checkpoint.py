"""Model folders that hold a config.json and one model.safetensors: reading both without a model library.

The file's layout: the header's length in 8 bytes (little-endian), the header as JSON with every tensor's dtype, shape and
data_offsets, then the tensors' bytes.
"""
from __future__ import annotations

import json
import mmap
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I8": torch.int8,
           "U8": torch.uint8, "I16": torch.int16, "I32": torch.int32, "I64": torch.int64}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    """All tensors of the file, on the host (views of one copy-on-write mapping: pages are read as they are used)."""
    with open(path, "rb") as f:
        size = os.fstat(f.fileno()).st_size
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        (n,) = struct.unpack("<Q", head)
        if 8 + n > size:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        header = json.loads(f.read(n))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        dtype, shape = _DTYPES.get(info["dtype"]), info["shape"]
        if dtype is None:
            raise ValueError(f"{path}: {name} has dtype {info['dtype']}")
        lo, hi = info["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if hi - lo != count * torch.empty(0, dtype=dtype).element_size() or 8 + n + hi > size:
            raise ValueError(f"{path}: {name} does not fit its offsets")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif (8 + n + lo) % torch.empty(0, dtype=dtype).element_size():
            out[name] = torch.frombuffer(bytearray(data[8 + n + lo:8 + n + hi]), dtype=dtype).view(shape)
        else:
            out[name] = torch.frombuffer(data, dtype=dtype, count=count, offset=8 + n + lo).view(shape)
    return out


def write_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    header, at, blobs = {}, 0, []
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
