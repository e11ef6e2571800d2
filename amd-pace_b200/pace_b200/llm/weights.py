"""Checkpoint folders: config.json + model.safetensors.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets) and the data; it is mapped, and a tensor is copied only where a model puts it.
"""
import json
import mmap
import os
import struct
from typing import Dict

import torch

_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    """name -> CPU tensor over the mapped file (read-only data: copy before changing a tensor)."""
    with open(path, "rb") as f:
        size = os.fstat(f.fileno()).st_size
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        mm = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    n = struct.unpack("<Q", mm[:8])[0]
    if 8 + n > size:
        raise ValueError(f"{path}: header is longer than the file")
    header = json.loads(mm[8: 8 + n].decode("utf-8"))
    out = {}
    for name, rec in header.items():
        if name == "__metadata__":
            continue
        dtype, shape, (lo, hi) = _DTYPES[rec["dtype"]], rec["shape"], rec["data_offsets"]
        count = 1
        for s in shape:
            count *= s
        if not 0 <= lo <= hi <= size - 8 - n or hi - lo != count * dtype.itemsize:
            raise ValueError(f"{path}: bad extent of tensor {name}")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        if (8 + n + lo) % dtype.itemsize:     # a header of odd length: the data cannot be viewed in place
            raw = torch.frombuffer(bytearray(mm[8 + n + lo: 8 + n + hi]), dtype=torch.uint8)
            out[name] = raw.view(dtype).view(shape)
        else:
            out[name] = torch.frombuffer(mm, dtype=dtype, count=count, offset=8 + n + lo).view(shape)
    return out


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    """The inverse of ``read_safetensors`` (synthetic checkpoints)."""
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, off = {}, [], 0
    for name, t in tensors.items():
        b = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
