"""Reader and writer of the safetensors container: an 8-byte little-endian header length, a JSON header
(name -> dtype, shape, data_offsets), then the tensors' bytes.  Reading maps the file; nothing is copied until a
tensor is moved or converted."""
from __future__ import annotations

import json
import mmap
import os
import struct
import warnings
from typing import Dict

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64, "I32": torch.int32,
           "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool, "F8_E4M3": torch.float8_e4m3fn}
_NAMES = {v: k for k, v in _DTYPES.items()}


def load_file(path: str) -> Dict[str, torch.Tensor]:
    """Tensors of ``path`` by name, as views of the mapped file (treat them as read-only)."""
    size = os.path.getsize(path)
    with open(path, "rb") as f:
        mapped = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
    if size < 8:
        raise ValueError(f"{path}: not a safetensors file")
    (header_len,) = struct.unpack("<Q", mapped[:8])
    if header_len > size - 8:
        raise ValueError(f"{path}: header length {header_len} exceeds the file")
    header = json.loads(mapped[8:8 + header_len])
    base, out = 8 + header_len, {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name!r} has unknown type {entry['dtype']!r}")
        dtype, shape = _DTYPES[entry["dtype"]], [int(d) for d in entry["shape"]]
        begin, end = entry["data_offsets"]
        numel = 1
        for d in shape:
            numel *= d
        if not 0 <= begin <= end <= size - base or end - begin != numel * dtype.itemsize:
            raise ValueError(f"{path}: tensor {name!r} has offsets that do not fit its shape or the file")
        if numel == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        with warnings.catch_warnings():
            warnings.simplefilter("ignore")   # the mapping is read-only
            out[name] = torch.frombuffer(mapped, dtype=torch.uint8, count=end - begin, offset=base + begin)
        if (base + begin) % dtype.itemsize:
            out[name] = out[name].clone()
        out[name] = out[name].view(dtype).reshape(shape)
    return out


def save_file(tensors: Dict[str, torch.Tensor], path: str) -> None:
    header, offset, blobs = {}, 0, []
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        blob = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [offset, offset + len(blob)]}
        offset += len(blob)
        blobs.append(blob)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for blob in blobs:
            f.write(blob)
