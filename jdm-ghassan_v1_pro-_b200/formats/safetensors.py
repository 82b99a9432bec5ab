"""Reader and writer of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the data.  Tensors are views of the mapped file; nothing is copied until a caller asks for it."""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Dict

import numpy as np
import torch

DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
          "I64": torch.int64, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def load(path: str) -> Dict[str, torch.Tensor]:
    """Name -> CPU tensor in the stored type and shape."""
    size = os.path.getsize(path)
    if size < 8:
        raise ValueError(f"{path}: not a safetensors file")
    with open(path, "rb") as f:
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)     # private pages: tensors over them are writable
    (n,) = struct.unpack("<Q", buf[:8])
    if n > size - 8:
        raise ValueError(f"{path}: header length {n} exceeds the file")
    head = json.loads(buf[8:8 + n].decode("utf-8"))
    out = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in DTYPES:
            raise ValueError(f"{path}: tensor '{name}' has unsupported type {e['dtype']}")
        dt = DTYPES[e["dtype"]]
        lo, hi = (int(v) for v in e["data_offsets"])
        shape = tuple(int(v) for v in e["shape"])
        count = int(np.prod(shape, dtype=np.int64)) if shape else 1
        item = torch.empty((), dtype=dt).element_size()
        if lo < 0 or hi > size - 8 - n or hi - lo != count * item:
            raise ValueError(f"{path}: tensor '{name}' lies outside the file or does not fit its shape")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dt)
            continue
        at = 8 + n + lo
        if at % item == 0:
            out[name] = torch.frombuffer(buf, dtype=dt, count=count, offset=at).reshape(shape)
        else:                                                       # a writer that did not pad its header
            raw = torch.frombuffer(bytearray(buf[at:at + count * item]), dtype=torch.uint8)
            out[name] = raw.view(dt).reshape(shape)
    return out


def save(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in DTYPES.items()}
    head, at, blobs = {}, 0, []
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        head[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    text = json.dumps(head).encode("utf-8")
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for b in blobs:
            f.write(b)
