"""Reader and writer of safetensors files: an 8-byte little-endian header length, a JSON header
(name -> dtype, shape, data_offsets) and the tensors' bytes."""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Dict

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "U8": torch.uint8, "I8": torch.int8}
_NAMES = {v: k for k, v in _DTYPES.items()}


def load_file(path: str) -> Dict[str, torch.Tensor]:
    """All tensors of the file, on the host (copies: the file is not kept open)."""
    size = os.path.getsize(path)
    out = {}
    with open(path, "rb") as f:
        if size < 8:
            raise ValueError(f"{path}: too short for a safetensors file")
        with mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ) as m:
            (n,) = struct.unpack("<Q", m[:8])
            if n > size - 8:
                raise ValueError(f"{path}: the header ends past the file")
            header = json.loads(m[8:8 + n])
            for name, h in header.items():
                if name == "__metadata__":
                    continue
                if h["dtype"] not in _DTYPES:
                    raise ValueError(f"{path}: {name} has the unknown type {h['dtype']}")
                dtype = _DTYPES[h["dtype"]]
                a, b = h["data_offsets"]
                count = 1
                for s in h["shape"]:
                    count *= s
                item = torch.empty((), dtype=dtype).element_size()
                if not 0 <= a <= b <= size - 8 - n or b - a != count * item:
                    raise ValueError(f"{path}: {name} does not fit its data range")
                raw = bytearray(m[8 + n + a:8 + n + b])
                t = torch.frombuffer(raw, dtype=dtype) if raw else torch.empty(0, dtype=dtype)
                out[name] = t.reshape(h["shape"])
    return out


def save_file(tensors: Dict[str, torch.Tensor], path: str) -> None:
    header, at = {}, 0
    host = {k: t.detach().cpu().contiguous() for k, t in tensors.items()}
    for name, t in host.items():
        nbytes = t.numel() * t.element_size()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + nbytes]}
        at += nbytes
    blob = json.dumps(header).encode()
    blob += b" " * (-len(blob) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(blob)))
        f.write(blob)
        for t in host.values():
            f.write(t.reshape(-1).view(torch.uint8).numpy().tobytes())
