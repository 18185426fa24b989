"""Reader (and a small writer) of the safetensors container: an 8-byte little-endian header length, that many
bytes of JSON (name -> dtype, shape, data_offsets), then the tensors' bytes."""
from __future__ import annotations

import json
import struct
from typing import Dict, Tuple

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
           "I8": torch.int8, "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "U8": torch.uint8,
           "BOOL": torch.bool}


def read_shapes(path: str) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of the tensors of a file."""
    with open(path, "rb") as f:
        raw = f.read(8)
        if len(raw) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        header = json.loads(f.read(struct.unpack("<Q", raw)[0]))
    return {name: tuple(info["shape"]) for name, info in header.items() if name != "__metadata__"}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        raw = f.read(8)
        if len(raw) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        header = json.loads(f.read(struct.unpack("<Q", raw)[0]))
        data = bytearray(f.read())
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        dtype = _DTYPES[info["dtype"]]
        if not 0 <= a <= b <= len(data):
            raise ValueError(f"{path}: tensor '{name}' lies outside the file")
        t = torch.frombuffer(memoryview(data)[a:b], dtype=torch.uint8) if b > a else torch.empty(0, dtype=torch.uint8)
        out[name] = t.clone().view(dtype).reshape(info["shape"])
    return out


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
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
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)
