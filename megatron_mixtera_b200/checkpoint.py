"""Reading and writing ``model.safetensors`` files: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
data_offsets), then the data."""
from __future__ import annotations

import json
import struct
from typing import Dict, Tuple

import numpy as np
import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32,
           "I64": torch.int64, "U8": torch.uint8, "I8": torch.int8}


def read_header(path: str) -> Tuple[Dict[str, dict], int]:
    """(entries without the metadata, offset of the data)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
    header.pop("__metadata__", None)
    return header, 8 + n


def tensor_shapes(path: str) -> Dict[str, tuple]:
    return {k: tuple(v["shape"]) for k, v in read_header(path)[0].items()}


def load_safetensors(path: str) -> Dict[str, torch.Tensor]:
    """All tensors of the file, on the host."""
    header, base = read_header(path)
    data = np.fromfile(path, dtype=np.uint8, offset=base)
    out = {}
    for name, e in header.items():
        lo, hi = e["data_offsets"]
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name!r} has unsupported dtype {e['dtype']}")
        out[name] = torch.from_numpy(data[lo:hi].copy()).view(_DTYPES[e["dtype"]]).view(e["shape"])
    return out


def save_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        blob = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
