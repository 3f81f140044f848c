"""Reading and writing safetensors files: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the tensors' bytes."""
from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Dict

import numpy as np
import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8,
           "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_safetensors(path) -> Dict[str, torch.Tensor]:
    """Name -> CPU tensor (views of one memory-mapped, copy-on-write file)."""
    data = np.memmap(path, dtype=np.uint8, mode="c")
    if data.size < 8:
        raise ValueError(f"{path}: not a safetensors file")
    (n,) = struct.unpack("<Q", data[:8].tobytes())
    if 8 + n > data.size:
        raise ValueError(f"{path}: header longer than the file")
    header = json.loads(data[8:8 + n].tobytes())
    body = torch.from_numpy(data[8 + n:])
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: {name} has the unsupported dtype {info['dtype']}")
        dtype = _DTYPES[info["dtype"]]
        begin, end = info["data_offsets"]
        count = 1
        for d in info["shape"]:
            count *= d
        if not 0 <= begin <= end <= body.numel() or end - begin != count * dtype.itemsize:
            raise ValueError(f"{path}: {name} does not fit its place in the file")
        raw = body[begin:end]
        if (8 + n + begin) % dtype.itemsize:
            raw = raw.clone()                       # unaligned in the file
        out[name] = raw.view(dtype).view(info["shape"])
    return out


def write_safetensors(path, tensors: Dict[str, torch.Tensor]) -> None:
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape),
                        "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(Path(path), "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for raw in blobs:
            f.write(raw)
