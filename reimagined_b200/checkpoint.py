"""Checkpoint folders: config.json beside model.safetensors.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets
relative to the end of the JSON) and the data.  Tensors come back as CPU torch tensors over one memory map.
"""
from __future__ import annotations

import json
import mmap
import os
from typing import Dict

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    size = os.path.getsize(path)
    with open(path, "rb") as f:
        head = f.read(8)
        n = int.from_bytes(head, "little")
        if len(head) < 8 or n > size - 8:
            raise ValueError(f"{path}: not a safetensors file")
        entries = json.loads(f.read(n))
        # a private mapping: torch wants writable memory, nothing is written back
        data = mmap.mmap(f.fileno(), 0, flags=mmap.MAP_PRIVATE, prot=mmap.PROT_READ | mmap.PROT_WRITE)
    out: Dict[str, torch.Tensor] = {}
    for name, e in entries.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: {name} has the unknown type {e['dtype']}")
        dtype, shape = _DTYPES[e["dtype"]], tuple(e["shape"])
        begin, end = e["data_offsets"]
        count = 1
        for s in shape:
            count *= s
        if begin < 0 or end - begin != count * dtype.itemsize or 8 + n + end > size:
            raise ValueError(f"{path}: {name} has inconsistent offsets")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        # the JSON may end anywhere: copy out bytes first when the data is not aligned to its type
        raw = torch.frombuffer(data, dtype=torch.uint8, count=end - begin, offset=8 + n + begin)
        out[name] = raw.clone().view(dtype).reshape(shape)
    return out


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    entries, blobs, at = {}, [], 0
    for name, t in tensors.items():
        blob = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        entries[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    head = json.dumps(entries).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head)
        for blob in blobs:
            f.write(blob)
