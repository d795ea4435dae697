"""Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets), and the data."""

from __future__ import annotations

import json
import math
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path):
    """{name: CPU tensor}"""
    with open(path, "rb") as f:
        data = bytearray(f.read())
    (n,) = struct.unpack_from("<Q", data, 0)
    header = json.loads(bytes(data[8:8 + n]).decode("utf-8"))
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has type {e['dtype']}")
        dt, (lo, hi), numel = _DTYPES[e["dtype"]], e["data_offsets"], math.prod(e["shape"])
        if hi - lo != numel * dt.itemsize or not 0 <= lo <= hi <= len(data) - 8 - n:
            raise ValueError(f"{path}: tensor {name} does not fit its data")
        raw = torch.frombuffer(data, dtype=torch.uint8, count=hi - lo, offset=8 + n + lo).clone() if hi > lo else torch.empty(0, dtype=torch.uint8)
        out[name] = raw.view(dt).reshape(e["shape"])
    return out


def write_safetensors(path, tensors):
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode("utf-8")
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
