"""Model folders: ``config.json`` and ``model.safetensors``.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and the
data.  Tensors are returned as CPU torch tensors that share one read of the file.
"""
from __future__ import annotations

import json
import pathlib
import struct
from typing import Dict

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder) -> dict:
    with open(pathlib.Path(folder) / "config.json", encoding="utf-8") as f:
        return json.load(f)


def read_safetensors(path) -> Dict[str, torch.Tensor]:
    size = pathlib.Path(path).stat().st_size
    with open(path, "rb") as f:
        head = f.read(8)
        n = struct.unpack("<Q", head)[0] if len(head) == 8 else -1
        if n < 0 or 8 + n > size:
            raise ValueError(f"{path} is not a safetensors file")
        header = json.loads(f.read(n))
        data = bytearray(f.read())
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise ValueError(f"{name}: unsupported dtype {info['dtype']}")
        dtype, shape, (lo, hi) = _DTYPES[info["dtype"]], list(info["shape"]), info["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if not 0 <= lo <= hi <= len(data) or hi - lo != count * dtype.itemsize:
            raise ValueError(f"{name}: data_offsets do not fit its shape or the file")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif lo % dtype.itemsize == 0:
            out[name] = torch.frombuffer(data, dtype=dtype, count=count, offset=lo).reshape(shape)
        else:
            out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=dtype).reshape(shape)
    return out


def write_safetensors(path, tensors: Dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for raw in blobs:
            f.write(raw)


def load_folder(folder) -> Dict[str, torch.Tensor]:
    return read_safetensors(pathlib.Path(folder) / "model.safetensors")
