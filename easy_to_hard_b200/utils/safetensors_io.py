"""Reading and writing of the safetensors container: an 8-byte little-endian header length, a JSON
header (name -> dtype, shape, data_offsets) and the raw little-endian data."""
from __future__ import annotations

import json
import struct
import warnings
from pathlib import Path
from typing import Dict, Mapping, Union

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32,
           "F64": torch.float64, "I64": torch.int64, "I32": torch.int32, "I16": torch.int16,
           "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def load_safetensors(path: Union[str, Path]) -> Dict[str, torch.Tensor]:
    """All tensors of the file on CPU."""
    with open(path, "rb") as fh:
        head = fh.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", head)[0]
        header = json.loads(fh.read(n))
        body = bytearray(fh.read())
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        dtype, shape = _DTYPES[info["dtype"]], info["shape"]
        lo, hi = info["data_offsets"]
        count = 1
        for s in shape:
            count *= s
        if hi > len(body) or hi - lo != count * dtype.itemsize:
            raise ValueError(f"{path}: tensor {name!r} does not fit the file")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
            continue
        with warnings.catch_warnings():
            warnings.simplefilter("ignore")
            if lo % dtype.itemsize:
                raw = torch.frombuffer(bytearray(body[lo:hi]), dtype=dtype)
            else:
                raw = torch.frombuffer(body, dtype=dtype, count=count, offset=lo)
        out[name] = raw.view(shape)
    return out


def save_safetensors(path: Union[str, Path], tensors: Mapping[str, torch.Tensor]) -> None:
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous()
        data = raw.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[raw.dtype], "shape": list(raw.shape),
                        "data_offsets": [at, at + len(data)]}
        blobs.append(data)
        at += len(data)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as fh:
        fh.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
