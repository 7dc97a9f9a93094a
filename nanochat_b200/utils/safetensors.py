"""
The safetensors file format: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the tensors' bytes.
"""

import json
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


class SafetensorsError(RuntimeError):
    pass


def read_safetensors(path):
    """name -> CPU tensor (views of one buffer)."""
    with open(path, "rb") as f:
        data = bytearray(f.read())
    if len(data) < 8:
        raise SafetensorsError(f"{path}: truncated")
    n = struct.unpack("<Q", data[:8])[0]
    if 8 + n > len(data):
        raise SafetensorsError(f"{path}: the header is longer than the file")
    try:
        header = json.loads(bytes(data[8:8 + n]))
    except ValueError as e:
        raise SafetensorsError(f"{path}: unreadable header: {e}") from e
    buf, out = memoryview(data)[8 + n:], {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise SafetensorsError(f"{path}: {name}: unsupported type {info['dtype']}")
        dtype, (lo, hi) = _DTYPES[info["dtype"]], info["data_offsets"]
        count = 1
        for s in info["shape"]:
            count *= s
        if not 0 <= lo <= hi <= len(buf) or hi - lo != count * dtype.itemsize:
            raise SafetensorsError(f"{path}: {name}: bytes {lo}..{hi} do not hold {info['shape']} of {info['dtype']}")
        raw = torch.frombuffer(buf[lo:hi], dtype=torch.uint8).clone() if count else torch.empty(0, dtype=torch.uint8)
        out[name] = raw.view(dtype).reshape(info["shape"])
    return out


def write_safetensors(path, tensors):
    header, parts, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        parts.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path + ".tmp", "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for p in parts:
            f.write(p)
    os.replace(path + ".tmp", path)
