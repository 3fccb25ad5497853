"""Reading a model folder: config.json and model.safetensors (an 8-byte little-endian header length, that many bytes of
JSON mapping a name to dtype, shape and data_offsets, then the data)."""

import json
import mmap
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I8": torch.int8, "U8": torch.uint8,
           "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "BOOL": torch.bool}


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path):
    """name -> CPU tensor (copies: the file is not kept open)."""
    out = {}
    with open(path, "rb") as f, mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ) as data:
        (n,) = struct.unpack("<Q", data[:8])
        if 8 + n > len(data):
            raise ValueError(f"{path}: the header runs past the end of the file")
        header = json.loads(data[8:8 + n])
        header.pop("__metadata__", None)
        for name, info in header.items():
            lo, hi = info["data_offsets"]
            dtype = _DTYPES[info["dtype"]]
            count = 1
            for s in info["shape"]:
                count *= s
            if not 0 <= lo <= hi <= len(data) - 8 - n or hi - lo != count * dtype.itemsize:
                raise ValueError(f"{path}: tensor {name} does not fit its data")
            raw = bytearray(data[8 + n + lo:8 + n + hi])
            out[name] = (torch.frombuffer(raw, dtype=dtype) if count else torch.empty(0, dtype=dtype)).reshape(info["shape"])
    return out


def write_safetensors(path, tensors):
    """name -> tensor, written in the same format (tests and converted checkpoints)."""
    names = {v: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        blob = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for blob in blobs:
            f.write(blob)
