"""Reading and writing model folders: config.json and model.safetensors.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and
the tensors' bytes.
"""

import json
import mmap
import os

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
_NAMES = {v: k for k, v in _DTYPES.items()}


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_safetensors(path):
    """name -> CPU tensor (copies: the file is not kept open)."""
    out = {}
    with open(path, "rb") as f:
        size = os.fstat(f.fileno()).st_size
        n = int.from_bytes(f.read(8), "little")
        if n > size - 8:
            raise ValueError(f"{path}: the header is longer than the file")
        header = json.loads(f.read(n))
        with mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ) as mm:
            for name, e in header.items():
                if name == "__metadata__":
                    continue
                lo, hi = e["data_offsets"]
                dtype = _DTYPES.get(e["dtype"])
                if dtype is None:
                    raise ValueError(f"{path}: tensor {name} has unsupported type {e['dtype']}")
                shape = list(e["shape"])
                count = 1
                for s in shape:
                    count *= s
                if hi - lo != count * dtype.itemsize or 8 + n + hi > size:
                    raise ValueError(f"{path}: tensor {name} has a bad extent")
                raw = bytearray(mm[8 + n + lo:8 + n + hi])
                out[name] = (torch.frombuffer(raw, dtype=dtype) if count else torch.empty(0, dtype=dtype)).view(shape)
    return out


def write_safetensors(path, tensors):
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little"))
        f.write(text)
        for raw in blobs:
            f.write(raw)


def write_model(folder, config, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
