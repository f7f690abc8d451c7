"""Reader of .safetensors files: 8 bytes little-endian header length, a JSON header name -> {dtype, shape, data_offsets},
then the raw little-endian data. Loading parses JSON and views bytes, nothing else."""

import json
import mmap
import struct

import numpy as np
import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I8": torch.int8,
           "I16": torch.int16, "I32": torch.int32, "I64": torch.int64, "U8": torch.uint8, "BOOL": torch.bool}


def load_safetensors(path):
    """-> dict name -> CPU tensor."""
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        (n,) = struct.unpack("<Q", head)
        if n > 1 << 28:
            raise ValueError(f"{path}: header too large")
        meta = json.loads(f.read(n).decode())
        mm = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
    base, out = 8 + n, {}
    for name, t in meta.items():
        if name == "__metadata__":
            continue
        if t["dtype"] not in _DTYPES:
            raise ValueError(f"{name}: unknown dtype {t['dtype']}")
        dtype, shape = _DTYPES[t["dtype"]], [int(s) for s in t["shape"]]
        a, b = (int(v) for v in t["data_offsets"])
        size = int(np.prod(shape, dtype=np.int64)) * torch.empty(0, dtype=dtype).element_size()
        if min(shape, default=0) < 0 or a < 0 or b - a != size or base + b > len(mm):
            raise ValueError(f"{name}: bad extent")
        raw = np.frombuffer(mm, dtype=np.uint8, count=size, offset=base + a).copy()
        out[name] = torch.from_numpy(raw).view(dtype).view(shape) if size else torch.empty(shape, dtype=dtype)
    return out


def save_safetensors(tensors, path):
    """The inverse of `load_safetensors` (contiguous CPU copies, in the order of the dict)."""
    names = {v: k for k, v in _DTYPES.items()}
    meta, parts, off = {}, [], 0
    for k, v in tensors.items():
        v = v.detach().contiguous().cpu()
        raw = v.view(-1).view(torch.uint8).numpy().tobytes() if v.numel() else b""
        meta[k] = {"dtype": names[v.dtype], "shape": list(v.shape), "data_offsets": [off, off + len(raw)]}
        parts.append(raw)
        off += len(raw)
    head = json.dumps(meta).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for raw in parts:
            f.write(raw)
