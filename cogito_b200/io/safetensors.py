"""Reader and writer of safetensors files: an 8-byte little-endian header length, a JSON header
``name -> {dtype, shape, data_offsets}``, then the data.  Tensors are views of a memory map until they are
moved, so a loader can take them to the device one at a time."""
from __future__ import annotations

import json
import mmap
import os
import struct

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64, "I32": torch.int32,
          "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
NAMES = {v: k for k, v in DTYPES.items()}


def load_safetensors(path: str) -> dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        size = os.fstat(f.fileno()).st_size
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)       # private pages: torch wants a writable buffer
    (n,) = struct.unpack_from("<Q", buf, 0)
    if 8 + n > size:
        raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
    header = json.loads(bytes(buf[8:8 + n]))
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in DTYPES:
            raise ValueError(f"{path}: tensor {name} has unsupported type {e['dtype']}")
        dt, shape, (lo, hi) = DTYPES[e["dtype"]], e["shape"], e["data_offsets"]
        count = 1
        for s in shape:
            count *= s
        if hi - lo != count * dt.itemsize or lo < 0 or 8 + n + hi > size:
            raise ValueError(f"{path}: tensor {name} does not fit its place")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dt)
            continue
        if (8 + n + lo) % dt.itemsize == 0:
            t = torch.frombuffer(buf, dtype=dt, count=count, offset=8 + n + lo)
        else:
            t = torch.frombuffer(bytearray(buf[8 + n + lo:8 + n + hi]), dtype=dt)
        out[name] = t.view(shape)
    return out


def save_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> int:
    header, blobs, off = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    tmp = path + ".tmp"
    with open(tmp, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
    os.replace(tmp, path)
    return 8 + len(head) + off
