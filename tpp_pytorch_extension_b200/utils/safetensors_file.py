"""Reader of safetensors files (an 8-byte little-endian length, that many bytes of JSON with dtype, shape and byte range per
tensor, then the data) into torch tensors over one memory map."""
import json
import mmap
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64, "I32": torch.int32,
           "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def load(path):
    """name -> CPU tensor. The tensors are views of the mapped file (copy-on-write: the file is never changed)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out = {}
    for name, t in header.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        dt = _DTYPES[t["dtype"]]
        count = 1
        for d in t["shape"]:
            count *= d
        if hi - lo != count * dt.itemsize or 8 + n + hi > len(buf):
            raise ValueError(f"{path}: the byte range of '{name}' does not fit its shape")
        if count == 0:
            out[name] = torch.empty(t["shape"], dtype=dt)
            continue
        if (8 + n + lo) % dt.itemsize == 0:
            v = torch.frombuffer(buf, dtype=dt, count=count, offset=8 + n + lo)
        else:  # an offset the type cannot be viewed at
            v = torch.frombuffer(bytearray(buf[8 + n + lo:8 + n + hi]), dtype=dt)
        out[name] = v.view(t["shape"])
    return out


def save(path, tensors):
    """Write name -> tensor in the same format (contiguous, in the given order)."""
    names = {v: k for k, v in _DTYPES.items()}
    header, pos, blobs = {}, 0, []
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        data = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [pos, pos + len(data)]}
        pos += len(data)
        blobs.append(data)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)
