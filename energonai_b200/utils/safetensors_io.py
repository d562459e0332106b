"""Reader of the safetensors file format: 8 bytes little-endian header length, a JSON header (name ->
dtype, shape, data_offsets relative to the end of the header), the data.  The file is mapped, so
only what is copied out is read."""
import json
import mmap
import struct

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def load_safetensors(path):
    """{name: CPU tensor}; the tensors share the (private) mapping of the file."""
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", head)[0]
        raw = f.read(n)
        if len(raw) != n:
            raise ValueError(f"{path}: truncated header")
        header = json.loads(raw)
        mapped = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    data = memoryview(mapped)[8 + n:]
    out = {}
    for name, d in header.items():
        if name == "__metadata__":
            continue
        if d["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: {name} has unknown dtype {d['dtype']}")
        dtype = _DTYPES[d["dtype"]]
        lo, hi = d["data_offsets"]
        count = 1
        for s in d["shape"]:
            count *= s
        if hi - lo != count * dtype.itemsize or hi > len(data):
            raise ValueError(f"{path}: {name} does not fit the file")
        if count == 0:
            out[name] = torch.empty(d["shape"], dtype=dtype)
            continue
        piece = data[lo:hi]
        if (8 + n + lo) % dtype.itemsize:
            piece = bytearray(piece)             # a misaligned tensor is copied
        out[name] = torch.frombuffer(piece, dtype=dtype).reshape(d["shape"])
    return out
