"""Reading and writing safetensors files without a dependency.

The format: an 8-byte little-endian length, that many bytes of JSON mapping each name to its dtype, shape and byte range
(counted from the end of the JSON), then the data.
"""
import json
import os
import struct

import numpy as np

_NP = {"F64": np.float64, "F32": np.float32, "F16": np.float16, "I64": np.int64, "I32": np.int32, "I16": np.int16, "I8": np.int8, "U8": np.uint8,
       "U32": np.uint32, "BOOL": np.bool_}


def bf16_to_f32(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x):
    """Bits of the nearest bfloat16 (ties to even)."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7fff + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def read_safetensors(path):
    """{name: array}; bfloat16 comes widened to float32, every other type as it is stored."""
    with open(path, "rb") as f:
        raw = f.read(8)
        if len(raw) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", raw)[0]
        header = json.loads(f.read(n))
    data = np.memmap(path, np.uint8, "r", offset=8 + n) if os.path.getsize(path) > 8 + n else np.zeros(0, np.uint8)
    out = {}
    for name, t in header.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        b = np.array(data[lo:hi])
        if t["dtype"] == "BF16":
            a = bf16_to_f32(b.view(np.uint16))
        elif t["dtype"] in _NP:
            a = b.view(_NP[t["dtype"]])
        else:
            raise ValueError(f"{path}: {name}: unsupported dtype {t['dtype']}")
        out[name] = a.reshape(t["shape"])
    return out


def write_safetensors(path, tensors):
    """Writes {name: array}; float32 arrays are stored as bfloat16, int32 as they are."""
    header, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        kind, b = ("I32", a.astype("<i4").tobytes()) if a.dtype.kind in "iu" else ("BF16", f32_to_bf16(a).astype("<u2").tobytes())
        header[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)
