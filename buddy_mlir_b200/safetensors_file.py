"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header
{name: {dtype, shape, data_offsets}}, the data."""
import json

import numpy as np

_DTYPES = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "I32": np.int32, "I8": np.int8}


def read(path):
    """{name: (dtype string, array)}; BF16 arrays hold the 16-bit patterns.  The arrays are views
    of the mapped file."""
    raw = np.memmap(path, dtype=np.uint8, mode="r")
    n = int.from_bytes(raw[:8].tobytes(), "little")
    if n <= 0 or 8 + n > raw.size:
        raise ValueError(f"{path}: not a safetensors file")
    header = json.loads(raw[8:8 + n].tobytes())
    out = {}
    for name, t in header.items():
        if name == "__metadata__":
            continue
        if t["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has unsupported type {t['dtype']}")
        dt = np.dtype(_DTYPES[t["dtype"]])
        lo, hi = t["data_offsets"]
        count = int(np.prod(t["shape"], dtype=np.int64))
        if hi - lo != count * dt.itemsize or 8 + n + hi > raw.size:
            raise ValueError(f"{path}: tensor {name} does not fit the file")
        a = np.frombuffer(raw, dtype=np.uint8, count=hi - lo, offset=8 + n + lo)
        if (a.ctypes.data % dt.itemsize) != 0:
            a = a.copy()
        out[name] = (t["dtype"], a.view(dt).reshape(t["shape"]))
    return out
