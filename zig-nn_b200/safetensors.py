"""safetensors container: an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the data. Reader (memory-mapped) and writer. Host-only module."""
import json
import struct

import numpy as np

_NUMPY = {"F32": np.float32, "F16": np.float16, "F64": np.float64, "BF16": np.uint16, "I32": np.int32, "I64": np.int64,
          "U8": np.uint8, "I8": np.int8, "BOOL": np.bool_}


class SafetensorsError(Exception):
    pass


def bf16_to_f32(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(a):
    """Round to nearest even; the bits as uint16."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class Tensor:
    """dtype: the file's name of it; data: the values, bf16 as uint16 bits."""

    def __init__(self, dtype, data):
        self.dtype, self.data = dtype, data
        self.shape = data.shape

    def f32(self):
        return bf16_to_f32(self.data).reshape(self.shape) if self.dtype == "BF16" else self.data.astype(np.float32)

    def bf16(self):
        return self.data if self.dtype == "BF16" else f32_to_bf16(self.f32()).reshape(self.shape)


def read(path):
    """name -> Tensor; the arrays are views into the mapped file."""
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise SafetensorsError("%s: too short" % path)
        n = struct.unpack("<Q", head)[0]
        raw = f.read(n)
        if len(raw) != n:
            raise SafetensorsError("%s: header cut off" % path)
    table = json.loads(raw)
    body = np.memmap(path, np.uint8, "r", offset=8 + n) if any(k != "__metadata__" for k in table) else np.empty(0, np.uint8)
    out = {}
    for name, t in table.items():
        if name == "__metadata__":
            continue
        if t["dtype"] not in _NUMPY:
            raise SafetensorsError("%s: dtype %s of %s" % (path, t["dtype"], name))
        dt = np.dtype(_NUMPY[t["dtype"]])
        lo, hi = t["data_offsets"]
        shape = tuple(t["shape"])
        if hi - lo != int(np.prod(shape, dtype=np.int64)) * dt.itemsize or hi > body.size:
            raise SafetensorsError("%s: extent of %s" % (path, name))
        data = body[lo:hi]
        if (8 + n + lo) % dt.itemsize:
            data = data.copy()
        out[name] = Tensor(t["dtype"], data.view(dt).reshape(shape))
    return out


def write(path, tensors):
    """tensors: name -> Tensor."""
    table, at = {}, 0
    for name, t in tensors.items():
        size = t.data.nbytes
        table[name] = {"dtype": t.dtype, "shape": list(t.shape), "data_offsets": [at, at + size]}
        at += size
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for t in tensors.values():
            f.write(np.ascontiguousarray(t.data).tobytes())
