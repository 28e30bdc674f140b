"""Reader of safetensors files: an 8-byte little-endian header length, a JSON header
(name -> dtype, shape, data_offsets) and the data.  Memory-mapped; bf16 comes as raw uint16."""
import json
import struct

import numpy as np

_TYPES = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "I32": np.int32, "I64": np.int64, "U8": np.uint8}


def bf16_to_f32(u16):
    return (u16.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(a):
    """Round to nearest even; the result is the raw uint16."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class SafeTensors:
    def __init__(self, path):
        with open(path, "rb") as f:
            n = struct.unpack("<Q", f.read(8))[0]
            self.header = json.loads(f.read(n))
        self.header.pop("__metadata__", None)
        self._data = np.memmap(path, np.uint8, "r", offset=8 + n)

    def __contains__(self, name):
        return name in self.header

    def names(self):
        return list(self.header)

    def shape(self, name):
        return tuple(self.header[name]["shape"])

    def raw(self, name):
        """The tensor in its stored type (bf16 as uint16)."""
        e = self.header[name]
        a, b = e["data_offsets"]
        return self._data[a:b].view(_TYPES[e["dtype"]]).reshape(e["shape"])

    def f32(self, name):
        a = self.raw(name)
        return bf16_to_f32(a) if self.header[name]["dtype"] == "BF16" else a.astype(np.float32)

    def bf16(self, name):
        a = self.raw(name)
        return a if self.header[name]["dtype"] == "BF16" else f32_to_bf16(a.astype(np.float32))


def save(path, tensors):
    """Write name -> array (uint16 arrays are stored as BF16)."""
    names = {np.dtype(np.float32): "F32", np.dtype(np.uint16): "BF16", np.dtype(np.int32): "I32"}
    head, blobs, at = {}, [], 0
    for k, a in tensors.items():
        a = np.ascontiguousarray(a)
        head[k] = dict(dtype=names[a.dtype], shape=list(a.shape), data_offsets=[at, at + a.nbytes])
        blobs.append(a)
        at += a.nbytes
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for a in blobs:
            f.write(a.tobytes())
