"""Model folders: config.json and model.safetensors (an 8-byte little-endian length, that many bytes of JSON mapping a
tensor's name to dtype, shape and data offsets, then the data)."""
import json
import os
import struct

import numpy as np

_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "I32": np.int32, "I64": np.int64}


class Tensors:
    """Named tensors of a safetensors file, mapped into memory. bf16 data is handed out as its bit patterns (uint16)."""

    def __init__(self, path):
        self.path = path
        self._map = np.memmap(path, np.uint8, "r")
        if self._map.size < 8:
            raise ValueError("%s: shorter than a safetensors header" % path)
        n = struct.unpack("<Q", self._map[:8].tobytes())[0]
        if n > self._map.size - 8:
            raise ValueError("%s: header longer than the file" % path)
        self._head = {k: v for k, v in json.loads(self._map[8:8 + n].tobytes()).items() if k != "__metadata__"}
        self._base = 8 + n

    def __contains__(self, name):
        return name in self._head

    def names(self):
        return list(self._head)

    def shape(self, name):
        return tuple(self._entry(name)["shape"])

    def _entry(self, name):
        if name not in self._head:
            raise KeyError("%s: no tensor %r" % (self.path, name))
        return self._head[name]

    def raw(self, name):
        e = self._entry(name)
        if e["dtype"] not in _DTYPES:
            raise ValueError("%s: tensor %r has dtype %s" % (self.path, name, e["dtype"]))
        a, b = e["data_offsets"]
        if not 0 <= a <= b <= self._map.size - self._base:
            raise ValueError("%s: data of %r lies outside the file" % (self.path, name))
        return np.frombuffer(self._map[self._base + a:self._base + b].tobytes(), _DTYPES[e["dtype"]]).reshape(e["shape"])

    def bf16(self, name, shape=None):
        """Bit patterns of a bf16 tensor, its shape checked."""
        if self._entry(name)["dtype"] != "BF16":
            raise ValueError("%s: tensor %r is %s, expected BF16" % (self.path, name, self._entry(name)["dtype"]))
        a = self.raw(name)
        if shape is not None and a.shape != tuple(shape):
            raise ValueError("%s: tensor %r has shape %s, expected %s" % (self.path, name, a.shape, tuple(shape)))
        return a

    def f32(self, name, shape=None):
        return bf16_to_f32(self.bf16(name, shape))


class ArrayTensors(Tensors):
    """The same interface over arrays in memory: float32 arrays are rounded to bf16, uint16 arrays are bf16 bits."""

    def __init__(self, arrays):
        self.path = "<arrays>"
        self._arr = {k: v if v.dtype == np.uint16 else f32_to_bf16(v) for k, v in arrays.items()}
        self._head = {k: {"dtype": "BF16", "shape": list(v.shape)} for k, v in self._arr.items()}

    def raw(self, name):
        self._entry(name)
        return self._arr[name]


def bf16_to_f32(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(a):
    """bf16 bit patterns, round to nearest even (finite values)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def write_safetensors(path, arrays):
    """Writes bf16 bit patterns (uint16) or float32 arrays (rounded to bf16)."""
    head, pos, parts = {}, 0, []
    for name, a in arrays.items():
        bits = np.ascontiguousarray(a if a.dtype == np.uint16 else f32_to_bf16(a))
        head[name] = {"dtype": "BF16", "shape": list(bits.shape), "data_offsets": [pos, pos + bits.nbytes]}
        pos += bits.nbytes
        parts.append(bits)
    j = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(j)) + j)
        for p in parts:
            f.write(p.tobytes())


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
