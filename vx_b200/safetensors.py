"""Reading a .safetensors file: 8 bytes of length (little-endian), that many
bytes of JSON (name -> dtype, shape, data_offsets into what follows), the data."""
import json
import struct

import numpy as np

_NUMPY = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "F64": np.float64,
          "I32": np.int32, "I64": np.int64, "U8": np.uint8}


class SafeTensors:
    """Tensors by name, mapped from the file and read when asked for."""

    def __init__(self, path):
        with open(path, "rb") as f:
            raw = f.read(8)
            if len(raw) < 8:
                raise ValueError("%s is too short for a safetensors file" % path)
            n = struct.unpack("<Q", raw)[0]
            if n > 1 << 30:
                raise ValueError("%s does not begin with a safetensors header" % path)
            self._entries = json.loads(f.read(n))
        self._entries.pop("__metadata__", None)
        self._path, self._base = path, 8 + n
        self._data = np.memmap(path, np.uint8, "r")

    def __contains__(self, name):
        return name in self._entries

    def names(self):
        return list(self._entries)

    def _entry(self, name):
        if name not in self._entries:
            raise ValueError("%s has no tensor %r" % (self._path, name))
        return self._entries[name]

    def shape(self, name):
        return tuple(self._entry(name)["shape"])

    def _array(self, name):
        e = self._entry(name)
        if e["dtype"] not in _NUMPY:
            raise ValueError("tensor %r has the type %s" % (name, e["dtype"]))
        lo, hi = e["data_offsets"]
        raw = self._data[self._base + lo:self._base + hi]
        return e["dtype"], np.frombuffer(raw.tobytes(), _NUMPY[e["dtype"]]).reshape(
            e["shape"])

    def f32(self, name, shape=None):
        """The tensor as f32; ValueError when it does not have `shape`."""
        dtype, a = self._array(name)
        if shape is not None and tuple(a.shape) != tuple(shape):
            raise ValueError("tensor %r is %s, expected %s"
                             % (name, list(a.shape), list(shape)))
        if dtype == "BF16":
            return (a.astype(np.uint32) << 16).view(np.float32)
        return a.astype(np.float32)


def to_bf16(a):
    """f32 values as bf16 bit patterns, rounded to the nearest even one."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)
