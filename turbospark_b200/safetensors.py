"""Reader (and, for tests and tools, writer) of safetensors files.

An 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets), then the data.
bfloat16 tensors are returned as uint16 bit patterns.
"""
import json
import mmap
import struct

import numpy as np

_DTYPES = {"BF16": np.dtype("<u2"), "F32": np.dtype("<f4"), "F16": np.dtype("<f2"), "I32": np.dtype("<i4"), "I64": np.dtype("<i8"),
           "U8": np.dtype("u1")}


class SafeTensors:
    def __init__(self, path):
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        if len(self._map) < 8:
            raise ValueError("%s: not a safetensors file" % path)
        n = struct.unpack("<Q", self._map[:8])[0]
        if n > len(self._map) - 8:
            raise ValueError("%s: header of %d bytes exceeds the file" % (path, n))
        self._index = json.loads(self._map[8:8 + n].decode("utf-8"))
        self._index.pop("__metadata__", None)
        self._base = 8 + n

    def __contains__(self, name):
        return name in self._index

    def names(self):
        return list(self._index)

    def dtype(self, name):
        return self._index[name]["dtype"]

    def shape(self, name):
        return tuple(self._index[name]["shape"])

    def get(self, name):
        """The tensor as a numpy array (a copy: data need not be aligned in the file)."""
        if name not in self._index:
            raise KeyError("tensor %s is missing" % name)
        e = self._index[name]
        if e["dtype"] not in _DTYPES:
            raise ValueError("tensor %s: type %s is not read" % (name, e["dtype"]))
        lo, hi = e["data_offsets"]
        dt = _DTYPES[e["dtype"]]
        count = int(np.prod(e["shape"], dtype=np.int64))
        if hi - lo != count * dt.itemsize or self._base + hi > len(self._map):
            raise ValueError("tensor %s: %d bytes do not hold shape %s" % (name, hi - lo, e["shape"]))
        return np.frombuffer(self._map[self._base + lo:self._base + hi], dtype=dt).reshape(e["shape"])


def write(path, tensors):
    """tensors: name -> array (uint16 arrays are stored as bfloat16 bit patterns)."""
    names = {np.dtype("<u2"): "BF16", np.dtype("<f4"): "F32", np.dtype("<i4"): "I32"}
    index, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        blob = a.tobytes()
        index[name] = {"dtype": names[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    head = json.dumps(index).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for b in blobs:
            f.write(b)
