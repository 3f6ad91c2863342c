"""Safetensors reader: the file is mapped and tensors are handed out as raw views, as gguf.py does for GGUF."""
import json
import math
import mmap
import struct

import numpy as np

from .types import BF16, F16, F32

DTYPES = {"BF16": (BF16, 2), "F16": (F16, 2), "F32": (F32, 4), "I32": (None, 4)}


class SafetensorsError(ValueError):
    pass


class SafetensorsFile:
    """`.tensors`: name -> (shape, ggml type or None for integer tables, offset, bytes)."""

    def __init__(self, path):
        self._f = open(path, "rb")
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        self._buf = memoryview(self._map)
        if len(self._buf) < 8:
            raise SafetensorsError("file is shorter than its header length")
        (n,) = struct.unpack_from("<Q", self._buf, 0)
        if 8 + n > len(self._buf):
            raise SafetensorsError("header runs past the end of the file")
        head = json.loads(bytes(self._buf[8:8 + n]).decode("utf-8"))
        self.tensors = {}
        for name, t in head.items():
            if name == "__metadata__":
                continue
            if t["dtype"] not in DTYPES:
                raise SafetensorsError(f"tensor {name} has unsupported dtype {t['dtype']}")
            kind, size = DTYPES[t["dtype"]]
            a, b = t["data_offsets"]
            count = 1
            for d in t["shape"]:
                count *= d
            if b - a != count * size or 8 + n + b > len(self._buf) or a < 0:
                raise SafetensorsError(f"tensor {name}: {b - a} bytes at {a} do not fit shape {t['shape']}")
            self.tensors[name] = (tuple(t["shape"]), kind, 8 + n + a, b - a)

    def has(self, name):
        return name in self.tensors

    def shape(self, name):
        if name not in self.tensors:
            raise SafetensorsError(f"tensor {name} is missing")
        return self.tensors[name][0]

    def get(self, name):
        """(rows, cols, ggml type, raw bytes): vectors are one row, scalars one number, stacked matrices one tall matrix."""
        shape = self.shape(name)
        _, kind, off, nbytes = self.tensors[name]
        if kind is None:
            raise SafetensorsError(f"tensor {name} is an integer table")
        cols = shape[-1] if shape else 1
        rows = math.prod(shape[:-1])
        return rows, cols, kind, np.frombuffer(self._buf, dtype=np.uint8, count=nbytes, offset=off)

    def close(self):
        self._buf.release()
        self._map.close()
        self._f.close()

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        try:
            self.close()
        except BufferError:  # a view handed out is still alive: the mapping goes with it
            pass
