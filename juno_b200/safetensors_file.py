"""Model folders: a writer for config.json + model.safetensors and the binding of the library's safetensors reader.

The container is an 8-byte little-endian header length, a JSON object name -> {dtype, shape, data_offsets}, then the data.
Weights are BF16; `to_bf16` rounds FP32 arrays to nearest even.
"""
from __future__ import annotations

import ctypes as C
import json
import os
import struct

import numpy as np

from . import _lib
from ._lib import check

DTYPES = {0: "BF16", 1: "F16", 2: "F32", 3: "I32"}


def to_bf16(a) -> np.ndarray:
    """FP32 -> BF16 bit patterns (uint16), round to nearest even."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(b) -> np.ndarray:
    return (np.asarray(b, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)


def write_safetensors(path, tensors) -> None:
    """tensors: name -> uint16 array (BF16 bit patterns) or float32 array, written in that order."""
    header, off = {}, 0
    for name, a in tensors.items():
        kind = {"uint16": "BF16", "float32": "F32", "int32": "I32"}[a.dtype.name]
        header[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [off, off + a.nbytes]}
        off += a.nbytes
    head = json.dumps(header, separators=(",", ":")).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())


def write_model_folder(path, config: dict, tensors) -> str:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return str(path)


class SafetensorsFile:
    """The library's mapped reader (juno_safetensors_*)."""

    def __init__(self, path):
        self._L = _lib.load()
        h = C.c_void_p()
        check(self._L.juno_safetensors_open(str(path).encode(), C.byref(h)), "juno_safetensors_open")
        self.handle = h

    def close(self) -> None:
        if self.handle:
            check(self._L.juno_safetensors_close(self.handle), "juno_safetensors_close")
            self.handle = None

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def names(self):
        n = C.c_int64()
        check(self._L.juno_safetensors_count(self.handle, C.byref(n)), "juno_safetensors_count")
        buf, out = C.create_string_buffer(512), []
        for i in range(n.value):
            check(self._L.juno_safetensors_name(self.handle, i, buf, 512), "juno_safetensors_name")
            out.append(buf.value.decode())
        return out

    def tensor(self, name: str):
        """(dtype name or None, shape, uint8 view of the mapped bytes; valid until close)."""
        t, nd, nb, dims, data = C.c_int32(), C.c_int32(), C.c_int64(), (C.c_int64 * 8)(), C.c_void_p()
        check(self._L.juno_safetensors_tensor(self.handle, name.encode(), C.byref(t), C.byref(nd), dims, C.byref(data), C.byref(nb)),
              "juno_safetensors_tensor")
        raw = np.ctypeslib.as_array(C.cast(data, C.POINTER(C.c_uint8)), shape=(nb.value,)) if nb.value else np.zeros(0, np.uint8)
        return DTYPES.get(t.value), tuple(dims[i] for i in range(nd.value)), raw
