"""A safetensors file as zero-copy views of its mapping.

Layout: 8 bytes little-endian header length, that many bytes of JSON (name -> dtype, shape, data_offsets), then the data.
"""
from __future__ import annotations

import json
import math
import mmap
import os

import numpy as np

_NUMPY = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I8": np.int8, "U8": np.uint8, "I32": np.int32, "I64": np.int64}


class SafetensorsError(ValueError):
    pass


class SafetensorsFile:
    """`array(name)` is the tensor in its own shape; bfloat16 comes as uint16 bit patterns."""

    def __init__(self, path: str) -> None:
        self._f = open(path, "rb")
        try:
            size = os.fstat(self._f.fileno()).st_size
            head = self._f.read(8)
            n = int.from_bytes(head, "little")
            if len(head) != 8 or n > size - 8:
                raise SafetensorsError(f"{path}: not a safetensors file")
            try:
                entries = json.loads(self._f.read(n))
            except ValueError as e:
                raise SafetensorsError(f"{path}: header is not JSON") from e
            self.tensors: dict[str, tuple[str, tuple[int, ...], int]] = {}
            for name, t in entries.items():
                if name == "__metadata__":
                    continue
                dtype, shape, (a, b) = t["dtype"], tuple(int(d) for d in t["shape"]), t["data_offsets"]
                if dtype not in _NUMPY:
                    raise SafetensorsError(f"{name}: dtype {dtype} is not supported")
                if not 0 <= a <= b <= size - 8 - n or b - a != math.prod(shape) * np.dtype(_NUMPY[dtype]).itemsize:
                    raise SafetensorsError(f"{name}: data_offsets do not match its shape or the file")
                self.tensors[name] = (dtype, shape, 8 + n + a)
            self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        except BaseException:
            self._f.close()
            raise

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def shape(self, name: str) -> tuple[int, ...]:
        if name not in self.tensors:
            raise SafetensorsError(f"missing tensor {name}")
        return self.tensors[name][1]

    def dtype(self, name: str) -> str:
        return self.tensors[name][0]

    def array(self, name: str) -> np.ndarray:
        shape = self.shape(name)
        dtype, _, offset = self.tensors[name]
        raw = np.frombuffer(self._map, dtype=np.uint8, count=math.prod(shape) * np.dtype(_NUMPY[dtype]).itemsize, offset=offset)
        return raw.view(_NUMPY[dtype]).reshape(shape) if offset % np.dtype(_NUMPY[dtype]).itemsize == 0 else np.frombuffer(raw.tobytes(), _NUMPY[dtype]).reshape(shape)

    def close(self) -> None:
        try:
            self._map.close()
        except BufferError:
            pass      # tensor views are still alive: the mapping goes away with the last of them
        finally:
            self._f.close()

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()


def write(path: str, tensors: dict[str, np.ndarray]) -> None:
    """Writes fp32, int32 and (as uint16 bit patterns) bfloat16 arrays."""
    kinds = {np.dtype(np.uint16): "BF16", np.dtype(np.float32): "F32", np.dtype(np.int32): "I32"}
    header, offset = {}, 0
    for name, a in tensors.items():
        header[name] = {"dtype": kinds[a.dtype], "shape": list(a.shape), "data_offsets": [offset, offset + a.nbytes]}
        offset += a.nbytes
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little"))
        f.write(head)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())
