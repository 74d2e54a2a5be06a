"""WeightProvider over a checkpoint folder: config.json and *.safetensors files (8-byte little-endian header length, that
many bytes of JSON {name: {dtype, shape, data_offsets}}, then the data)."""
from __future__ import annotations

import glob
import json
import os
import struct

import numpy as np

from .bundle import GpuBundleError, WeightTensor

# numpy has no bf16: those tensors stay as their 16-bit patterns, WeightTensor.dtype says what they are
_ST_DTYPES = {"BF16": (np.uint16, "bfloat16"), "F16": (np.float16, "float16"), "F32": (np.float32, "float32"), "I32": (np.int32, "int32"),
              "I64": (np.int64, "int64"), "U8": (np.uint8, "uint8"), "I8": (np.int8, "int8")}


class CheckpointProvider:
    def __init__(self, path: str):
        from .architectures import config_from_json
        cpath = os.path.join(path, "config.json")
        if not os.path.exists(cpath):
            raise GpuBundleError(f"not a checkpoint folder (no config.json): {path}")
        with open(cpath) as fh:
            try:
                self._config = config_from_json(json.load(fh))
            except json.JSONDecodeError as e:
                raise GpuBundleError(f"config.json: {e}") from e
        self._entries = {}
        for f in sorted(glob.glob(os.path.join(path, "*.safetensors"))):
            self._index(f)
        if not self._entries:
            raise GpuBundleError(f"no tensors (*.safetensors) in {path}")

    def _index(self, file: str) -> None:
        size = os.path.getsize(file)
        with open(file, "rb") as fh:
            head = fh.read(8)
            n = struct.unpack("<Q", head)[0] if len(head) == 8 else size
            if 8 + n > size:
                raise GpuBundleError(f"{file}: truncated header")
            try:
                header = json.loads(fh.read(n))
            except ValueError as e:
                raise GpuBundleError(f"{file}: {e}") from e
        for name, e in header.items():
            if name == "__metadata__":
                continue
            a, b = e["data_offsets"]
            if e["dtype"] not in _ST_DTYPES:
                raise GpuBundleError(f"{name}: unsupported dtype {e['dtype']}")
            dt = np.dtype(_ST_DTYPES[e["dtype"]][0])
            if not 0 <= a <= b <= size - 8 - n or b - a != int(np.prod(e["shape"], dtype=np.int64)) * dt.itemsize:
                raise GpuBundleError(f"{name}: data range does not fit shape {e['shape']} or the file")
            self._entries[name] = (file, 8 + n + a, e["dtype"], tuple(e["shape"]))

    def config(self):
        return self._config

    def tensor_names(self):
        return list(self._entries)

    def has_tensor(self, name: str) -> bool:
        return name in self._entries

    def tensor(self, name: str) -> WeightTensor:
        if name not in self._entries:
            raise GpuBundleError(f"tensor not found: {name}")
        file, off, st, shape = self._entries[name]
        dt, label = _ST_DTYPES[st]
        data = np.fromfile(file, dtype=dt, count=int(np.prod(shape, dtype=np.int64)), offset=off)
        return WeightTensor(data.reshape(shape), shape, label)
