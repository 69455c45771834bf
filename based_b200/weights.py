"""Reader of safetensors files: an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape,
data_offsets), then the data.  The file is mapped, not read: a tensor costs I/O when it is copied to its place."""
import json
import mmap
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class SafeTensors:
    """Tensors by name.  ``get`` checks the shape and remembers what was asked for, so that a loader can report
    tensors it did not use."""

    def __init__(self, path: str):
        self._file = open(path, "rb")
        size = os.fstat(self._file.fileno()).st_size
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        self._map = mmap.mmap(self._file.fileno(), 0, access=mmap.ACCESS_COPY)
        n = struct.unpack("<Q", self._map[:8])[0]
        if 8 + n > size:
            raise ValueError(f"{path}: header runs past the end of the file")
        header = json.loads(self._map[8:8 + n])
        self._base = 8 + n
        self._entries = {k: v for k, v in header.items() if k != "__metadata__"}
        for name, e in self._entries.items():
            a, b = e["data_offsets"]
            if not 0 <= a <= b <= size - self._base:
                raise ValueError(f"{path}: {name} runs past the end of the file")
        self.used = set()

    def __contains__(self, name):
        return name in self._entries

    def __iter__(self):
        return iter(self._entries)

    def shape(self, name):
        return tuple(self._entries[name]["shape"])

    def get(self, name: str, shape=None) -> torch.Tensor:
        """A CPU view of the tensor; ``shape`` (None entries match anything) is checked when given."""
        if name not in self._entries:
            raise KeyError(f"missing tensor {name!r}")
        e = self._entries[name]
        have = tuple(e["shape"])
        if shape is not None and (len(shape) != len(have) or any(s is not None and s != h for s, h in zip(shape, have))):
            raise ValueError(f"{name}: shape {have}, expected {tuple(shape)}")
        self.used.add(name)
        dt = _DTYPES[e["dtype"]]
        count = 1
        for s in have:
            count *= s
        if count == 0:
            return torch.empty(have, dtype=dt)
        start = self._base + e["data_offsets"][0]
        size = torch.empty(0, dtype=dt).element_size()
        if e["data_offsets"][1] - e["data_offsets"][0] != count * size:
            raise ValueError(f"{name}: {have} of {e['dtype']} does not fill its bytes")
        if start % size:   # torch.frombuffer wants aligned data
            return torch.frombuffer(bytearray(self._map[start:start + count * size]), dtype=dt).view(have)
        return torch.frombuffer(self._map, dtype=dt, count=count, offset=start).view(have)

    def unused(self):
        return sorted(set(self._entries) - self.used)


class TensorDict:
    """The same interface over a dict of tensors."""

    def __init__(self, tensors):
        self._t, self.used = dict(tensors), set()

    def __contains__(self, name):
        return name in self._t

    def __iter__(self):
        return iter(self._t)

    def shape(self, name):
        return tuple(self._t[name].shape)

    def get(self, name, shape=None):
        if name not in self._t:
            raise KeyError(f"missing tensor {name!r}")
        t = self._t[name]
        if shape is not None and (len(shape) != t.dim() or any(s is not None and s != h for s, h in zip(shape, t.shape))):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        self.used.add(name)
        return t

    def unused(self):
        return sorted(set(self._t) - self.used)
