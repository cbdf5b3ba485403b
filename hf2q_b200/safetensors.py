"""safetensors container: 8-byte little-endian header length, a JSON table name -> {dtype, shape, data_offsets}, then
the tensors' bytes.  Memory-mapped reader, and a writer for tests and tools."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import torch

_DTYPES = {"F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I32": torch.int32, "I64": torch.int64, "U8": torch.uint8}
_NAMES = {v: k for k, v in _DTYPES.items()}


class SafetensorsFile:
    def __init__(self, path):
        self.path = Path(path)
        self._f = open(self.path, "rb")
        self._mm = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_COPY)
        if len(self._mm) < 8:
            raise ValueError(f"{path}: truncated safetensors file")
        (n,) = struct.unpack_from("<Q", self._mm, 0)
        if 8 + n > len(self._mm):
            raise ValueError(f"{path}: truncated safetensors header")
        self.tensors = {k: v for k, v in json.loads(self._mm[8:8 + n]).items() if k != "__metadata__"}
        self._data = 8 + n
        for name, t in self.tensors.items():
            if t["dtype"] not in _DTYPES:
                raise ValueError(f"{name}: dtype {t['dtype']} is not handled by this reader")
            if self._data + t["data_offsets"][1] > len(self._mm):
                raise ValueError(f"{name}: payload runs past the end of the file")

    def close(self) -> None:
        self._mm.close()
        self._f.close()

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def load_tensor(self, name: str) -> torch.Tensor:
        """A CPU copy of the tensor."""
        if name not in self.tensors:
            raise ValueError(f"{self.path}: no tensor '{name}'")
        t = self.tensors[name]
        lo, hi = t["data_offsets"]
        if hi == lo:
            return torch.empty(t["shape"], dtype=_DTYPES[t["dtype"]])
        flat = torch.frombuffer(bytearray(self._mm[self._data + lo:self._data + hi]), dtype=_DTYPES[t["dtype"]])
        return flat.reshape(t["shape"])


def save(path, tensors: dict) -> None:
    table, payload, off = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().flatten().view(torch.uint8).numpy().tobytes()
        table[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        payload.append(raw)
        off += len(raw)
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(payload))
