"""Reader of a .safetensors file: 8 bytes of little-endian length, that much JSON (name -> dtype, shape, byte range of
the data that follows), the data. Tensors are views of the mapped file until they are copied to a device."""
from __future__ import annotations

import json
import mmap
from typing import Dict, List

_DTYPES = {"BF16": ("bfloat16", 2), "F16": ("float16", 2), "F32": ("float32", 4), "I32": ("int32", 4), "I64": ("int64", 8),
           "U8": ("uint8", 1), "I8": ("int8", 1)}


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        size = len(self._map)
        n = int.from_bytes(self._map[:8], "little") if size >= 8 else size
        if size < 8 or n > size - 8:
            raise ValueError(f"{path}: a header of {n} bytes in a file of {size}")
        header = json.loads(self._map[8:8 + n])
        header.pop("__metadata__", None)
        self._start, self._entries = 8 + n, header
        for name, e in header.items():
            lo, hi = e["data_offsets"]
            count = 1
            for d in e["shape"]:
                count *= d
            if e["dtype"] not in _DTYPES:
                raise ValueError(f"{path}: {name} has element type {e['dtype']}")
            if not 0 <= lo <= hi <= size - self._start or hi - lo != count * _DTYPES[e["dtype"]][1]:
                raise ValueError(f"{path}: {name} of shape {e['shape']} in bytes [{lo}, {hi})")

    def names(self) -> List[str]:
        return list(self._entries)

    def __contains__(self, name: str) -> bool:
        return name in self._entries

    def tensor(self, name: str):
        """A CPU tensor of the file's element type (a copy: the file may go away)."""
        import torch
        if name not in self._entries:
            raise KeyError(f"{self.path} has no tensor {name}")
        e = self._entries[name]
        lo, hi = e["data_offsets"]
        dtype = getattr(torch, _DTYPES[e["dtype"]][0])
        if lo == hi:
            return torch.empty(e["shape"], dtype=dtype)
        return torch.frombuffer(bytearray(self._map[self._start + lo:self._start + hi]), dtype=dtype).reshape(e["shape"])


def write_safetensors(path: str, tensors: Dict[str, object]) -> None:
    """Write CPU tensors to a file."""
    import torch
    codes = {v[0]: k for k, v in _DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = t.view(torch.uint8).reshape(-1).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": codes[str(t.dtype).removeprefix("torch.")], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head)
        for b in blobs:
            f.write(b)
