"""Reader and writer of safetensors files: an 8-byte little-endian header length, the JSON header (name -> dtype, shape,
data_offsets) and the raw little-endian data.  The file is memory-mapped; a tensor is copied when it is asked for."""
from __future__ import annotations

import json
import mmap

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}
NAMES = {v: k for k, v in DTYPES.items()}


class SafetensorsFile:
    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            n = int.from_bytes(f.read(8), "little")
            header = json.loads(f.read(n))
            f.seek(0, 2)
            size = f.tell()
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        self._base = 8 + n
        header.pop("__metadata__", None)
        self._entries = header
        for name, e in header.items():
            a, b = e["data_offsets"]
            count = 1
            for s in e["shape"]:
                count *= s
            if e["dtype"] not in DTYPES:
                raise ValueError(f"{path}: tensor {name} has the unknown dtype {e['dtype']}")
            if not (0 <= a <= b <= size - self._base) or b - a != count * DTYPES[e["dtype"]].itemsize:
                raise ValueError(f"{path}: the data range of tensor {name} does not fit its shape")

    def keys(self):
        return self._entries.keys()

    def __contains__(self, name: str) -> bool:
        return name in self._entries

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self._entries[name]["shape"])

    def __getitem__(self, name: str) -> torch.Tensor:
        if name not in self._entries:
            raise KeyError(f"{self.path} has no tensor {name}")
        e = self._entries[name]
        a, b = e["data_offsets"]
        if a == b:
            return torch.empty(e["shape"], dtype=DTYPES[e["dtype"]])
        buf = bytearray(self._map[self._base + a:self._base + b])
        return torch.frombuffer(buf, dtype=DTYPES[e["dtype"]]).reshape(e["shape"])


def save(path: str, tensors: dict[str, torch.Tensor]):
    header, at = {}, 0
    for name, t in tensors.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + n]}
        at += n
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little"))
        f.write(head)
        for t in tensors.values():
            f.write(t.detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes())
