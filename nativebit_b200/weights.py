"""Reading checkpoints in the safetensors format: an 8-byte little-endian length, that many bytes of JSON (tensor name
-> dtype, shape, data_offsets), then the data."""
from __future__ import annotations

import json
import os
import struct

import numpy as np
import torch

_TYPES = {"BF16": (np.uint16, torch.bfloat16), "F16": (np.float16, torch.float16), "F32": (np.float32, torch.float32),
          "I32": (np.int32, torch.int32), "I64": (np.int64, torch.int64), "U8": (np.uint8, torch.uint8)}


class Checkpoint:
    """Tensors of one file by name, uploaded on demand.  `unread()` names those nobody asked for."""

    def __init__(self, path: str, device):
        self.path, self.device = path, device
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            head = f.read(8)
            n = struct.unpack("<Q", head)[0] if len(head) == 8 else size
            if 8 + n > size:
                raise ValueError(f"{path} is not a safetensors file")
            self._index = json.loads(f.read(n))
        self._index.pop("__metadata__", None)
        self._base = 8 + n
        self._data = np.memmap(path, dtype=np.uint8, mode="r")
        self._read: set[str] = set()

    def __contains__(self, name: str) -> bool:
        return name in self._index

    def get(self, name: str, shape: tuple | None = None) -> torch.Tensor:
        """The tensor on the device, in its stored dtype; `shape`: the one it must have (None entries: any)."""
        if name not in self._index:
            raise KeyError(f"{self.path} has no tensor {name!r}")
        e = self._index[name]
        if shape is not None and (len(shape) != len(e["shape"]) or any(s is not None and s != g for s, g in zip(shape, e["shape"]))):
            raise ValueError(f"tensor {name!r} has shape {e['shape']}, expected {list(shape)}")
        a, b = e["data_offsets"]
        np_type, t_type = _TYPES[e["dtype"]]
        raw = np.array(self._data[self._base + a:self._base + b]).view(np_type).reshape(e["shape"])
        t = torch.from_numpy(raw)
        self._read.add(name)
        return (t.view(t_type) if t.dtype != t_type else t).to(self.device)

    def unread(self) -> list[str]:
        return sorted(set(self._index) - self._read)


def load_checkpoint(folder: str, device, build, spare: tuple = ()):
    """build(tensor) with tensor(name, shape) -> the weight on the device; every tensor of the file must be asked for, except
    those whose names begin with one of `spare`."""
    ckpt = Checkpoint(f"{folder}/model.safetensors", device)
    model = build(lambda n, s: ckpt.get(n, s))
    unknown = [n for n in ckpt.unread() if not n.startswith(spare)] if spare else ckpt.unread()
    if unknown:
        raise ValueError(f"the checkpoint has tensors that the configuration does not name: {unknown[:8]}")
    torch.cuda.synchronize(device)           # the kernels request weights before they wait for earlier work of the stream
    return model


def write_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> None:
    """The writer's side of the format (exporters, tests)."""
    names = {v[1]: k for k, v in _TYPES.items()}
    index, blobs, at = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().cpu().contiguous()
        raw = (t.view(torch.uint16) if t.dtype == torch.bfloat16 else t).numpy().tobytes()
        index[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    head = json.dumps(index).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
