"""Model folders: config.json plus weights in safetensors files (8-byte little-endian header length, a JSON header
name -> dtype, shape, data_offsets, then the data)."""
from __future__ import annotations

import json
import mmap
import os

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


class Weights:
    """Named host tensors of a model folder, read through a memory map.  `take` hands a tensor out once and checks its
    shape; `unused` lists what nothing asked for."""

    def __init__(self, tensors: dict[str, torch.Tensor]):
        self.tensors = tensors
        self.taken: set[str] = set()

    @classmethod
    def open(cls, folder: str) -> "Weights":
        tensors: dict[str, torch.Tensor] = {}
        files = sorted(f for f in os.listdir(folder) if f.endswith(".safetensors"))
        if not files:
            raise FileNotFoundError(f"no safetensors file in {folder}")
        for name in files:
            tensors.update(read_safetensors(os.path.join(folder, name)))
        return cls(tensors)

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def take(self, name: str, *shape: int) -> torch.Tensor:
        t = self.tensors.get(name)
        if t is None:
            raise KeyError(f"the checkpoint has no tensor {name!r}")
        if tuple(t.shape) != tuple(shape):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(shape)}")
        self.taken.add(name)
        return t

    def shape(self, name: str, default: tuple[int, ...]) -> tuple[int, ...]:
        """Shape of a tensor whose sizes the configuration does not give (`default` where weights are made up)."""
        if name not in self.tensors:
            raise KeyError(f"the checkpoint has no tensor {name!r}")
        return tuple(self.tensors[name].shape)

    def unused(self) -> list[str]:
        return sorted(set(self.tensors) - self.taken)


class RandomWeights:
    """Stand-in for a checkpoint: matrices ~ N(0, 1 / fan-in), norms near 1, drawn on the device."""

    def __init__(self, device, seed: int = 0):
        self.device, self.g = device, torch.Generator(device=device).manual_seed(seed)

    def take(self, name: str, *shape: int) -> torch.Tensor:
        t = torch.randn(*shape, generator=self.g, device=self.device)
        return (1.0 + 0.1 * t if len(shape) == 1 else t * shape[-1] ** -0.5).to(torch.bfloat16)

    def shape(self, name: str, default: tuple[int, ...]) -> tuple[int, ...]:
        return default


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        m = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)  # private pages: torch wants a writable buffer
    n = int.from_bytes(m[:8], "little")
    if n <= 0 or 8 + n > len(m):
        raise ValueError(f"{path}: not a safetensors file")
    out = {}
    for name, info in json.loads(m[8 : 8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        dtype, shape = DTYPES[info["dtype"]], info["shape"]
        count = 1
        for s in shape:
            count *= s
        if count * dtype.itemsize != hi - lo or 8 + n + hi > len(m):
            raise ValueError(f"{path}: {name} does not fit its place")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif (8 + n + lo) % dtype.itemsize == 0:
            out[name] = torch.frombuffer(m, dtype=dtype, count=count, offset=8 + n + lo).view(shape)
        else:
            out[name] = torch.frombuffer(bytearray(m[8 + n + lo : 8 + n + hi]), dtype=dtype).view(shape)
    return out


def write_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> None:
    names = {v: k for k, v in DTYPES.items()}
    header, at = {}, 0
    for name, t in tensors.items():
        size = t.numel() * t.element_size()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + size]}
        at += size
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for t in tensors.values():
            f.write(t.detach().cpu().contiguous().view(torch.uint8).numpy().tobytes())
