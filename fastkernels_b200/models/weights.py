"""Weights by name: model.safetensors (one file or an index of several), or random
tensors of given shapes."""
from __future__ import annotations

import json
import mmap
import struct
from pathlib import Path

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32,
           "F64": torch.float64, "I8": torch.int8, "U8": torch.uint8, "I16": torch.int16,
           "I32": torch.int32, "I64": torch.int64, "BOOL": torch.bool}


class TensorSource:
    """Named tensors."""

    def names(self):
        raise NotImplementedError

    def shape(self, name: str) -> tuple:
        raise NotImplementedError

    def get(self, name: str) -> torch.Tensor:
        raise NotImplementedError

    def __contains__(self, name: str) -> bool:
        return name in self.names()


class SafetensorsSource(TensorSource):
    """Tensors of a model folder: an 8-byte little-endian header length, that many
    bytes of JSON (name -> dtype, shape, data_offsets), then the data, per file."""

    def __init__(self, folder):
        folder = Path(folder)
        index = folder / "model.safetensors.index.json"
        if index.exists():
            files = sorted(set(json.loads(index.read_text())["weight_map"].values()))
        else:
            files = ["model.safetensors"]
        self._maps, self._where = [], {}
        for fi, name in enumerate(files):
            with open(folder / name, "rb") as f:
                mm = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
            n = struct.unpack("<Q", mm[:8])[0]
            for key, meta in json.loads(mm[8:8 + n]).items():
                if key != "__metadata__":
                    self._where[key] = (fi, 8 + n, meta)
            self._maps.append(mm)

    def names(self):
        return self._where.keys()

    def shape(self, name):
        return tuple(self._where[name][2]["shape"])

    def get(self, name):
        if name not in self._where:
            raise KeyError(f"the model folder has no tensor '{name}'")
        fi, base, meta = self._where[name]
        a, b = meta["data_offsets"]
        raw = bytearray(self._maps[fi][base + a:base + b])
        t = torch.frombuffer(raw, dtype=_DTYPES[meta["dtype"]]) if b > a else \
            torch.empty(0, dtype=_DTYPES[meta["dtype"]])
        return t.reshape(meta["shape"])


class DictSource(TensorSource):
    """Tensors that are already in memory."""

    def __init__(self, tensors: dict):
        self._t = tensors

    def names(self):
        return self._t.keys()

    def shape(self, name):
        return tuple(self._t[name].shape)

    def get(self, name):
        return torch.as_tensor(self._t[name])


class RandomSource(TensorSource):
    """Tensors drawn on demand: `init(name, shape, generator)` makes one."""

    def __init__(self, shapes: dict, init, seed: int, device):
        self._shapes, self._init = shapes, init
        self._gen = torch.Generator(device=device).manual_seed(seed)

    def names(self):
        return self._shapes.keys()

    def shape(self, name):
        return tuple(self._shapes[name])

    def get(self, name):
        return self._init(name, self._shapes[name], self._gen)


class Packer:
    """Tensors of a source as a model's kernels take them: on the device, matrices in the
    model's type, vectors in fp32, zero-padded where asked."""

    def __init__(self, source: TensorSource, device, dtype, width: int, stride: int):
        self.source, self.device, self.dtype = source, device, dtype
        self.width, self.stride = width, stride      # of the residual rows

    def zeros(self, *shape) -> torch.Tensor:
        return torch.zeros(shape, dtype=self.dtype, device=self.device)

    def matrix(self, name: str) -> torch.Tensor:
        return self.source.get(name).to(device=self.device, dtype=self.dtype)

    def padded(self, w, rows: int, cols: int) -> torch.Tensor:
        if isinstance(w, str):
            w = self.matrix(w)
        out = self.zeros(rows, cols)
        out[:w.shape[0], :w.shape[1]] = w
        return out

    def vector(self, name: str, pad: int | None = None, dtype=torch.float32) -> torch.Tensor:
        v = self.source.get(name).to(device=self.device, dtype=dtype).reshape(-1)
        out = torch.zeros(v.numel() if pad is None else pad, dtype=dtype, device=self.device)
        out[:v.numel()] = v
        return out
