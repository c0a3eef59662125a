"""Where a model's tensors come from: a safetensors file, a dict in memory, or a seed.

A source is called with a tensor name and the shape the model wants, and returns the tensor on the model's device in
the model's dtype.  The file format is read here directly: an 8-byte little-endian length, that many bytes of JSON
(name -> dtype, shape, data_offsets), then the data.
"""
import hashlib
import json
import math
import os
import struct

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool}


class Scope:
    """A source under a name prefix."""

    def __init__(self, source, prefix):
        self.source, self.prefix = source, prefix

    def __call__(self, name, shape):
        return self.source(self.prefix + name, shape)

    def shape(self, name, default):
        return self.source.shape(self.prefix + name, default)

    def scoped(self, prefix):
        return Scope(self.source, self.prefix + prefix)


class WeightSource:
    def __init__(self, dtype, device):
        self.dtype, self.device = dtype, torch.device(device)
        self.used = set()

    def _raw(self, name, shape):
        raise NotImplementedError

    def __call__(self, name, shape):
        t = self._raw(name, tuple(shape))
        if tuple(t.shape) != tuple(shape):
            raise ValueError(f"tensor '{name}' has shape {tuple(t.shape)}, the configuration wants {tuple(shape)}")
        self.used.add(name)
        return t.to(device=self.device, dtype=self.dtype if t.is_floating_point() else t.dtype).contiguous()

    def shape(self, name, default):
        """Shape of a tensor that fixes a size by itself; `default` where the source has no tensors of its own."""
        return tuple(default)

    def scoped(self, prefix):
        return Scope(self, prefix)

    def check_all_used(self):
        """Nothing by default; a file or dict reports tensors that no part of the model asked for."""


class DictWeights(WeightSource):
    def __init__(self, tensors, dtype, device):
        super().__init__(dtype, device)
        self.tensors = tensors

    def _raw(self, name, shape):
        if name not in self.tensors:
            raise KeyError(f"no tensor named '{name}'")
        return self.tensors[name]

    def shape(self, name, default):
        if name not in self.tensors:
            raise KeyError(f"no tensor named '{name}'")
        return tuple(self.tensors[name].shape)

    def check_all_used(self):
        left = sorted(set(self.tensors) - self.used)
        if left:
            raise ValueError(f"{len(left)} tensors belong to no part of the model, e.g. '{left[0]}'")


class SafetensorsWeights(DictWeights):
    """One file, memory-mapped; a tensor is copied when it is asked for."""

    def __init__(self, path, dtype, device):
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) < 8:
                raise ValueError(f"{path}: not a safetensors file")
            n = struct.unpack("<Q", head)[0]
            if n > size - 8:
                raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
            index = json.loads(f.read(n))
        index.pop("__metadata__", None)
        data = torch.from_file(path, shared=False, size=size, dtype=torch.uint8)[8 + n:]
        tensors = {}
        for name, e in index.items():
            a, b = e["data_offsets"]
            dt, shape = _DTYPES[e["dtype"]], tuple(e["shape"])
            if not 0 <= a <= b <= data.numel() or b - a != math.prod(shape) * dt.itemsize:
                raise ValueError(f"{path}: tensor '{name}' has bad offsets")
            raw = data[a:b]
            if raw.data_ptr() % dt.itemsize:
                raw = raw.clone()
            tensors[name] = raw.view(dt).reshape(shape)
        super().__init__(tensors, dtype, device)


class RandomWeights(WeightSource):
    """Seeded weights drawn on the device: matrices N(0, 1 / in), vectors around `vectors[suffix]` (mean, spread)."""

    def __init__(self, seed, dtype, device, vectors=None):
        super().__init__(dtype, device)
        self.seed, self.vectors = seed, vectors or {}

    def _raw(self, name, shape):
        key = int.from_bytes(hashlib.blake2b(f"{self.seed}/{name}".encode(), digest_size=6).digest(), "little")
        g = torch.Generator(device=self.device).manual_seed(key)
        t = torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
        if len(shape) > 1:
            return t * shape[-1] ** -0.5
        mean, spread = next((v for s, v in self.vectors.items() if name.endswith(s)), (0.0, 0.1))
        return mean + spread * t
