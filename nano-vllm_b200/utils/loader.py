"""Checkpoint reading: the tensors of every *.safetensors file of a model folder, by name, without a copy in host memory.

File layout: 8-byte little-endian header length, JSON header (name -> dtype, shape, data_offsets), data.
Plays the part of nanovllm/utils/loader.py:12-28; the models' load_full_weights distributes the tensors.
"""
from __future__ import annotations

import glob
import json
import mmap
import os
import struct
from collections.abc import Mapping

import torch

DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32, "I64": torch.int64,
          "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class Checkpoint(Mapping):
    """name -> tensor over the memory-mapped files of a folder (the tensors are read-only views)."""

    def __init__(self, model_dir: str):
        self._where: dict[str, tuple] = {}
        self._maps = []
        paths = sorted(glob.glob(os.path.join(model_dir, "*.safetensors")))
        if not paths:
            raise FileNotFoundError(f"no .safetensors file in {model_dir}")
        for path in paths:
            with open(path, "rb") as f:
                size = os.fstat(f.fileno()).st_size
                data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
            self._maps.append(data)
            (n,) = struct.unpack_from("<Q", data, 0)
            if n > size - 8:
                raise ValueError(f"{path}: truncated header")
            for name, d in json.loads(bytes(data[8:8 + n])).items():
                if name == "__metadata__":
                    continue
                a, b = d["data_offsets"]
                if 8 + n + b > size:
                    raise ValueError(f"{path}: tensor {name} lies outside the file")
                self._where[name] = (data, 8 + n + a, b - a, d["dtype"], d["shape"])

    def __getitem__(self, name: str) -> torch.Tensor:
        data, at, nbytes, dtype, shape = self._where[name]
        if nbytes == 0:
            return torch.empty(shape, dtype=DTYPES[dtype])
        raw = torch.frombuffer(data, dtype=torch.uint8, count=nbytes, offset=at)
        t = DTYPES[dtype]
        if at % t.itemsize:
            raw = raw.clone()
        return raw.view(t).view(shape)

    def __iter__(self):
        return iter(self._where)

    def __len__(self):
        return len(self._where)


def load_exactly(model, weights: Mapping) -> None:
    """Every tensor of a checkpoint into model.load_weight(name, tensor); names and shapes must be exactly those of
    model.weight_shapes()."""
    want = model.weight_shapes()
    missing, extra = sorted(set(want) - set(weights)), sorted(set(weights) - set(want))
    if missing or extra:
        raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, unexpected {extra[:4]}")
    for name in want:
        w = weights[name]
        if tuple(w.shape) != want[name]:
            raise ValueError(f"{name}: shape {tuple(w.shape)}, expected {want[name]}")
        model.load_weight(name, w)
