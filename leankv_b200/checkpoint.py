"""Reading a model folder: ``config.json`` and safetensors weights, without third-party loaders.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
data_offsets) and the data. Files are memory-mapped; tensors are views until they are moved or converted.
"""

from __future__ import annotations

import json
import os
import struct
import warnings

import torch

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool}


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
    size = os.path.getsize(path)
    data = torch.from_file(path, shared=False, size=size, dtype=torch.uint8)
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        dtype = _DTYPES.get(e["dtype"])
        if dtype is None:
            raise ValueError(f"{path}: tensor {name} has unknown dtype {e['dtype']}")
        lo, hi = e["data_offsets"]
        count = 1
        for d in e["shape"]:
            count *= d
        if hi - lo != count * dtype.itemsize or 8 + n + hi > size:
            raise ValueError(f"{path}: tensor {name} does not fit its data range")
        raw = data[8 + n + lo:8 + n + hi]
        if raw.data_ptr() % dtype.itemsize:
            raw = raw.clone()
        with warnings.catch_warnings():
            warnings.simplefilter("ignore")
            out[name] = raw.view(dtype).reshape(e["shape"])
    return out


def read_weights(model_dir: str) -> dict[str, torch.Tensor]:
    """Every tensor of ``model.safetensors``, or of the shards ``model.safetensors.index.json`` lists."""
    single = os.path.join(model_dir, "model.safetensors")
    if os.path.exists(single):
        return read_safetensors(single)
    with open(os.path.join(model_dir, "model.safetensors.index.json")) as f:
        shards = sorted(set(json.load(f)["weight_map"].values()))
    out = {}
    for s in shards:
        out.update(read_safetensors(os.path.join(model_dir, s)))
    return out


class TensorBag:
    """The tensors of a checkpoint, taken by name and expected shape; what is missing or misshapen is an
    error, what is left over a warning."""

    def __init__(self, tensors: dict[str, torch.Tensor]):
        self._t, self._used = tensors, set()

    def take(self, name: str, *shape: int) -> torch.Tensor:
        if name not in self._t:
            raise ValueError(f"checkpoint has no tensor {name}")
        t = self._t[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, expected {shape}")
        self._used.add(name)
        return t

    def shape(self, name: str) -> tuple:
        if name not in self._t:
            raise ValueError(f"checkpoint has no tensor {name}")
        return tuple(self._t[name].shape)

    def finish(self) -> None:
        left = sorted(set(self._t) - self._used)
        if left:
            warnings.warn(f"checkpoint has tensors that no layer uses: {', '.join(left[:8])}")
