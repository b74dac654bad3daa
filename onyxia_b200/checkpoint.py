"""Model folders: ``config.json`` beside ``model.safetensors``.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name → dtype, shape, data_offsets) and
the data. Tensors are views of the mapped file; nothing is read before it is used.
"""
from __future__ import annotations

import json
import os

import numpy as np

from . import ir
from .ir import HostTensor

# bf16 has no numpy type: its bit patterns travel as uint16
_DTYPES = {"BF16": np.uint16, "F16": np.float16, "F32": np.float32, "F64": np.float64, "I32": np.int32, "I64": np.int64,
           "U8": np.uint8, "I8": np.int8, "BOOL": np.bool_}


def widen(a: np.ndarray, dtype: str) -> np.ndarray:
    """The values as f32."""
    if dtype == "BF16":
        return (a.astype(np.uint32) << 16).view(np.float32)
    return a.astype(np.float32)


class Weights:
    """Named tensors; ``array`` gives the stored form, the other two what modules hold."""

    def __init__(self, tensors: dict):
        self._t = tensors  # name → (safetensors dtype name, array)

    @staticmethod
    def from_f32(arrays: dict) -> "Weights":
        return Weights({k: ("F32", np.asarray(v, dtype=np.float32)) for k, v in arrays.items()})

    @staticmethod
    def from_bf16(arrays: dict) -> "Weights":
        """uint16 arrays of bf16 bit patterns."""
        return Weights({k: ("BF16", v) for k, v in arrays.items()})

    def __contains__(self, name: str) -> bool:
        return name in self._t

    def names(self) -> list:
        return list(self._t)

    def shape(self, name: str) -> tuple:
        return tuple(self._get(name)[1].shape)

    def _get(self, name: str):
        if name not in self._t:
            raise KeyError(f"the checkpoint has no tensor '{name}'")
        return self._t[name]

    def f32(self, name: str) -> np.ndarray:
        dtype, a = self._get(name)
        return widen(a, dtype)

    def bf16_bits(self, name: str) -> np.ndarray:
        dtype, a = self._get(name)
        if dtype == "BF16":
            return a
        return HostTensor.bf16(widen(a, dtype)).data.view(np.uint16).reshape(a.shape)

    def stored(self, name: str, dtype: int) -> np.ndarray:
        """The tensor as a module of activation type `dtype` holds it (bf16 as bit patterns)."""
        return self.bf16_bits(name) if dtype == ir.BF16 else self.f32(name)


def host_tensor(a: np.ndarray, dtype: int) -> HostTensor:
    return HostTensor.bf16(a) if dtype == ir.BF16 else HostTensor.from_numpy(a)


def read_safetensors(path: str) -> Weights:
    with open(path, "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        size = os.fstat(f.fileno()).st_size
        if n > size - 8:
            raise ValueError(f"{path}: not a safetensors file")
        header = json.loads(f.read(n))
    data = np.memmap(path, dtype=np.uint8, mode="r") if size > 8 + n else np.zeros(8 + n, np.uint8)
    out = {}
    for name, d in header.items():
        if name == "__metadata__":
            continue
        if d["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor '{name}' has unsupported dtype {d['dtype']}")
        lo, hi = d["data_offsets"]
        np_dt = np.dtype(_DTYPES[d["dtype"]])
        count = int(np.prod(d["shape"], dtype=np.int64))
        if hi - lo != count * np_dt.itemsize or 8 + n + hi > size:
            raise ValueError(f"{path}: tensor '{name}' does not fit its data")
        raw = data[8 + n + lo:8 + n + hi]
        a = np.frombuffer(raw.tobytes(), dtype=np_dt) if (8 + n + lo) % np_dt.itemsize else raw.view(np_dt)
        out[name] = (d["dtype"], a.reshape(d["shape"]))
    return Weights(out)


def write_safetensors(path: str, weights: Weights) -> None:
    header, at = {}, 0
    for name in weights.names():
        dtype, a = weights._get(name)
        header[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little"))
        f.write(text)
        for name in weights.names():
            f.write(np.ascontiguousarray(weights._get(name)[1]).tobytes())


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)
