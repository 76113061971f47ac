"""Model folders: ``config.json`` beside ``model.safetensors``, and the registry of the
architectures that can be opened from one."""
from __future__ import annotations

import json
import os
import struct
from dataclasses import dataclass
from typing import Callable

import numpy as np

# safetensors dtype -> the numpy type its bytes are viewed as (bfloat16 stays as its bit patterns)
_DTYPES = {"BF16": "<u2", "F16": "<f2", "F32": "<f4", "I32": "<i4", "I64": "<i8", "U8": "u1"}


class CheckpointError(ValueError):
    """A model folder that does not describe a model of its architecture."""


def read_safetensors(path: str) -> dict:
    """name -> (safetensors dtype, array view into the mapped file)."""
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise CheckpointError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", head)[0]
        index = json.loads(f.read(n))
    data = np.memmap(path, np.uint8, mode="r", offset=8 + n) if os.path.getsize(path) > 8 + n else np.zeros(0, np.uint8)
    out = {}
    for name, t in index.items():
        if name == "__metadata__":
            continue
        if t["dtype"] not in _DTYPES:
            raise CheckpointError(f"{path}: tensor {name} has dtype {t['dtype']}")
        lo, hi = t["data_offsets"]
        dt = np.dtype(_DTYPES[t["dtype"]])
        if hi - lo != dt.itemsize * int(np.prod(t["shape"], dtype=np.int64)) or hi > data.size:
            raise CheckpointError(f"{path}: tensor {name} does not fit its shape or the file")
        out[name] = (t["dtype"], np.ascontiguousarray(data[lo:hi]).view(dt).reshape(t["shape"]))
    return out


def write_safetensors(path: str, tensors: dict) -> None:
    """tensors: name -> (safetensors dtype, array)."""
    index, off = {}, 0
    for name, (dtype, a) in tensors.items():
        index[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [off, off + a.nbytes]}
        off += a.nbytes
    head = json.dumps(index).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for _, a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(a) -> np.ndarray:
    """Bit patterns of the nearest bfloat16 values (ties to even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


class TensorFile:
    """The tensors of one model, checked by name, type and shape as they are taken."""

    def __init__(self, tensors: dict):
        self._t = tensors

    def shape(self, name: str) -> tuple:
        if name not in self._t:
            raise CheckpointError(f"tensor {name} is missing")
        return tuple(self._t[name][1].shape)

    def bf16(self, name: str, *shape: int) -> np.ndarray:
        if name not in self._t:
            raise CheckpointError(f"tensor {name} is missing")
        dtype, a = self._t[name]
        if dtype != "BF16" or a.shape != shape:
            raise CheckpointError(f"tensor {name}: expected BF16 {list(shape)}, found {dtype} {list(a.shape)}")
        return a

    def f32(self, name: str, *shape: int) -> np.ndarray:
        return bf16_to_f32(self.bf16(name, *shape))


@dataclass(frozen=True)
class Architecture:
    """parse: config dict -> configuration; decoder: (ctx, configuration, TensorFile, options) -> Decoder;
    write_package: (path, configuration, TensorFile, options), a ``.smeltpkg`` directory."""
    parse: Callable
    decoder: Callable
    write_package: Callable


_ARCHITECTURES: dict[str, Architecture] = {}


def register(name: str, arch: Architecture) -> None:
    _ARCHITECTURES[name] = arch


def architectures() -> list[str]:
    from . import kesedra, pesedra  # noqa: F401  (they register themselves)

    return sorted(_ARCHITECTURES)


def architecture(config: dict) -> Architecture:
    name = config.get("architecture")
    if name not in architectures():
        raise CheckpointError(f"architecture {name!r} is not one of {architectures()}")
    return _ARCHITECTURES[name]


def read_model(folder: str):
    """(architecture, configuration, tensors) of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    arch = architecture(config)
    return arch, arch.parse(config), TensorFile(read_safetensors(os.path.join(folder, "model.safetensors")))


def open_model(ctx, folder: str, **options):
    """A decoder of the architecture the folder's ``config.json`` names.  Options: ``precision``
    ("bfloat16" or "float32"), ``capacity`` (positions; 0 = all the model has), ``max_chunk``."""
    arch, config, tensors = read_model(folder)
    return arch.decoder(ctx, config, tensors, **options)


def convert(folder: str, path: str, **options) -> None:
    """Writes a model folder as a ``.smeltpkg`` directory; options as in ``open_model``."""
    arch, config, tensors = read_model(folder)
    arch.write_package(path, config, tensors, **options)
