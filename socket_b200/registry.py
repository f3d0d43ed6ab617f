"""Model registry: the architecture named in a folder's config.json decides which decoder is built.

A model folder holds `config.json` (with the key `architecture`) and `model.safetensors`.
"""
from __future__ import annotations

import json
import os
from typing import Dict, Mapping, Optional, Tuple

import numpy as np
import torch
from torch import Tensor

from .decoder import Decoder

SAFETENSOR_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64,
                     "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
                     "BOOL": torch.bool}


# ---------------------------------------------------------------------------------- checkpoints
def read_safetensors(path: str) -> Dict[str, Tensor]:
    """Tensors of a .safetensors file as views of its mapped pages: an 8-byte little-endian length, that
    many bytes of JSON (name -> dtype, shape, data_offsets), then the data."""
    size = os.path.getsize(path)
    with open(path, "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        if n > size - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        header = json.loads(f.read(n))
    data = np.memmap(path, dtype=np.uint8, mode="c", offset=8 + n) if size > 8 + n else np.zeros(0, np.uint8)
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        dt = SAFETENSOR_DTYPES[e["dtype"]]
        count = int(np.prod(e["shape"], dtype=np.int64))
        if not 0 <= a <= b <= data.size or b - a != count * dt.itemsize:
            raise ValueError(f"{path}: {name} does not fit the file")
        raw = data[a:b]
        if raw.ctypes.data % dt.itemsize:
            raw = raw.copy()
        out[name] = torch.from_numpy(raw).view(dt).view(e["shape"]) if count else torch.empty(e["shape"], dtype=dt)
    return out


def write_safetensors(path: str, tensors: Mapping[str, Tensor]) -> None:
    names = {v: k for k, v in SAFETENSOR_DTYPES.items()}
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.detach().cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for raw in blobs:
            f.write(raw)


# ---------------------------------------------------------------------------------- architectures
def _radapel(config: Mapping, shapes: Optional[Mapping[str, Tuple[int, ...]]]) -> Decoder:
    from .radapel import Radapel, RadapelConfig
    return Radapel(RadapelConfig.from_dict(config, shapes))


def _timalorn(config: Mapping, shapes) -> Decoder:
    from .timalorn import Timalorn, TimalornConfig
    return Timalorn(TimalornConfig.from_dict(config))


def _transformer(config: Mapping, shapes) -> Decoder:
    from .model import ModelArgs, Transformer
    return Transformer(ModelArgs(**{k: v for k, v in config.items() if k != "architecture"}))


ARCHITECTURES = {
    "Radapel": (_radapel, ("blocks",)),
    "Timalorn": (_timalorn, ("blocks",)),
    "Transformer": (_transformer, ("step",)),
}


def _architecture(config: Mapping):
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name]


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def libraries_of(config: Mapping) -> Tuple[str, ...]:
    """The CUDA libraries (`build.py`) the architecture's kernels live in."""
    return _architecture(config)[1]


def build_model(config: Mapping, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None,
                dtype: torch.dtype = torch.bfloat16, device="cuda") -> Decoder:
    """The architecture's decoder with empty weights."""
    old = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        with torch.device(device):
            return _architecture(config)[0](config, shapes)
    finally:
        torch.set_default_dtype(old)


def load_model(folder: str, dtype: torch.dtype = torch.bfloat16, device="cuda") -> Decoder:
    """The decoder of a model folder with its weights."""
    tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
    model = build_model(read_config(folder), {k: tuple(v.shape) for k, v in tensors.items()}, dtype, device)
    model.load_tensors(tensors)
    return model
