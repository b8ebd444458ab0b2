"""Reader of a model directory's ``.safetensors`` files: header parsing and memory-mapped tensors by name.

A file is an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape, data_offsets; the
offsets count from the end of the header) and the raw data.  ``SafetensorsDir.loader()`` adapts the directory to
``models.weights.WeightSource``.
"""
from __future__ import annotations

import json
import mmap
import os
import struct
import warnings
from typing import Callable, Dict, List, Optional, Tuple

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
           "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
           "BOOL": torch.bool, "F8_E4M3": torch.float8_e4m3fn}


def _header(f) -> Tuple[Dict[str, dict], int]:
    size = os.fstat(f.fileno()).st_size
    raw = f.read(8)
    if len(raw) != 8:
        raise ValueError("not a safetensors file: shorter than its length field")
    n = struct.unpack("<Q", raw)[0]
    if n > size - 8:
        raise ValueError("not a safetensors file: the header does not fit the file")
    head = json.loads(f.read(n))
    head.pop("__metadata__", None)
    return head, 8 + n


def _files(path: str) -> List[str]:
    return sorted(os.path.join(path, n) for n in os.listdir(path) if n.endswith(".safetensors"))


def tensor_shapes(path: str) -> Dict[str, Tuple[int, ...]]:
    """name -> shape over all files of the directory (headers only)."""
    out: Dict[str, Tuple[int, ...]] = {}
    for p in _files(path):
        with open(p, "rb") as f:
            out.update({k: tuple(e["shape"]) for k, e in _header(f)[0].items()})
    return out


def checkpoint_shapes(path: str) -> Dict[str, Tuple[int, ...]]:
    """name -> shape of a model directory: its .safetensors files, or converted shards (``ckpt.converter``)."""
    if _files(path):
        return tensor_shapes(path)
    from .converter import ConvertedCheckpoint
    ck = ConvertedCheckpoint(path)
    shapes = {k: tuple(e["shape"]) for k, (_, e) in ck.index.items()}
    ck.close()
    return shapes


def checkpoint_loader(path: str) -> Callable[[str, Tuple[int, ...]], torch.Tensor]:
    """Loader of a model directory in either format."""
    if _files(path):
        return SafetensorsDir(path).loader()
    from .converter import ConvertedCheckpoint
    ck = ConvertedCheckpoint(path)
    inner = ck.loader()

    def load(name, shape):
        if name not in ck:
            raise KeyError(f"the checkpoint has no tensor {name!r}")
        return inner(name, shape)
    return load


class SafetensorsDir:
    def __init__(self, path: str):
        self.index: Dict[str, Tuple[memoryview, dict]] = {}
        for p in _files(path):
            with open(p, "rb") as f:
                head, base = _header(f)
                view = memoryview(mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ))
            for name, e in head.items():
                a, b = e["data_offsets"]
                if not 0 <= a <= b <= len(view) - base:
                    raise ValueError(f"{p}: tensor {name!r} lies outside the file")
                self.index[name] = (view[base + a: base + b], e)
        if not self.index:
            raise FileNotFoundError(f"no .safetensors tensors under {path}")

    def get(self, name: str) -> torch.Tensor:
        buf, e = self.index[name]
        dt = _DTYPES[e["dtype"]]
        if len(buf) == 0:
            return torch.empty(e["shape"], dtype=dt)
        with warnings.catch_warnings():
            warnings.simplefilter("ignore", UserWarning)          # read-only mapping: tensors are never written
            t = torch.frombuffer(buf, dtype=torch.uint8)
        if t.data_ptr() % t.new_empty(0).to(dt).element_size():
            t = t.clone()
        return t.view(dt).view(*e["shape"])

    def loader(self) -> Callable[[str, Tuple[int, ...]], torch.Tensor]:
        """Every tensor the model asks for has to be there: a missing name is an error, not a random weight."""
        def load(name, shape):
            if name not in self.index:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            return self.get(name)
        return load
