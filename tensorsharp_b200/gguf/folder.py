"""A model folder (``config.json`` + ``model.safetensors``) behind the interface of :class:`~.reader.GGUFFile`.

A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and
the data.  Tensors are exposed as zero-copy ``uint8`` views of the mapped file with the GGML type of their element, so
the weight loaders of :class:`~..models.base.ModelBase` take a folder as they take a GGUF file.  ``general.architecture``
is the configuration's ``architecture`` in lower case; every other metadata key is looked up in the top level of
config.json, and ``config`` holds the whole document.
"""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Any, Dict

import numpy as np

from .constants import GGMLType
from .reader import GGUFFile, GGUFFormatError, GGUFTensorInfo

CONFIG_NAME = "config.json"
WEIGHTS_NAME = "model.safetensors"

_TYPES = {"BF16": GGMLType.BF16, "F16": GGMLType.F16, "F32": GGMLType.F32, "F64": GGMLType.F64,
          "I8": GGMLType.I8, "I16": GGMLType.I16, "I32": GGMLType.I32, "I64": GGMLType.I64}
_BYTES = {"BF16": 2, "F16": 2, "F32": 4, "F64": 8, "I8": 1, "I16": 2, "I32": 4, "I64": 8}


def is_model_folder(path: str) -> bool:
    return os.path.isdir(path) and os.path.isfile(os.path.join(path, CONFIG_NAME))


def is_checkpoint(path: str) -> bool:
    """Whether ``path`` is something a model can be loaded from: a file, or a model folder."""
    return os.path.isfile(path) or is_model_folder(path)


def checkpoint_bytes(path: str) -> int:
    """Size on disk of a model file, or of the weights of a model folder."""
    return os.path.getsize(os.path.join(path, WEIGHTS_NAME) if os.path.isdir(path) else path)


class ModelFolder(GGUFFile):
    """An open model folder; ``offset`` of a tensor is relative to ``data_offset``, as in a GGUF file."""

    def __init__(self, path: str):
        self.path = path
        with open(os.path.join(path, CONFIG_NAME), "r", encoding="utf-8") as f:
            self.config: Dict[str, Any] = json.load(f)
        self.metadata = {k: v for k, v in self.config.items() if not isinstance(v, (dict, list))}
        self.metadata["general.architecture"] = str(self.config.get("architecture", "")).lower()
        self.metadata_types = {}
        self.tensors: Dict[str, GGUFTensorInfo] = {}
        self.version = 0
        self.alignment = 1
        weights = os.path.join(path, WEIGHTS_NAME)
        self._fh = open(weights, "rb")
        self._size = os.fstat(self._fh.fileno()).st_size
        if self._size < 8:
            self._fh.close()
            raise GGUFFormatError(f"{weights}: too small to be a safetensors file ({self._size} bytes)")
        self._mm = mmap.mmap(self._fh.fileno(), 0, access=mmap.ACCESS_READ)
        self._buf = memoryview(self._mm)
        try:
            self._parse_safetensors(weights)
        except Exception:
            self.close()
            raise

    def _parse_safetensors(self, weights: str) -> None:
        n, = struct.unpack_from("<Q", self._buf, 0)
        self.data_offset = 8 + n
        if self.data_offset > self._size:
            raise GGUFFormatError(f"{weights}: header of {n} bytes runs past end of file")
        try:
            header = json.loads(bytes(self._buf[8:self.data_offset]))
        except ValueError as exc:
            raise GGUFFormatError(f"{weights}: header is not JSON ({exc})") from exc
        for name, e in header.items():
            if name == "__metadata__":
                continue
            kind, shape, (a, b) = e["dtype"], tuple(int(d) for d in e["shape"]), e["data_offsets"]
            if kind not in _TYPES:
                raise GGUFFormatError(f"{weights}: tensor {name!r} has unsupported type {kind}")
            count = int(np.prod(shape, dtype=np.int64)) if shape else 1
            if b - a != count * _BYTES[kind] or a < 0 or self.data_offset + b > self._size:
                raise GGUFFormatError(f"{weights}: tensor {name!r} of shape {shape} does not fit its bytes [{a}, {b})")
            self.tensors[name] = GGUFTensorInfo(name, tuple(reversed(shape)) or (1,), _TYPES[kind], int(a), int(b - a))


def open_checkpoint(path: str) -> GGUFFile:
    """A model folder or a GGUF file, whichever ``path`` is."""
    return ModelFolder(path) if os.path.isdir(path) else GGUFFile(path)


def write_safetensors(path: str, tensors: Dict[str, "object"]) -> None:
    """Write torch tensors (bfloat16, float16, float32, int32) as a safetensors file."""
    import torch
    kinds = {torch.bfloat16: "BF16", torch.float16: "F16", torch.float32: "F32", torch.int32: "I32"}
    header, off = {}, 0
    for name, t in tensors.items():
        n = t.numel() * t.element_size()
        header[name] = {"dtype": kinds[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + n]}
        off += n
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for t in tensors.values():
            f.write(t.detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes())
