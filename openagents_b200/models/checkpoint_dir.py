"""Checkpoints that come as a folder: ``config.json`` and ``model.safetensors``.

A safetensors file is an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape, data_offsets) and
the tensors' bytes.  The reader maps the file and checks every entry against the file's size before it hands out a view.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np
import torch

from ..gguf import GgmlType
from .config import config_from_json
from .qweight import RawTensor, WeightSource

_DTYPES = {"BF16": (2, torch.bfloat16, GgmlType.BF16), "F16": (2, torch.float16, GgmlType.F16), "F32": (4, torch.float32, GgmlType.F32),
           "I32": (4, torch.int32, None)}
_MAX_HEADER = 100 << 20


class SafetensorsFile:
    def __init__(self, path: str):
        size = os.path.getsize(path)
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        self.map = np.memmap(path, dtype=np.uint8, mode="r")
        n = struct.unpack("<Q", bytes(self.map[:8]))[0]
        if n > min(_MAX_HEADER, size - 8):
            raise ValueError(f"{path}: the header does not fit the file")
        try:
            header = json.loads(bytes(self.map[8: 8 + n]).decode("utf-8"))
        except (UnicodeDecodeError, json.JSONDecodeError) as e:
            raise ValueError(f"{path}: bad header") from e
        if not isinstance(header, dict):
            raise ValueError(f"{path}: bad header")
        self.base, room = 8 + n, size - 8 - n
        self.entries: dict[str, tuple[str, tuple[int, ...], int, int]] = {}
        for name, e in header.items():
            if name == "__metadata__":
                continue
            try:
                dt, shape, (lo, hi) = e["dtype"], tuple(int(x) for x in e["shape"]), (int(x) for x in e["data_offsets"])
            except (TypeError, KeyError, ValueError) as err:
                raise ValueError(f"{path}: bad entry for {name!r}") from err
            count = 1
            for x in shape:
                count *= x
            if dt not in _DTYPES or min(shape, default=1) < 0 or not 0 <= lo <= hi <= room or hi - lo != count * _DTYPES[dt][0]:
                raise ValueError(f"{path}: bad entry for {name!r}")
            self.entries[name] = (dt, shape, lo, hi)

    def tensor(self, name: str) -> torch.Tensor:
        """The tensor on the host, in its stored type (a copy)."""
        dt, shape, lo, hi = self.entries[name]
        raw = torch.from_numpy(np.array(self.map[self.base + lo: self.base + hi]))
        return raw.view(_DTYPES[dt][1]).reshape(shape)


class CheckpointDirSource(WeightSource):
    """Tensors of a checkpoint folder by their own names, copied to ``device`` on demand."""

    def __init__(self, path: str, device):
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            self.json = json.load(f)
        self.file = SafetensorsFile(os.path.join(path, "model.safetensors"))
        self.device = device
        ranks = {}
        for name, (_, shape, _, _) in self.file.entries.items():      # sizes only a tensor's shape gives
            if name.startswith("l") and name.endswith((".mix.a1", ".mix.dq", ".mix.w1")) and len(shape) == 2 and name[1:-7].isdigit():
                ranks[int(name[1:-7])] = shape[0]
        self.cfg = config_from_json(self.json, ranks, name=os.path.basename(os.path.normpath(path)))
        self.metadata: dict = {}
        from .weights import tensor_specs
        for spec in tensor_specs(self.cfg):
            e = self.file.entries.get(spec.name)
            if e is None:
                raise ValueError(f"{path}: tensor {spec.name!r} is missing")
            if (e[1] or (1,)) != tuple(spec.shape):        # a number may be stored without an axis
                raise ValueError(f"{path}: tensor {spec.name!r} has shape {list(e[1])}, expected {list(spec.shape)}")

    def has(self, name):
        return name in self.file.entries

    def get(self, name):
        dt, shape, _, _ = self.file.entries[name]
        t, shape = _DTYPES[dt][2], shape or (1,)
        if t is None:
            raise ValueError(f"tensor {name!r} holds integers")
        return RawTensor(t, shape, self.file.tensor(name).reshape(-1).view(torch.uint8).to(self.device))
