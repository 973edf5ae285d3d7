"""What the models that come as a folder (``config.json``, ``model.safetensors``) share: the layer runs of a loop, tensors
padded to what the kernels want aligned, and the choice between bf16 and 32-bit execution."""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch
import torch.nn.functional as TF

from ..gguf.constants import GGMLType
from ..quant.qweight import QuantWeight
from .base import ModelBase


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class FolderModel(ModelBase):
    supports_float32 = True
    mixed_batches = True

    # ------------------------------------------------------------------ configuration
    def parse_layers(self) -> None:
        """``layers`` and ``loop`` of config.json: the layer runs in execution order, ``runs[i] = (layer, pass)`` with the pass
        number at a run that begins one and None elsewhere."""
        j = self.gguf.config
        self.layer_specs: List[dict] = list(j["layers"])
        n = len(self.layer_specs)
        loop = j.get("loop") or {}
        self.loop = (int(loop.get("start", 0)), int(loop.get("stop", 0)), int(loop.get("times", 1))) if loop else (0, 0, 1)
        a, b, times = self.loop
        if not (0 <= a <= b <= n and times >= 0):
            raise ValueError(f"{self.path}: loop {loop} does not fit {n} layers")
        self.runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for t in range(times):
            self.runs += [(i, t if loop and i == a else None) for i in range(a, b)]
        self.runs += [(i, None) for i in range(b, n)]
        self.width = int(j["width"])

    def refuse_parallel(self) -> None:
        if self.tp_size > 1 or self.ep_size > 1:
            raise ValueError(f"{self.gguf.config.get('architecture')} runs on one GPU (no tensor- or expert-parallel path)")

    # ------------------------------------------------------------------ weights
    def _host(self, name: str) -> torch.Tensor:
        """A stored matrix or vector on the host, in its stored float type."""
        ti = self.gguf.tensors.get(name)
        if ti is None:
            raise KeyError(f"{self.path}: tensor {name!r} not found")
        kinds = {GGMLType.BF16: torch.bfloat16, GGMLType.F16: torch.float16, GGMLType.F32: torch.float32}
        if ti.ggml_type not in kinds:
            raise ValueError(f"{self.path}: tensor {name!r} has type {ti.ggml_type.name}, a float type is needed")
        raw = torch.frombuffer(bytearray(self.gguf.tensor_bytes_view(name)), dtype=kinds[ti.ggml_type])
        return raw.view(ti.shape)

    def _mat(self, name: str, rows: Optional[int] = None, cols: Optional[int] = None) -> torch.Tensor:
        """A stored matrix, padded with zero rows / columns."""
        w = self._host(name)
        return TF.pad(w, (0, (cols or w.shape[1]) - w.shape[1], 0, (rows or w.shape[0]) - w.shape[0]))

    def _vec(self, name: str, n: int) -> torch.Tensor:
        w = self._host(name).float()
        return TF.pad(w, (0, n - w.shape[-1])).to(self.device).contiguous()

    def _qw(self, w: torch.Tensor, name: str) -> QuantWeight:
        """A float matrix ``[N, K]`` or stack ``[E, N, K]`` as the linear kernels take it."""
        t = GGMLType.BF16 if w.dtype == torch.bfloat16 else GGMLType.F32
        w = w if t == GGMLType.BF16 else w.float()
        return QuantWeight.from_raw(w.contiguous().view(-1).view(torch.uint8), t, tuple(w.shape), self.device, name)

    def _heads(self, name: str, H: int, d: int, dp: int) -> torch.Tensor:
        """[H * d, width] -> [H * dp, D], every head padded with zero rows."""
        w = self._mat(name, cols=self.cfg.hidden)
        if w.shape[0] != H * d:
            raise ValueError(f"{self.path}: tensor {name!r} has {w.shape[0]} rows, {H} heads of {d} need {H * d}")
        return TF.pad(w.view(H, d, -1), (0, 0, 0, dp - d)).reshape(H * dp, -1)

    def _head_vec(self, name: str, H: int, d: int, dp: int) -> torch.Tensor:
        return TF.pad(self._host(name).float().view(H, d), (0, dp - d)).reshape(-1)

    def _out(self, name: str, H: int, d: int, dp: int):
        """Output projection [D, H * d] with the heads' columns padded."""
        D = self.cfg.hidden
        return self._qw(TF.pad(self._mat(name, rows=D).view(D, H, d), (0, dp - d)).reshape(D, H * dp), name)

    @staticmethod
    def _rows(w: QuantWeight, first: int, end: int) -> QuantWeight:
        """Rows [first, end) of a float matrix, on the same memory."""
        per = w.planes[0].numel() // w.rows
        return QuantWeight(w.ggml_type, end - first, w.K, [w.planes[0][first * per:end * per]], 1, w.name)

    # ------------------------------------------------------------------ execution
    @property
    def bf16(self) -> bool:
        return self.device.type == "cuda" and self.compute_dtype == torch.bfloat16
