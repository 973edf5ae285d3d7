"""Sogulix: a hybrid of latent attention and a generalized delta rule in parallel layers, with a range of layers that runs
several times with the same weights.

A layer:  x += m (ls1 mixer(shift(norm1(x))) + ls2 ff(norm2(x)))  with RMS norms whose weights are offsets from 1
(factor 1 + w); ``shift`` moves every channel towards the previous token's normalised value.
  latent_attention   queries through a normed latent; one normed latent per token for the keys and values of all heads, plus
                     one rotated key part they share; sliding window, a sink per head in the softmax
  general_delta      S <- diag(w) S - (a u)(u^T S) + k v^T per head with unit keys u, a decay w and a removal rate a per key
                     channel; o = S^T r, divided by its root mean square, times sigmoid of a gate
  ff                 down(silu(gate x) up x)
  loop               ahead of every pass  x = W_in [x; x0]  with the normed embedding x0; every pass of a layer has its own
                     cache rows and states: both are kept per layer *run*, in execution order.
The logits are capped: c tanh(z / c).

Weights come from a model folder.  Sizes that the kernels want aligned are padded with zeros at load time: columns (width,
feed-forward, ranks) to 8, attention heads to 16, delta heads to 32; norms keep their true divisors.  The first projections
of a mixer are one matrix.  m is folded into the layer scales.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn.functional as TF

from ..ops import functional as F
from ..ops.functional import Act, Batch, LatentSpec
from .base import ModelConfig, register_architecture
from .folder import FolderModel, round_up


@dataclass
class DeltaSpec:
    """Sizes of one delta-rule mixer (``D``: the padded head size)."""
    H: int
    n: int
    D: int
    rank: int


@register_architecture("sogulix")
class SogulixModel(FolderModel):
    supports_kv_truncation = False           # recurrent state and the token shift's previous row
    graphs_with_state = True
    native_sources = ("error.cpp", "elementwise.cu", "parallel_norm.cu", "general_delta.cu", "general_delta_chunk.cu", "attention_latent.cu", "float32.cu", "attention.cu",
                      "attention_vd.cu", "attention_decode_mma.cu", "gemm_tcgen05.cu", "gemv.cu", "gemv_bf16.cu", "gemv_mma.cu", "gemv_stream.cu",
                      "moe.cu", "sampler.cu")

    # ------------------------------------------------------------------ configuration
    def parse_base_config(self) -> ModelConfig:
        self.parse_layers()
        j = self.gguf.config
        self.residual_mult = float(j.get("residual_mult", 1.0))
        self.logit_softcap = float(j.get("logit_softcap") or 0.0)
        first = self.layer_specs[0]["mixer"] if self.layer_specs else {}
        return ModelConfig(arch=self.arch, n_layers=len(self.runs), hidden=round_up(self.width, 8), n_heads=int(first.get("heads", 0)),
                           n_kv_heads=1, head_dim=int(first.get("dim", 0)), vocab=int(j["vocab"]), eps=float(j["norm"]["eps"]),
                           context_length=int(j.get("context_length", 4096)))

    def parse_config(self) -> None:
        self.refuse_parallel()
        for i, s in enumerate(self.layer_specs):
            if s["type"] not in ("latent_attention", "general_delta"):
                raise ValueError(f"{self.path}: layer {i} has unknown type {s['type']!r}")
            if s["mlp"] is not None and s["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"{self.path}: layer {i} has unknown feed-forward {s['mlp'].get('kind')!r}")

    # ------------------------------------------------------------------ weights
    def _norm1p(self, name: str) -> torch.Tensor:
        """The factor 1 + w of a norm stored as its offset from 1 (0 in the padding)."""
        w = self._host(name).float() + 1.0
        return TF.pad(w, (0, self.cfg.hidden - w.shape[0])).to(self.device).contiguous()

    def _per_head(self, name: str, H: int, d: int, dp: int, cols: Optional[int] = None) -> torch.Tensor:
        """[H * d, K] -> [H * dp, K (padded to ``cols``)], every head padded with zero rows."""
        w = self._mat(name, cols=cols)
        if w.shape[0] != H * d:
            raise ValueError(f"{self.path}: tensor {name!r} has {w.shape[0]} rows, {H} heads of {d} need {H * d}")
        return TF.pad(w.view(H, d, -1), (0, 0, 0, dp - d)).reshape(H * dp, -1)

    def _head_vec(self, name: str, H: int, d: int, dp: int) -> torch.Tensor:
        return TF.pad(self._host(name).float().view(H, d), (0, dp - d)).reshape(-1).to(self.device).contiguous()

    def _out(self, name: str, H: int, d: int, dp: int):
        """Output projection [D, H * d] with the heads' columns padded."""
        D = self.cfg.hidden
        return self._qw(TF.pad(self._mat(name, rows=D).view(D, H, d), (0, dp - d)).reshape(D, H * dp), name)

    def _latent(self, p: str, m: dict) -> Dict[str, object]:
        D = self.cfg.hidden
        H, dim, rot, vdim, rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        turn = m.get("rot") or {"dims": rot, "base": 1.0}
        if int(turn["dims"]) != rot or rot % 2:
            raise ValueError(f"{p}: the rotation covers {turn['dims']} of {rot} rotated dimensions")
        q_rank = self._host(p + "dq").shape[0]
        window = int(m["mask"]["size"]) if m.get("mask") else 0
        s = LatentSpec(H, dim, rot, vdim, rank, q_rank, float(m["scale"]), window, float(turn["base"]),
                       F.rotary_freqs(rot, float(turn["base"]), self.device))
        if max(s.Dk, s.Dv) > 256 or rank > 512 or s.row > 704:
            raise ValueError(f"{p}: head sizes {dim} + {rot} / {vdim} or latent size {rank} are above 256 / 512")
        down = torch.cat([self._mat(p + "dq", rows=s.qp, cols=D), self._mat(p + "dkv", cols=D)])
        down = TF.pad(down, (0, 0, 0, round_up(down.shape[0], 8) - down.shape[0]))
        uq = self._per_head(p + "uq", H, dim + rot, s.Dk, s.qp)
        uk = self._mat(p + "uk", cols=s.rank_p)
        uv = self._per_head(p + "uv", H, vdim, s.Dv, s.rank_p)
        L = {"latent": s, "down": self._qw(down, p + "down"), "uq": self._qw(uq, p + "uq"), "wuk": uk.to(self.device).contiguous(),
             "wuv": uv.to(self.device).contiguous(), "qn": self._vec(p + "dq.norm", q_rank), "kn": self._vec(p + "dkv.norm", rank),
             "sinks": self._vec(p + "sink", H), "wo": self._out(p + "o", H, vdim, s.Dv), "expand": None}
        if self.bf16:
            # keys and values of all heads from whole cached rows; the rotated part is handed on by an identity block
            k = torch.zeros(H, s.Dk, s.row, dtype=torch.bfloat16)
            k[:, :dim, :rank] = uk.view(H, dim, -1)[..., :rank]
            k[:, dim:dim + rot, rank:rank + rot] = torch.eye(rot)
            v = torch.zeros(H * s.Dv, s.row, dtype=torch.bfloat16)
            v[:, :rank] = uv[:, :rank]
            L["expand"] = self._qw(torch.cat([k.view(H * s.Dk, s.row), v]), p + "expand")
        return L

    def _delta(self, p: str, m: dict) -> Dict[str, object]:
        D = self.cfg.hidden
        H, n = int(m["heads"]), int(m["dim"])
        rank = self._host(p + "w1").shape[0]
        s = DeltaSpec(H, n, round_up(n, 32), rank)
        if s.D > 256 or rank > 4096:
            raise ValueError(f"{p}: head size {n} or decay rank {rank} are above 256 / 4096")
        rp = round_up(rank, 8)
        parts = [self._per_head(p + x, H, n, s.D, D) for x in ("r", "k", "v", "a", "g")] + [self._mat(p + "w1", rows=rp, cols=D)]
        return {"delta": s, "proj": self._qw(torch.cat(parts), p + "proj"), "w2": self._qw(self._per_head(p + "w2", H, n, s.D, rp), p + "w2"),
                "w0": self._head_vec(p + "w0", H, n, s.D), "ab": self._head_vec(p + "a.b", H, n, s.D),
                "on": self._head_vec(p + "norm", H, n, s.D), "wo": self._out(p + "o", H, n, s.D)}

    def load_weights(self) -> None:
        if self.kv_dtype == torch.float8_e4m3fn:
            raise ValueError("Sogulix has no 8-bit KV cache")
        D, m = self.cfg.hidden, self.residual_mult
        if self.device.type == "cuda":
            self.kv_dtype = self.compute_dtype          # bf16 pages, or f32 pages in a 32-bit run
        self.tok_emb = self._qw(self._mat("embed", cols=D), "embed")
        self.lm_head = self._qw(self._mat("head", cols=D), "head")
        self.emb_norm, self.out_norm = self._norm1p("embed.norm"), self._norm1p("final.norm")
        self.loop_in = None
        if any(t is not None for _, t in self.runs):
            w = self._mat("loop.in", rows=D)
            if w.shape[1] != 2 * self.width:
                raise ValueError(f"{self.path}: loop.in has {w.shape[1]} columns, not twice the width")
            self.loop_in = self._qw(TF.pad(w.view(D, 2, self.width), (0, D - self.width)).reshape(D, 2 * D), "loop.in")
        self.layers: List[Dict[str, object]] = []
        for i, s in enumerate(self.layer_specs):
            p = f"l{i}."
            L = {"norm1": self._norm1p(p + "norm1"), "shift": self._vec(p + "shift", D), "ls1": self._vec(p + "ls1", D) * m, "gate_up": None,
                 "norm2": None, "ls2": None}
            L.update(self._latent(p + "mix.", s["mixer"]) if s["type"] == "latent_attention" else self._delta(p + "mix.", s["mixer"]))
            if s["mlp"] is not None:
                ff = round_up(int(s["mlp"]["ff"]), 8)
                L["norm2"], L["ls2"] = self._norm1p(p + "norm2"), self._vec(p + "ls2", D) * m
                L["gate_up"] = self._qw(torch.cat([self._mat(f"{p}mlp.{n}", ff, D) for n in ("gate", "up")]), p + "gate_up")
                L["ff_down"] = self._qw(self._mat(p + "mlp.down", D, ff), p + "ff_down")
            self.layers.append(L)
        self._make_state()

    # ------------------------------------------------------------------ cache and state
    def _make_state(self) -> None:
        """One f32 row per sequence slot for everything that is carried from token to token: per layer run the row ahead of
        the token shift, and S of a delta-rule mixer.  ``shift_state`` / ``delta_state`` are views into it."""
        D, off, at = self.cfg.hidden, 0, []
        for i, _ in self.runs:
            s = self.layers[i].get("delta")
            at.append(off)
            off += D + (s.H * s.D * s.D if s is not None else 0)
        self.state = torch.zeros((max(self.max_seqs, 1), max(off, 1)), dtype=torch.float32, device=self.device)
        self.shift_state, self.delta_state = [], []
        for (i, _), o in zip(self.runs, at):
            s = self.layers[i].get("delta")
            self.shift_state.append(self.state[:, o:o + D])
            self.delta_state.append(self.state[:, o + D:o + D + s.H * s.D * s.D].unflatten(1, (s.H, s.D, s.D)) if s is not None else None)

    def recurrent_state_tensors(self) -> list:
        return [self.state]

    def reset_recurrent_state(self, slot: int) -> None:
        self.state[slot].zero_()

    def kv_layer_shapes(self):
        """A latent layer caches one row per token and no separate value."""
        return [(1, self.layers[i]["latent"].row, 0) if "latent" in self.layers[i] else None for i, _ in self.runs]

    def kv_window_layers(self) -> Dict[int, int]:
        return {r: self.layers[i]["latent"].window for r, (i, _) in enumerate(self.runs) if "latent" in self.layers[i] and self.layers[i]["latent"].window}

    # ------------------------------------------------------------------ execution
    def _mid(self, T: int) -> torch.dtype:
        """Type of what a product hands to the next step: f32, or bf16 for prompts."""
        return torch.bfloat16 if self.bf16 and T > F.GEMV_MAX_M else torch.float32

    def latent_mixer(self, a: Act, L, run: int, batch: Batch) -> torch.Tensor:
        """Down projections, norms, cache write, attention -> ``[T, H * Dv]`` (before the output projection)."""
        s = L["latent"]
        if self.kv.is_window_layer(run):
            batch = batch.windowed()
        y = F.linear(a, L["down"], out_dtype=torch.float32)
        cq = F.latent_cache(y, s, L["qn"], L["kn"], self.kv.k[run], batch, self.cfg.eps)
        q = F.linear(cq, L["uq"], out_dtype=torch.bfloat16 if self.bf16 and not batch.is_decode else torch.float32)
        return F.latent_attention(q, self.kv.k[run], batch, s, wuk=L["wuk"], wuv=L["wuv"], expand=L["expand"], sinks=L["sinks"])

    def delta_mixer(self, a: Act, L, run: int, batch: Batch) -> torch.Tensor:
        """Projections and the recurrence with its norm and gate -> ``[T, H * D]``."""
        s = L["delta"]
        y = F.linear(a, L["proj"], out_dtype=torch.float32)
        return F.general_delta(y, L["w2"], L["w0"], L["ab"], L["on"], self.delta_state[run], batch, H=s.H, D=s.D, n=s.n, rank=s.rank,
                               eps=self.cfg.eps, dtype=self.compute_dtype if self.device.type == "cuda" else torch.float32)

    def feed_forward(self, a: Act, L) -> torch.Tensor:
        g = F.linear(a, L["gate_up"], act="swiglu", out_dtype=torch.bfloat16 if self.bf16 else torch.float32)
        return F.linear(Act(g), L["ff_down"], out_dtype=self._mid(g.shape[0]))

    def forward_batch(self, batch: Batch, want_logits: bool = True) -> Optional[torch.Tensor]:
        c, n, D, dt = self.cfg, self.width, self.cfg.hidden, self.compute_dtype
        h = self.inject_pending_embeddings(F.embed(self.tok_emb, batch.tokens))
        want_logits = want_logits and batch.last_idx.numel() > 0
        every_row = batch.is_decode and batch.last_idx.numel() == batch.T     # decode: all rows give logits, in their order
        both = None                                     # [x | x0]: what enters a pass of the loop
        if self.loop_in is not None:
            both = torch.empty((batch.T, 2 * D), dtype=dt, device=h.device)
        _, h, _ = F.parallel_seam(h, c.eps, n, w=(self.emb_norm, self.emb_norm), out=(None, both[:, D:] if both is not None else None), outputs=1,
                                  dtype=torch.float32)
        y: Tuple = (None, None)
        scale: Tuple = (None, None)
        last = len(self.runs) - 1
        for r, (i, begins) in enumerate(self.runs):
            L = self.layers[i]
            if begins is not None:
                F.parallel_seam(h, c.eps, n, y=y, scale=scale, out=(both[:, :D], None), outputs=1)
                h, y = F.linear(Act(both), self.loop_in, out_dtype=torch.float32), (None, None)
            ff = L["gate_up"] is not None
            h, a, a2 = F.parallel_seam(h, c.eps, n, y=y, scale=scale, w=(L["norm1"], L["norm2"]), outputs=2 if ff else 1, dtype=dt,
                                       shift=L["shift"], state=self.shift_state[r], batch=batch)
            o = (self.latent_mixer if "latent" in L else self.delta_mixer)(Act(a), L, r, batch)
            if r == last:
                if not want_logits:
                    return None
                if not every_row:                       # past the last cache and state only the wanted rows matter
                    o, h, a2 = (t.index_select(0, batch.last_idx) if t is not None else None for t in (o, h, a2))
            y = (F.linear(Act(o), L["wo"], out_dtype=self._mid(o.shape[0])), self.feed_forward(Act(a2), L) if ff else None)
            scale = (L["ls1"], L["ls2"])
        if not self.runs and not every_row:
            h = h.index_select(0, batch.last_idx)
        _, a, _ = F.parallel_seam(h, c.eps, n, y=y, scale=scale, w=(self.out_norm, None), outputs=1, dtype=dt)
        return F.softcap(F.linear(Act(a), self.lm_head, out_dtype=torch.float32), self.logit_softcap)
