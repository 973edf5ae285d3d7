"""Fobolorn: a decoder with sandwich layer norms, gated grouped-query attention without rotary embedding, a softmax-routed
mixture of experts with a gated shared expert, and a range of layers that runs several times with the same weights.

A layer:  x += post1(attention(pre1(x)));  x += post2(experts(pre2(x)))  with layer norms (weight and bias).
  attention   q, k RMS-normed per head (value heads may have another size); q scaled by 1 + c ln(floor((p + 1) / n) + 1) at
              position p; causal softmax(scale q k); head h times sigmoid(g_h), g from the layer's input; output projection
  experts     softmax over all router logits, the top ones renormalised and scaled; plus the shared expert times
              sigmoid(s), s from the layer's input; every expert is down(silu(gate x) up x)
  loop        layers [start, stop) run ``times`` times; pass t first adds row t of ``loop.step``.  Every pass of a layer has
              its own K / V cache: the cache's layers are the layer *runs* in execution order.

Weights come from a model folder (config.json, model.safetensors).  Sizes that the kernels want aligned are padded with
zeros at load time: columns (width, feed-forward) to 8, head sizes to 16; norms keep their true divisors.  The shared expert
is cut into slices of the experts' size, which run as further experts of every token, so that one grouped product serves
both.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn.functional as TF

from ..ops import functional as F
from ..ops.functional import Act, Batch
from .base import ModelConfig, register_architecture
from .folder import FolderModel, round_up


@dataclass
class AttnSpec:
    """Sizes of one attention mixer (``Dk`` / ``Dv``: padded head sizes)."""
    H: int
    G: int
    dim: int
    vdim: int
    Dk: int
    Dv: int
    scale: float
    q_temp: Optional[Tuple[float, float]]


@dataclass
class MoeSpec:
    E: int
    top: int
    scale: float
    shared: int              # slices of the shared expert (0: none)


@register_architecture("fobolorn")
class FobolornModel(FolderModel):
    native_sources = ("error.cpp", "elementwise.cu", "sandwich_norm.cu", "float32.cu", "attention.cu", "attention_vd.cu",
                      "attention_decode_mma.cu", "gemm_tcgen05.cu", "gemv.cu", "gemv_bf16.cu", "gemv_mma.cu", "gemv_stream.cu", "moe.cu", "sampler.cu")

    # ------------------------------------------------------------------ configuration
    def parse_base_config(self) -> ModelConfig:
        self.parse_layers()
        j, n = self.gguf.config, len(self.layer_specs)
        first = self.layer_specs[0]["mixer"] if n else {}
        return ModelConfig(arch=self.arch, n_layers=len(self.runs), hidden=round_up(self.width, 8), n_heads=int(first.get("heads", 0)),
                           n_kv_heads=int(first.get("kv_heads", 0)), head_dim=int(first.get("dim", 0)), vocab=int(j["vocab"]),
                           eps=float(j["norm"]["eps"]), context_length=int(j.get("context_length", 4096)))

    def parse_config(self) -> None:
        self.refuse_parallel()
        for i, s in enumerate(self.layer_specs):
            if s["type"] != "attention":
                raise ValueError(f"{self.path}: layer {i} has unknown type {s['type']!r}")
            if s["mlp"] is not None and s["mlp"].get("kind", "moe") != "moe":
                raise ValueError(f"{self.path}: layer {i} has unknown feed-forward {s['mlp'].get('kind')!r}")

    # ------------------------------------------------------------------ weights
    def _norm(self, name: str) -> Tuple[torch.Tensor, torch.Tensor]:
        return self._vec(name, self.cfg.hidden), self._vec(name + ".b", self.cfg.hidden)

    def _attention(self, p: str, m: dict) -> Dict[str, object]:
        D = self.cfg.hidden
        H, G, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        if H % G:
            raise ValueError(f"{p}: {H} heads are not a multiple of {G} key / value heads")
        s = AttnSpec(H, G, dim, vdim, round_up(dim, 16), round_up(vdim, 16), float(m["scale"]),
                     (float(m["q_temp"]["coef"]), float(m["q_temp"]["every"])) if m.get("q_temp") else None)
        if max(s.Dk, s.Dv) > 256:
            raise ValueError(f"{p}: head sizes {dim} / {vdim} are above 256")

        def heads(name, n, d, dp):                      # [n * d, K] -> [n * dp, D], every head padded
            w = self._mat(p + name, cols=D).view(n, d, D)
            return TF.pad(w, (0, 0, 0, dp - d)).reshape(n * dp, D)
        parts = [heads("q", H, dim, s.Dk), heads("k", G, dim, s.Dk), heads("v", G, vdim, s.Dv), self._mat(p + "g", cols=D)]
        w = torch.cat(parts)
        w = TF.pad(w, (0, 0, 0, round_up(w.shape[0], 8) - w.shape[0]))            # rows of the result stay 16-byte aligned
        wo = TF.pad(self._mat(p + "o", rows=D).view(D, H, vdim), (0, s.Dv - vdim)).reshape(D, H * s.Dv)
        return {"spec": s, "wqkvg": self._qw(w, p + "qkvg"), "wo": self._qw(wo, p + "o"),
                "qn": self._vec(p + "q.norm", s.Dk), "kn": self._vec(p + "k.norm", s.Dk)}

    def _moe(self, p: str, m: dict) -> Dict[str, object]:
        D = self.cfg.hidden
        r = m["router"]
        E, top, ff = int(r["experts"]), int(r["top"]), round_up(int(m["expert"]["ff"]), 8)
        shared = m.get("shared")
        gate = [self._mat(f"{p}e{e}.gate", ff, D) for e in range(E)]
        up = [self._mat(f"{p}e{e}.up", ff, D) for e in range(E)]
        down = [self._mat(f"{p}e{e}.down", D, ff) for e in range(E)]
        router = self._mat(p + "router", cols=D)
        slices = 0
        if shared:
            # silu(gate x) * up x is separate per feature, so the shared expert is the sum of its slices of ff features
            slices = -(-int(shared["ff"]) // ff)
            sg, su = (self._mat(f"{p}shared.{n}", slices * ff, D) for n in ("gate", "up"))
            sd = self._mat(p + "shared.down", D, slices * ff)
            gate += list(sg.split(ff))
            up += list(su.split(ff))
            down += list(sd.split(ff, 1))
            router = torch.cat([router, self._mat(p + "shared.sg", cols=D)])
        if top > min(E, 32) or E + slices > 1024:
            raise ValueError(f"{p}: top {top} of {E} experts with {slices} shared slices (limits: 32, 1024)")
        return {"spec": MoeSpec(E, top, float(r["scale"]), slices), "router": self._qw(router, p + "router"),
                "gate_up": self._qw(torch.stack([torch.cat([g, u]) for g, u in zip(gate, up)]), p + "gate_up"),
                "down": self._qw(torch.stack(down), p + "down")}

    def load_weights(self) -> None:
        if self.kv_dtype == torch.float8_e4m3fn:
            raise ValueError("Fobolorn has no 8-bit KV cache")
        D = self.cfg.hidden
        if self.device.type == "cuda":
            self.kv_dtype = self.compute_dtype          # bf16 pages, or f32 pages in a 32-bit run
        self.tok_emb = self._qw(self._mat("embed", cols=D), "embed")
        self.lm_head = self._qw(self._mat("head", cols=D), "head")
        self.out_norm = self._norm("final.norm")
        self.step_vec = self._vec("loop.step", D) if any(t is not None for _, t in self.runs) else None
        self.layers: List[Dict[str, object]] = []
        for i, s in enumerate(self.layer_specs):
            p = f"l{i}."
            L = {"norm1": self._norm(p + "norm1"), "norm1b": self._norm(p + "norm1b"), **self._attention(p + "mix.", s["mixer"]), "mlp": None}
            if s["mlp"] is not None:
                L["norm2"], L["norm2b"] = self._norm(p + "norm2"), self._norm(p + "norm2b")
                L["mlp"] = self._moe(p + "mlp.", s["mlp"])
            self.layers.append(L)

    def kv_layer_shapes(self):
        return [(s.G, s.Dk, s.Dv) for s in (self.layers[i]["spec"] for i, _ in self.runs)]

    # ------------------------------------------------------------------ execution
    def attention(self, a: Act, L, run: int, batch: Batch) -> torch.Tensor:
        """Projections, per-head norms, cache write and gated attention -> ``[T, H * Dv]``."""
        s, T = L["spec"], batch.T
        y = F.linear(a, L["wqkvg"], out_dtype=torch.bfloat16 if self.bf16 and T > F.GEMV_MAX_M else torch.float32)
        nq, nk, nv = s.H * s.Dk, s.G * s.Dk, s.G * s.Dv
        q = F.qkv_rope_cache(y[:, :nq].view(T, s.H, s.Dk), y[:, nq:nq + nk].view(T, s.G, s.Dk),
                             y[:, nq + nk:nq + nk + nv].view(T, s.G, s.Dv), Hq=s.H, Hkv=s.G, Dh=s.Dk, Dv=s.Dv, norm_n=s.dim, batch=batch,
                             k_cache=self.kv.k[run], v_cache=self.kv.v[run], rope=None, qn=L["qn"], kn=L["kn"], eps=self.cfg.eps,
                             q_temp=s.q_temp)
        g0 = nq + nk + nv
        return F.attention(q, self.kv.k[run], self.kv.v[run], batch, scale=s.scale, Hq=s.H, Hkv=s.G, Dh=s.Dk, Dv=s.Dv, gate=y[:, g0:g0 + s.H])

    def experts(self, a: Act, m):
        """Routed and shared experts; their rows are summed by the norm that follows."""
        s = m["spec"]
        logits = F.linear(a, m["router"], out_dtype=torch.float32)
        ids, w = F.route_softmax_renorm(logits, s.E, s.top, s.scale, s.shared)
        return F.moe_expert_parts(a, ids, w, m["gate_up"], m["down"], act="swiglu")

    def forward_batch(self, batch: Batch, want_logits: bool = True) -> Optional[torch.Tensor]:
        c, n, dt = self.cfg, self.width, self.compute_dtype
        h = self.inject_pending_embeddings(F.embed(self.tok_emb, batch.tokens))
        want_logits = want_logits and batch.last_idx.numel() > 0
        every_row = batch.is_decode and batch.last_idx.numel() == batch.T     # decode: all rows give logits, in their order

        def seam(y, post, nxt):
            """Close a sublayer (``y`` through its post norm) and open the one at ``nxt``: (run, sublayer) or None."""
            pre, add = self.out_norm, None
            if nxt is not None:
                i, t = self.runs[nxt[0]]
                pre = self.layers[i][nxt[1]]
                if nxt[1] == "norm1" and t is not None:
                    add = self.step_vec[t]
            return F.residual_layernorm(h, c.eps, n, y=y, post=post, add=add, pre=pre, dtype=dt)

        last = len(self.runs) - 1
        a = seam(None, None, (0, "norm1") if self.runs else None)
        for r, (i, _) in enumerate(self.runs):
            L = self.layers[i]
            o = self.attention(a, L, r, batch)
            if r == last:
                if not want_logits:
                    return None
                if not every_row:                       # past the last cache write only the wanted rows matter
                    o, h = o.index_select(0, batch.last_idx), h.index_select(0, batch.last_idx)
            nxt = (r + 1, "norm1") if r < last else None
            y = F.linear(Act(o), L["wo"], out_dtype=torch.bfloat16 if self.bf16 and o.shape[0] > F.GEMV_MAX_M else torch.float32)
            if L["mlp"] is not None:
                a = seam(y, L["norm1b"], (r, "norm2"))
                a = seam(self.experts(a, L["mlp"]), L["norm2b"], nxt)
            else:
                a = seam(y, L["norm1b"], nxt)
        if not self.runs and not every_row:
            a = Act(a.b.index_select(0, batch.last_idx))
        return F.linear(a, self.lm_head, out_dtype=torch.float32) if want_logits else None
