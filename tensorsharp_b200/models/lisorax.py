"""Lisorax: a decoder whose layers run a mixer and a mixture of experts side by side on one norm, the mixer through a convolution
over time; three kinds of mixers.

A layer:  h = norm1(x);  x += mixer(h + conv(h)) + experts(h)  with RMS norms and a causal convolution per channel.
  attention   grouped-query attention without rotation: a short convolution on queries, keys and values, a query temperature that
              grows with the position, capped scores, a distance bias r1 ln(1 + r2 d) per head, and sigmoid(score + pb) as the
              weight of a key, not normalised.  A layer may read another layer's cached keys and values instead of its own
  rglru       y = gelu(W_y h + b);  u = conv(W_x h + b) + b;  S <- a S + sqrt(1 - a^2) i u  with log a = -8 r softplus(lam) and gates
              r, i = sigmoid of a matrix per block of channels times u;  output projection of S y
  mlstm       S <- e^f S + e^i k v^T per head with log gates f, i, a normaliser and a running maximum; the heads' outputs divided by
              their root mean square, times a sigmoid gate
  experts     the top experts of a biased router, softmax over the chosen logits; every expert is down(silu(gate x) up x)
The embedding is scaled; the logits use the embedding table as it is.

Weights come from a model folder.  Sizes that the kernels want aligned are padded with zeros at load time: columns (width,
feed-forward, blocks of channels) to 8, attention heads to 16, mLSTM heads to 32 / 16; norms keep their true divisors.  All first
projections of a mixer are one matrix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn.functional as TF

from ..ops import functional as F
from ..ops.functional import Act, Batch, MlstmSpec, RglruSpec
from .base import ModelConfig, register_architecture
from .folder import FolderModel, round_up

RATE = -8.0          # log a = RATE * r * softplus(lam)


@dataclass
class AttnSpec:
    """Sizes of one attention mixer (``Dk`` / ``Dv``: padded head sizes); ``donor``: the layer whose cache it reads."""
    H: int
    G: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    q_temp: Optional[Tuple[float, float]]
    donor: Optional[int]

    def __post_init__(self):
        self.Dk, self.Dv = round_up(self.dim, 16), round_up(self.vdim, 16)


@register_architecture("lisorax")
class LisoraxModel(FolderModel):
    supports_kv_truncation = False           # recurrent state and the convolutions' last inputs
    graphs_with_state = True
    native_sources = ("error.cpp", "elementwise.cu", "conv_seam.cu", "short_conv.cu", "rglru.cu", "mlstm.cu", "float32.cu", "attention.cu", "attention_vd.cu",
                      "attention_decode_mma.cu", "gemm_tcgen05.cu", "gemv.cu", "gemv_bf16.cu", "gemv_mma.cu", "gemv_stream.cu", "moe.cu", "sampler.cu")

    # ------------------------------------------------------------------ configuration
    def parse_base_config(self) -> ModelConfig:
        self.parse_layers()
        j = self.gguf.config
        self.embed_scale = float((j.get("embedding") or {}).get("scale", 1.0))
        first = next((s["mixer"] for s in self.layer_specs if s["type"] == "attention"), {})
        return ModelConfig(arch=self.arch, n_layers=len(self.runs), hidden=round_up(self.width, 8), n_heads=int(first.get("heads", 0)),
                           n_kv_heads=int(first.get("kv_heads", 0)), head_dim=int(first.get("dim", 0)), vocab=int(j["vocab"]), eps=float(j["norm"]["eps"]),
                           context_length=int(j.get("context_length", 4096)))

    def parse_config(self) -> None:
        self.refuse_parallel()
        if len(self.runs) != len(self.layer_specs):
            raise ValueError(f"{self.path}: layers do not run in a loop")
        for i, s in enumerate(self.layer_specs):
            if s["type"] not in ("attention", "rglru", "mlstm"):
                raise ValueError(f"{self.path}: layer {i} has unknown type {s['type']!r}")
            if s["mlp"] is not None and s["mlp"].get("kind", "moe") != "moe":
                raise ValueError(f"{self.path}: layer {i} has unknown feed-forward {s['mlp'].get('kind')!r}")

    # ------------------------------------------------------------------ weights
    def _taps(self, name: str, H: int, d: int, dp: int) -> torch.Tensor:
        """A convolution's weights [H * d, taps] as [taps, H * dp] f32, the current token's last."""
        w = self._host(name).float()
        if w.shape[0] != H * d or not 1 <= w.shape[1] <= F.CONV_MAX_TAPS:
            raise ValueError(f"{self.path}: tensor {name!r} has shape {tuple(w.shape)}; {H * d} channels and 1 to {F.CONV_MAX_TAPS} taps are needed")
        return TF.pad(w.view(H, d, -1), (0, 0, 0, dp - d)).reshape(H * dp, -1).t().contiguous().to(self.device)

    def _attention(self, p: str, i: int, m: dict) -> Dict[str, object]:
        temp, donor = m.get("q_temp"), m.get("kv_from")
        s = AttnSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), float(m.get("softcap") or 0.0),
                     (float(temp["coef"]), float(temp["every"])) if temp else None, int(donor) if donor is not None else None)
        if s.H % s.G:
            raise ValueError(f"{p}: {s.H} heads are not a multiple of {s.G} key / value heads")
        if max(s.Dk, s.Dv) > 256:
            raise ValueError(f"{p}: head sizes {s.dim} / {s.vdim} are above 256")
        parts = [("q", s.H, s.dim, s.Dk)]
        if s.donor is None:
            parts += [("k", s.G, s.dim, s.Dk), ("v", s.G, s.vdim, s.Dv)]
        else:
            src = self.layers[s.donor].get("attn") if 0 <= s.donor < i else None
            if src is None or src.donor is not None or (src.G, src.dim, src.vdim) != (s.G, s.dim, s.vdim):
                raise ValueError(f"{p}: layer {s.donor} has no keys and values of these sizes for layer {i}")
        return {"attn": s, "proj": self._qw(torch.cat([self._heads(p + x, *z) for x, *z in parts]), p + "proj"),
                "conv": torch.cat([self._taps(f"{p}{x}.conv", *z) for x, *z in parts], 1), "bias": (self._vec(p + "r1", s.H), self._vec(p + "r2", s.H)),
                "pb": self._vec(p + "pb", s.H), "wo": self._out(p + "o", s.H, s.vdim, s.Dv)}

    def _rglru(self, p: str, m: dict) -> Dict[str, object]:
        s = RglruSpec(int(m["width"]), int(m["blocks"]))
        if s.width % s.blocks:
            raise ValueError(f"{p}: {s.width} channels are not a multiple of {s.blocks} blocks")
        B, n, b = s.blocks, s.size, s.block
        gates = torch.cat([TF.pad(self._host(p + x).view(B, n, n), (0, b - n, 0, b - n)) for x in ("ra", "ri")], 1)
        bias = torch.stack([self._head_vec(f"{p}{x}.b", B, n, b) for x in ("ra", "ri")])
        rate = RATE * TF.softplus(self._head_vec(p + "lam", B, n, b).double())
        vec = [self._head_vec(p + x, B, n, b) for x in ("y.b", "x.b", "conv.b")]
        return {"rglru": s, "proj": self._qw(torch.cat([self._heads(p + x, B, n, b) for x in ("y", "x")]), p + "proj"),
                "proj_b": torch.cat(vec[:2]).to(self.device).contiguous(), "conv": self._taps(p + "conv", B, n, b), "conv_b": vec[2].to(self.device).contiguous(),
                "gates": self._qw(gates, p + "gates"), "gate_b": bias.to(self.device).contiguous(), "rate": rate.float().to(self.device).contiguous(),
                "wo": self._out(p + "o", B, n, b)}

    def _mlstm(self, p: str, m: dict) -> Dict[str, object]:
        D = self.cfg.hidden
        s = MlstmSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
        if max(s.D, s.E) > 256:
            raise ValueError(f"{p}: head sizes {s.dim} / {s.vdim} are above 256")
        parts = [self._heads(p + "q", s.H, s.dim, s.D), self._heads(p + "k", s.H, s.dim, s.D), self._heads(p + "v", s.H, s.vdim, s.E),
                 self._heads(p + "g", s.H, s.vdim, s.E), self._mat(p + "i", cols=D), self._mat(p + "f", cols=D)]
        ends = [0]
        for w in parts:
            ends.append(ends[-1] + w.shape[0])
        proj = self._qw(torch.cat(parts), p + "proj")
        return {"mlstm": s, "proj": proj, "main": self._rows(proj, 0, ends[4]), "gates": self._rows(proj, ends[4], ends[6]), "cols": ends,
                "gate_b": torch.cat([self._vec(p + "i.b", s.H), self._vec(p + "f.b", s.H)]),
                "on": self._head_vec(p + "norm", s.H, s.vdim, s.E).to(self.device).contiguous(), "wo": self._out(p + "o", s.H, s.vdim, s.E)}

    def _moe(self, p: str, m: dict) -> Dict[str, object]:
        D, r = self.cfg.hidden, m["router"]
        E, top, ff = int(r["experts"]), int(r["top"]), round_up(int(m["expert"]["ff"]), 8)
        if not 1 <= top <= min(E, 32) or E > 1024:
            raise ValueError(f"{p}: top {top} of {E} experts (limits: 32, 1024)")
        router = self._mat(p + "router", cols=D)
        if router.shape[0] != E:
            raise ValueError(f"{p}: the router has {router.shape[0]} outputs for {E} experts")
        gate_up = torch.stack([torch.cat([self._mat(f"{p}e{e}.{x}", ff, D) for x in ("gate", "up")]) for e in range(E)])
        return {"top": top, "router": self._qw(router, p + "router"), "router_b": self._vec(p + "router.b", E), "gate_up": self._qw(gate_up, p + "gate_up"),
                "down": self._qw(torch.stack([self._mat(f"{p}e{e}.down", D, ff) for e in range(E)]), p + "down")}

    def load_weights(self) -> None:
        if self.kv_dtype == torch.float8_e4m3fn:
            raise ValueError("Lisorax has no 8-bit KV cache")
        D = self.cfg.hidden
        if self.device.type == "cuda":
            self.kv_dtype = self.compute_dtype          # bf16 pages, or f32 pages in a 32-bit run
        self.tok_emb = self._qw(self._mat("embed", cols=D), "embed")
        self.out_norm = self._vec("final.norm", D)
        self.layers: List[Dict[str, object]] = []
        for i, s in enumerate(self.layer_specs):
            p, m = f"l{i}.", s["mixer"]
            L = {"norm1": self._vec(p + "norm1", D), "canon": self._taps(p + "canon1", 1, self.width, D), "mlp": None}
            L.update(self._attention(p + "mix.", i, m) if s["type"] == "attention" else self._rglru(p + "mix.", m) if s["type"] == "rglru" else
                     self._mlstm(p + "mix.", m))
            if s["mlp"] is not None:
                L["mlp"] = self._moe(p + "mlp.", s["mlp"])
            self.layers.append(L)
        self._make_state()

    # ------------------------------------------------------------------ cache and state
    def _make_state(self) -> None:
        """One f32 row per sequence slot for everything that is carried from token to token, cut into views per layer: ``canon`` and
        ``conv`` (the convolutions' last inputs, oldest first), ``S`` (the recurrence), ``n`` and ``m`` (mLSTM)."""
        shapes: List[Dict[str, tuple]] = []
        for L in self.layers:
            d: Dict[str, tuple] = {"canon": (L["canon"].shape[0] - 1, self.cfg.hidden)}
            if "conv" in L:
                d["conv"] = (L["conv"].shape[0] - 1, L["conv"].shape[1])
            if "rglru" in L:
                d["S"] = (L["rglru"].W,)
            elif "mlstm" in L:
                s = L["mlstm"]
                d.update(S=(s.H, s.E, s.D), n=(s.H, s.D), m=(s.H,))
            shapes.append(d)
        total = sum(round_up(torch.Size(z).numel(), 4) for d in shapes for z in d.values())
        self.state = torch.zeros((max(self.max_seqs, 1), max(total, 4)), dtype=torch.float32, device=self.device)
        self.carried: List[Dict[str, torch.Tensor]] = []
        at = 0
        for d in shapes:
            views = {}
            for name, z in d.items():
                n = torch.Size(z).numel()
                views[name] = self.state[:, at:at + n].unflatten(1, z)
                at += round_up(n, 4)
            self.carried.append(views)

    def recurrent_state_tensors(self) -> list:
        return [self.state]

    def reset_recurrent_state(self, slot: int) -> None:
        self.state[slot].zero_()

    def kv_layer_shapes(self):
        return [(L["attn"].G, L["attn"].Dk, L["attn"].Dv) if "attn" in L else None for L in self.layers]

    def kv_donors(self) -> Dict[int, int]:
        return {i: L["attn"].donor for i, L in enumerate(self.layers) if "attn" in L and L["attn"].donor is not None}

    # ------------------------------------------------------------------ execution
    def _mid(self, T: int) -> torch.dtype:
        """Type of what a product hands to the next step: f32, or bf16 for prompts."""
        return torch.bfloat16 if self.bf16 and T > F.GEMV_MAX_M else torch.float32

    @property
    def _act_dtype(self) -> torch.dtype:
        return self.compute_dtype if self.device.type == "cuda" else torch.float32

    def attention_mixer(self, a: Act, L, i: int, batch: Batch) -> torch.Tensor:
        """Projections, short convolutions, cache write and attention -> ``[T, H * Dv]``; a layer with a donor writes nothing."""
        s = L["attn"]
        y = F.linear(a, L["proj"], out_dtype=self._mid(batch.T))
        caches = (self.kv.k[i], self.kv.v[i])
        own = dict(k_cache=caches[0], v_cache=caches[1]) if s.donor is None else {}
        q = F.conv_qkv_cache(y, L["conv"], self.carried[i]["conv"], batch, nq=s.H * s.Dk, dtype=caches[0].dtype, q_temp=s.q_temp, **own)
        return F.attention(q.view(batch.T, s.H, s.Dk), *caches, batch, scale=s.scale, Hq=s.H, Hkv=s.G, Dh=s.Dk, Dv=s.Dv, softcap=s.softcap,
                           log_bias=L["bias"], sigmoid_bias=L["pb"])

    def rglru_mixer(self, a: Act, L, i: int, batch: Batch) -> torch.Tensor:
        """Both branches, convolution, gates and recurrence -> ``[T, W]``."""
        y, c = F.linear(a, L["proj"], bias=L["proj_b"], out_dtype=self._mid(batch.T)), self.carried[i]
        return F.rglru(y, L["rglru"], L["conv"], L["conv_b"], L["gates"], L["gate_b"], L["rate"], c["conv"], c["S"], batch, dtype=self._act_dtype)

    def mlstm_mixer(self, a: Act, L, i: int, batch: Batch) -> torch.Tensor:
        """Projections and the matrix memory with its norm and gate -> ``[T, H * E]``.  The gates' projections stay f32."""
        s, cols, c = L["mlstm"], L["cols"], self.carried[i]
        if self._mid(batch.T) == torch.float32:
            y = F.linear(a, L["proj"], out_dtype=torch.float32)
            z = y[:, cols[4]:]
        else:
            y, z = F.linear(a, L["main"], out_dtype=torch.bfloat16), F.linear(a, L["gates"], out_dtype=torch.float32)
        return F.mlstm(y, s, tuple(cols[:4]), z, L["gate_b"], L["on"], c["S"], c["n"], c["m"], batch, eps=self.cfg.eps, dtype=self._act_dtype)

    def experts(self, a: Act, m) -> F.MoeParts:
        """The chosen experts' rows; they are summed by the seam that follows."""
        logits = F.linear(a, m["router"], bias=m["router_b"], out_dtype=torch.float32)
        ids, w = F.route_topk_softmax(logits, m["top"])
        return F.moe_expert_parts(a, ids, w, m["gate_up"], m["down"], act="swiglu")

    def forward_batch(self, batch: Batch, want_logits: bool = True) -> Optional[torch.Tensor]:
        c, n, dt = self.cfg, self.width, self.compute_dtype
        h = self.inject_pending_embeddings(F.embed(self.tok_emb, batch.tokens, self.embed_scale))
        want_logits = want_logits and batch.last_idx.numel() > 0
        every_row = batch.is_decode and batch.last_idx.numel() == batch.T     # decode: all rows give logits, in their order
        y, parts, last = None, None, len(self.layers) - 1
        for i, L in enumerate(self.layers):
            h, v, x = F.conv_seam(h, c.eps, n, w=L["norm1"], y=y, parts=parts, taps=L["canon"], state=self.carried[i]["canon"], batch=batch,
                                  plain=L["mlp"] is not None, dtype=dt)
            mixer = self.attention_mixer if "attn" in L else self.rglru_mixer if "rglru" in L else self.mlstm_mixer
            o = mixer(Act(x), L, i, batch)
            if i == last:
                if not want_logits:
                    return None
                if not every_row:                       # past the last cache and state only the wanted rows matter
                    o, h, v = (t.index_select(0, batch.last_idx) if t is not None else None for t in (o, h, v))
            y = F.linear(Act(o), L["wo"], out_dtype=self._mid(o.shape[0]))
            parts = self.experts(Act(v), L["mlp"]) if L["mlp"] is not None else None
        if not want_logits:
            return None
        if last < 0:
            h = h.index_select(0, batch.last_idx)
        _, v, _ = F.conv_seam(h, c.eps, n, w=self.out_norm, y=y, parts=parts, dtype=dt)
        return F.linear(Act(v), self.tok_emb, out_dtype=torch.float32)
