"""Kegetar: a hybrid in which a layer's mixer is either attention whose values are its own keys, or windowed attention and gated
linear attention side by side; dense or grouped expert feed-forwards; norms on the sublayers' outputs only.

A layer:  x += m norm1(mixer(x));  x += m norm2(ff(x))  with RMS norms whose weights are offsets from 1 (factor 1 + w); the
sublayers read the stream itself.  The stream starts as the token's embedding plus that of the pair (previous token, token).
  parallel    (norm(left) + norm(right)) / 2
    left      grouped-query attention, per-head RMS norms on queries and keys, rotation of neighbouring pairs with YaRN scaling,
              a sliding window beside which the first tokens stay visible, a sigmoid gate per output column
    right     gated linear attention: S <- diag(a) S + k v^T per head, a = sigmoid(z)^(1/tau) per key channel, o = S^T q, divided by
              its root mean square, times silu of a gate
  attention   queries and keys normed over all heads together, values = keys ahead of the norm, a distance bias per head, a
              sliding window.  The cache holds one row per token for keys and values (ops/functional.py: joint_norm_cache)
  dense       down(gelu(gate x) up x) with biases
  moe         softmax routing with a choice correction, restricted to the best groups of neighbours; some of the entries are
              identity experts, which hand the input on; clamped expert activation; a shared expert of every token
A layer may use another one's weights; its cache and state are its own.

Weights come from a model folder.  Sizes that the kernels want aligned are padded with zeros at load time: columns (width,
feed-forward, ranks) to 8, attention heads to 16, linear-attention heads to 32 / 16; norms keep their true divisors.  All first
projections of a mixer are one matrix.  m is folded into the norms' weights.  The shared expert is cut into slices of the
experts' size, which run as the first experts of every token, so that one grouped product serves both.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn.functional as TF

from ..ops import functional as F
from ..ops.functional import Act, Batch, GatedLinearSpec, RopeSpec
from .base import ModelConfig, register_architecture
from .folder import FolderModel, round_up


@dataclass
class AttnSpec:
    """Sizes of one attention mixer (``Dk`` / ``Dv``: padded head sizes)."""
    H: int
    G: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int

    def __post_init__(self):
        self.Dk, self.Dv = round_up(self.dim, 16), round_up(self.vdim, 16)


@dataclass
class MoeSpec:
    E: int                   # routed experts with tensors
    entries: int             # router outputs: experts and identity experts
    top: int
    groups: int
    keep: int
    shared: int              # slices of the shared expert (0: none)
    clamp: Tuple[float, float, int]


@register_architecture("kegetar")
class KegetarModel(FolderModel):
    supports_kv_truncation = False           # recurrent state
    graphs_with_state = True
    native_sources = ("error.cpp", "elementwise.cu", "post_norm.cu", "gated_linear.cu", "float32.cu", "attention.cu", "attention_vd.cu",
                      "attention_decode_mma.cu", "gemm_tcgen05.cu", "gemv.cu", "gemv_bf16.cu", "gemv_mma.cu", "gemv_stream.cu", "moe.cu", "sampler.cu")

    # ------------------------------------------------------------------ configuration
    def parse_base_config(self) -> ModelConfig:
        self.parse_layers()
        j = self.gguf.config
        self.residual_mult = float(j.get("residual_mult", 1.0))
        self.pairs = j["embedding"]["bigram"]
        first = self.layer_specs[0]["mixer"] if self.layer_specs else {}
        first = first.get("left", first)
        return ModelConfig(arch=self.arch, n_layers=len(self.runs), hidden=round_up(self.width, 8), n_heads=int(first.get("heads", 0)),
                           n_kv_heads=int(first.get("kv_heads", 0)), head_dim=int(first.get("dim", 0)), vocab=int(j["vocab"]), eps=float(j["norm"]["eps"]),
                           context_length=int(j.get("context_length", 4096)))

    def parse_config(self) -> None:
        self.refuse_parallel()
        for i, s in enumerate(self.layer_specs):
            if s["type"] not in ("parallel", "attention"):
                raise ValueError(f"{self.path}: layer {i} has unknown type {s['type']!r}")
            if s["mlp"] is not None and s["mlp"].get("kind", "dense") not in ("dense", "moe"):
                raise ValueError(f"{self.path}: layer {i} has unknown feed-forward {s['mlp'].get('kind')!r}")

    def weights_of(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = []
        while self.layer_specs[i].get("weights_of") is not None:
            seen.append(i)
            i = int(self.layer_specs[i]["weights_of"])
            if not 0 <= i < len(self.layer_specs) or i in seen:
                raise ValueError(f"{self.path}: layer {seen[0]} has no layer to take its weights from")
        if any(self.layer_specs[k]["type"] != self.layer_specs[i]["type"] or self.layer_specs[k]["mlp"] != self.layer_specs[i]["mlp"]
               or self.layer_specs[k]["mixer"] != self.layer_specs[i]["mixer"] for k in seen):
            raise ValueError(f"{self.path}: layer {seen[0]} differs from layer {i}, whose weights it uses")
        return i

    # ------------------------------------------------------------------ weights
    def _post(self, name: str) -> torch.Tensor:
        """m (1 + w) of a norm stored as its offset from 1 (0 in the padding)."""
        w = (self._host(name).float() + 1.0) * self.residual_mult
        return TF.pad(w, (0, self.cfg.hidden - w.shape[0])).to(self.device).contiguous()

    def _attn_spec(self, p: str, m: dict, vdim: int) -> AttnSpec:
        mask = m.get("mask") or {}
        s = AttnSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), vdim, float(m["scale"]), int(mask.get("size", 0)), int(mask.get("keep_first", 0)))
        if s.H % s.G:
            raise ValueError(f"{p}: {s.H} heads are not a multiple of {s.G} key / value heads")
        if max(s.Dk, s.Dv) > 256:
            raise ValueError(f"{p}: head sizes {s.dim} / {s.vdim} are above 256")
        return s

    def _parallel(self, p: str, m: dict) -> Dict[str, object]:
        D, left, right = self.cfg.hidden, m["left"], m["right"]
        a = self._attn_spec(p, left, int(left["vdim"]))
        g = GatedLinearSpec(int(right["heads"]), int(right["dim"]), int(right["vdim"]), float(right["tau"]))
        if max(g.D, g.E) > 256:
            raise ValueError(f"{p}: head sizes {g.dim} / {g.vdim} are above 256")
        turn = left.get("rot") or {"dims": 0, "base": 1.0}
        key = (int(turn["dims"]), float(turn["base"]), tuple(sorted((turn.get("scaling") or {}).items())))
        if key[0] % 2 or key[0] > a.dim:
            raise ValueError(f"{p}: {key[0]} of {a.dim} dimensions cannot be rotated in pairs")
        if key not in self.turns:                      # layers with the same rotation share one table per step
            freq, gain = F.yarn_freqs(key[0], key[1], turn.get("scaling"), self.device)
            self.turns[key] = RopeSpec(key[0], key[1], mode=1, attn_factor=gain, freq=freq) if key[0] else None
        rank = self._host(p + "right.a1").shape[0]
        rp = round_up(rank, 8)
        parts = [self._heads(p + "left.q", a.H, a.dim, a.Dk), self._heads(p + "left.k", a.G, a.dim, a.Dk), self._heads(p + "left.v", a.G, a.vdim, a.Dv),
                 self._heads(p + "left.g", a.H, a.vdim, a.Dv), self._heads(p + "right.q", g.H, g.dim, g.D), self._heads(p + "right.k", g.H, g.dim, g.D),
                 self._heads(p + "right.v", g.H, g.vdim, g.E), self._heads(p + "right.g", g.H, g.vdim, g.E), self._mat(p + "right.a1", rows=rp, cols=D)]
        ends = [0]
        for w in parts:
            ends.append(ends[-1] + w.shape[0])
        w2 = TF.pad(self._mat(p + "right.a2", cols=rp).view(g.H, g.dim, rp), (0, 0, 0, g.D - g.dim)).reshape(g.H * g.D, rp)
        return {"left": a, "right": g, "rope": self.turns[key], "proj": self._qw(torch.cat(parts), p + "proj"), "cols": ends,
                "qn": self._vec(p + "left.q.norm", a.Dk), "kn": self._vec(p + "left.k.norm", a.Dk), "wo": self._out(p + "left.o", a.H, a.vdim, a.Dv),
                "w2": self._qw(w2, p + "right.a2"), "zb": self._head_vec(p + "right.a2.b", g.H, g.dim, g.D).to(self.device).contiguous(),
                "on": self._vec(p + "right.norm", g.E), "wo2": self._out(p + "right.o", g.H, g.vdim, g.E),
                "branch": (self._vec(p + "left.out", D), self._vec(p + "right.out", D))}

    def _attention(self, p: str, m: dict) -> Dict[str, object]:
        s = self._attn_spec(p, m, int(m["dim"]))
        w = torch.cat([self._heads(p + "q", s.H, s.dim, s.Dk), self._heads(p + "k", s.G, s.dim, s.Dk)])
        b = torch.cat([self._head_vec(p + "q.b", s.H, s.dim, s.Dk), self._head_vec(p + "k.b", s.G, s.dim, s.Dk)])
        kn = self._head_vec(p + "k.norm", s.G, s.dim, s.Dk).view(s.G, 1, s.Dk).expand(s.G, s.H // s.G, s.Dk).reshape(-1)
        return {"attn": s, "proj": self._qw(w, p + "qk"), "bias": b.to(self.device).contiguous(),
                "qn": (self._head_vec(p + "q.norm", s.H, s.dim, s.Dk) * kn).to(self.device).contiguous(), "slopes": F.alibi_slopes(s.H, self.device),
                "wo": self._out(p + "o", s.H, s.dim, s.Dk)}

    def _dense(self, p: str, m: dict) -> Dict[str, object]:
        D, ff = self.cfg.hidden, round_up(int(m["ff"]), 8)
        return {"gate_up": self._qw(torch.cat([self._mat(p + n, ff, D) for n in ("gate", "up")]), p + "gate_up"),
                "gate_up_b": torch.cat([self._vec(p + n, ff) for n in ("gate.b", "up.b")]),
                "down": self._qw(self._mat(p + "down", D, ff), p + "down"), "down_b": self._vec(p + "down.b", D)}

    def _moe(self, p: str, m: dict) -> Dict[str, object]:
        D, r, shared = self.cfg.hidden, m["router"], m.get("shared")
        E, ff = int(r["experts"]), round_up(int(m["expert"]["ff"]), 8)
        entries, groups = E + int(r.get("identity") or 0), r.get("groups") or {"count": 1, "keep": 1}
        slices = -(-int(shared["ff"]) // ff) if shared else 0
        limit = float(m["expert"]["limit"])
        s = MoeSpec(E, entries, int(r["top"]), int(groups["count"]), int(groups["keep"]), slices, (limit, float(shared["limit"]) if shared else limit, slices))
        if s.top > 32 or E + slices > 1024 or entries > 1024 or entries % s.groups or not s.top <= s.keep * (entries // s.groups) <= entries:
            raise ValueError(f"{p}: top {s.top} of {entries} entries in {s.keep} of {s.groups} groups with {slices} shared slices")
        router = self._mat(p + "router", cols=D)
        if router.shape[0] != entries:
            raise ValueError(f"{p}: the router has {router.shape[0]} outputs for {entries} experts and identity experts")
        gate = [self._mat(f"{p}e{e}.gate", ff, D) for e in range(E)]
        up = [self._mat(f"{p}e{e}.up", ff, D) for e in range(E)]
        down = [self._mat(f"{p}e{e}.down", D, ff) for e in range(E)]
        if shared:
            # the activation is separate per feature, so the shared expert is the sum of its slices of ff features
            sg, su = (self._mat(f"{p}shared.{n}", slices * ff, D) for n in ("gate", "up"))
            gate, up = list(sg.split(ff)) + gate, list(su.split(ff)) + up
            down = list(self._mat(p + "shared.down", D, slices * ff).split(ff, 1)) + down
        return {"moe": s, "router": self._qw(router, p + "router"), "correction": self._vec(p + "correction", entries),
                "gate_up": self._qw(torch.stack([torch.cat([g, u]) for g, u in zip(gate, up)]), p + "gate_up"),
                "down": self._qw(torch.stack(down), p + "down")}

    def load_weights(self) -> None:
        if self.kv_dtype == torch.float8_e4m3fn:
            raise ValueError("Kegetar has no 8-bit KV cache")
        D = self.cfg.hidden
        if self.device.type == "cuda":
            self.kv_dtype = self.compute_dtype          # bf16 pages, or f32 pages in a 32-bit run
        self.tok_emb, self.pair_emb = self._qw(self._mat("embed", cols=D), "embed"), self._qw(self._mat("bigram", cols=D), "bigram")
        if self.pair_emb.rows != int(self.pairs["buckets"]) + 1:
            raise ValueError(f"{self.path}: bigram has {self.pair_emb.rows} rows, {self.pairs['buckets']} buckets need one more")
        self.lm_head = self._qw(self._mat("head", cols=D), "head")
        self.out_norm = TF.pad(self._host("final.norm").float() + 1.0, (0, D - self.width)).to(self.device).contiguous()
        self.turns: Dict[tuple, Optional[RopeSpec]] = {}
        made: Dict[int, Dict[str, object]] = {}
        for i in sorted({self.weights_of(i) for i in range(len(self.layer_specs))}):
            p, s = f"l{i}.", self.layer_specs[i]
            L = made[i] = {"norm1": self._post(p + "norm1"), "mlp": None}
            L.update(self._parallel(p + "mix.", s["mixer"]) if s["type"] == "parallel" else self._attention(p + "mix.", s["mixer"]))
            if s["mlp"] is not None:
                L["norm2"] = self._post(p + "norm2")
                L["mlp"] = (self._moe if s["mlp"].get("kind", "dense") == "moe" else self._dense)(p + "mlp.", s["mlp"])
        self.layers: List[Dict[str, object]] = [made[self.weights_of(i)] for i in range(len(self.layer_specs))]
        self._make_state()

    # ------------------------------------------------------------------ cache and state
    def _make_state(self) -> None:
        """One f32 row per sequence slot for the matrices of all linear-attention runs (``memory``: views into it), and the last
        token of every slot's sequence (-1: none yet)."""
        off, at = 0, []
        for i, _ in self.runs:
            g = self.layers[i].get("right")
            at.append(off)
            off += g.H * g.E * g.D if g is not None else 0
        self.state = torch.zeros((max(self.max_seqs, 1), max(off, 4)), dtype=torch.float32, device=self.device)
        self.last_token = torch.full((max(self.max_seqs, 1),), -1, dtype=torch.int32, device=self.device)
        self.memory = []
        for (i, _), o in zip(self.runs, at):
            g = self.layers[i].get("right")
            self.memory.append(self.state[:, o:o + g.H * g.E * g.D].unflatten(1, (g.H, g.E, g.D)) if g is not None else None)

    def recurrent_state_tensors(self) -> list:
        return [self.state, self.last_token]

    def reset_recurrent_state(self, slot: int) -> None:
        self.state[slot].zero_()
        self.last_token[slot] = -1

    def kv_layer_shapes(self):
        """An attention layer caches one row [keys | factor] per token and no separate values."""
        out = []
        for i, _ in self.runs:
            s = self.layers[i].get("left")
            out.append((s.G, s.Dk, s.Dv) if s is not None else (1, self.layers[i]["attn"].G * self.layers[i]["attn"].Dk + 8, 0))
        return out

    def kv_window_layers(self) -> Dict[int, int]:
        """Layers that never look behind their window (kept first tokens stay in the cache)."""
        specs = [self.layers[i].get("left") or self.layers[i]["attn"] for i, _ in self.runs]
        return {r: s.window for r, s in enumerate(specs) if s.window and not s.keep_first}

    # ------------------------------------------------------------------ execution
    def _mid(self, T: int) -> torch.dtype:
        """Type of what a product hands to the next step: f32, or bf16 for prompts."""
        return torch.bfloat16 if self.bf16 and T > F.GEMV_MAX_M else torch.float32

    def parallel_mixer(self, a: Act, L, run: int, batch: Batch) -> Tuple[torch.Tensor, torch.Tensor]:
        """Both halves ahead of their output projections: ``[T, H * Dv]`` (attention), ``[T, H * E]`` (linear attention)."""
        s, g, c, T = L["left"], L["right"], L["cols"], batch.T
        y = F.linear(a, L["proj"], out_dtype=self._mid(T))
        o2 = F.gated_linear(y, g, (c[4], c[5], c[6], c[7], c[8]), L["w2"], L["zb"], L["on"], self.memory[run], batch, eps=self.cfg.eps,
                            dtype=self.compute_dtype if self.device.type == "cuda" else torch.float32)
        if self.kv.is_window_layer(run):
            batch = batch.windowed()
        q = F.qkv_rope_cache(y[:, :c[1]].view(T, s.H, s.Dk), y[:, c[1]:c[2]].view(T, s.G, s.Dk), y[:, c[2]:c[3]].view(T, s.G, s.Dv), Hq=s.H, Hkv=s.G,
                             Dh=s.Dk, Dv=s.Dv, norm_n=s.dim, batch=batch, k_cache=self.kv.k[run], v_cache=self.kv.v[run], rope=L["rope"], qn=L["qn"],
                             kn=L["kn"], eps=self.cfg.eps)
        o = F.attention(q, self.kv.k[run], self.kv.v[run], batch, scale=s.scale, Hq=s.H, Hkv=s.G, Dh=s.Dk, Dv=s.Dv, window=s.window,
                        keep_first=s.keep_first, gate=y[:, c[3]:c[4]])
        return o, o2

    def attention_mixer(self, a: Act, L, run: int, batch: Batch) -> torch.Tensor:
        """Attention ahead of its output projection, ``[T, H * Dk]``."""
        s = L["attn"]
        if self.kv.is_window_layer(run):
            batch = batch.windowed()
        nq, nk = s.H * s.Dk, s.G * s.Dk
        y = F.linear(a, L["proj"], bias=L["bias"], out_dtype=self._mid(batch.T))
        q = F.joint_norm_cache(y, L["qn"], self.kv.k[run], batch, nq=nq, nk=nk, q_n=s.H * s.dim, k_n=s.G * s.dim, eps=self.cfg.eps)
        return F.attention(q.view(batch.T, s.H, s.Dk), self.kv.k[run], self.kv.k[run], batch, scale=s.scale, Hq=s.H, Hkv=s.G, Dh=s.Dk,
                           window=s.window, slopes=L["slopes"], own_values=True)

    def feed_forward(self, x: torch.Tensor, m):
        if "moe" not in m:
            g = F.linear(Act(x), m["gate_up"], bias=m["gate_up_b"], act="geglu", out_dtype=torch.bfloat16 if self.bf16 else torch.float32)
            return F.linear(Act(g), m["down"], bias=m["down_b"], out_dtype=self._mid(x.shape[0]))
        s = m["moe"]
        logits = F.linear(Act(x), m["router"], out_dtype=torch.float32)
        ids, w = F.route_softmax_groups(logits, m["correction"], s.top, groups=s.groups, keep=s.keep, n_real=s.E, n_always=s.shared)
        return F.moe_expert_parts(Act(x), ids, w, m["gate_up"], m["down"], act="swiglu_oai", clamp=s.clamp, identity=True)

    def forward_batch(self, batch: Batch, want_logits: bool = True) -> Optional[torch.Tensor]:
        c, n, dt = self.cfg, self.width, self.compute_dtype
        h, x = F.embed_pairs(self.tok_emb, self.pair_emb, batch, self.last_token, mul_prev=int(self.pairs["mul_prev"]),
                             mul_cur=int(self.pairs["mul_cur"]), dtype=dt)
        if self._pending_embeddings:
            h = self.inject_pending_embeddings(h)
            x = h.to(x.dtype)
        want_logits = want_logits and batch.last_idx.numel() > 0
        every_row = batch.is_decode and batch.last_idx.numel() == batch.T     # decode: all rows give logits, in their order
        last = len(self.runs) - 1
        if last < 0:
            x = F.post_norm_seam(h, c.eps, n, pre=self.out_norm, dtype=dt)
        for r, (i, _) in enumerate(self.runs):
            L = self.layers[i]
            if "left" in L:
                o, o2 = self.parallel_mixer(Act(x), L, r, batch)
            else:
                o, o2 = self.attention_mixer(Act(x), L, r, batch), None
            if r == last:
                if not want_logits:
                    return None
                if not every_row:                       # past the last cache and state only the wanted rows matter
                    o, o2, h = (t.index_select(0, batch.last_idx) if t is not None else None for t in (o, o2, h))
            mid, ff = self._mid(o.shape[0]), L["mlp"]
            final = self.out_norm if r == last else None
            y = F.linear(Act(o), L["wo"], out_dtype=mid)
            both = dict(z=F.linear(Act(o2), L["wo2"], out_dtype=mid), branch=L["branch"], mix=0.5) if o2 is not None else {}
            x = F.post_norm_seam(h, c.eps, n, y=y, post=L["norm1"], pre=final if ff is None else None, dtype=dt, **both)
            if ff is not None:
                x = F.post_norm_seam(h, c.eps, n, y=self.feed_forward(x, ff), post=L["norm2"], pre=final, dtype=dt)
        if last < 0:
            if not want_logits:
                return None
            x = x.index_select(0, batch.last_idx)
        return F.linear(Act(x), self.lm_head, out_dtype=torch.float32)
