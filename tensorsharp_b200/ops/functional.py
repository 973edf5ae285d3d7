"""The op set the model graphs are written against.

Every function has exactly two implementations: the sm_100a kernels (tensors on a CUDA
device) and the fp32 PyTorch restatement in :mod:`reference` (tensors on the CPU), which
is both the CPU backend and the numerical oracle.  On a CUDA device there is no fallback:
a missing kernel library raises.

Data conventions
  * the residual stream ``h`` is float32 ``[T, D]`` (T = packed tokens of all sequences)
  * :class:`Act` carries a normalised activation as bf16 and / or as int8 groups of 32
    with ``(scale, sum)`` pairs, which is what the quantised GEMV consumes
  * the KV cache is paged: ``k_cache / v_cache`` are ``[n_slots, Hkv, Dh]``
"""
from __future__ import annotations

import math
import os
from dataclasses import dataclass, field
from typing import Optional, Tuple

import torch

from ..quant.qweight import QuantWeight
from . import reference as ref

GEMV_MAX_M = 16   # "small batch": token count up to which the models take their decode-style paths (int8 activations, mailbox exchanges)
# Dense projections of 9 to 16 rows go to the tensor-core GEMM on the bf16 weight copy all the same: measured on the
# Qwen3-4B shape at batch 16, 10.95 ms per step with the weight-streaming GEMVs against 8.15 ms (TSB_GEMV_MAX_M moves it)
DENSE_GEMV_MAX_M = min(GEMV_MAX_M, int(os.environ.get("TSB_GEMV_MAX_M", "8")))


@dataclass
class Act:
    """A (normalised) activation in the forms the linear kernels consume."""
    b: Optional[torch.Tensor] = None      # [T, K] bf16 (CUDA) or f32 (CPU, and CUDA models that run in 32 bits)
    q: Optional[torch.Tensor] = None      # [T, K] int8
    ds: Optional[torch.Tensor] = None     # [T, K/32, 2] f32 (scale, sum)

    @property
    def T(self) -> int:
        return (self.b if self.b is not None else self.q).shape[0]


@dataclass
class RopeSpec:
    rot_dim: int
    theta_base: float
    mode: int = 0                 # 0 NeoX, 1 adjacent pairs
    freq_scale: float = 1.0
    ext_factor: float = 0.0
    attn_factor: float = 1.0
    corr_lo: float = 0.0
    corr_hi: float = 0.0
    freq_factors: Optional[torch.Tensor] = None
    # frequency of every pair (float64, on the compute device) in place of the base and scaling above; cos and sin are
    # multiplied by attn_factor
    freq: Optional[torch.Tensor] = None


@dataclass
class Batch:
    """Packed batch metadata (all int tensors live on the compute device)."""
    tokens: torch.Tensor          # [T] int32
    positions: torch.Tensor       # [T] int32
    slots: torch.Tensor           # [T] int64 flat KV slot per token
    cu_q: torch.Tensor            # [B+1] int32
    kv_lens: torch.Tensor         # [B] int32 (cache length after this step)
    block_table: torch.Tensor     # [B, P] int32
    last_idx: torch.Tensor        # int64 rows of the packed dim whose logits are wanted ([B]: each sequence's last token)
    seq_slots: torch.Tensor       # [B] int64 recurrent-state slot per sequence
    max_q_len: int
    max_kv_len: int
    is_decode: bool               # every sequence contributes exactly one query
    page_size: int
    # host copies for the CPU path and for planning
    h_cu_q: Tuple[int, ...] = ()
    h_kv_lens: Tuple[int, ...] = ()
    cache: dict = field(default_factory=dict)   # per-forward memo (RoPE tables); cleared by the step runner
    # Sliding-window layers that keep a ring of pages (runtime/paged_kv.py): their own slot per token and their own block
    # table (logical page -> physical page of the ring).  None when the pool keeps every page of every layer.
    slots_w: Optional[torch.Tensor] = None
    block_table_w: Optional[torch.Tensor] = None

    def windowed(self) -> "Batch":
        """The view of this batch that a sliding-window layer uses: the same tokens and lengths with the ring's slots
        and block table in place of the full ones (the batch itself when the pool has no ring)."""
        if self.block_table_w is None:
            return self
        w = self.cache.get("_windowed")
        if w is None or w.slots is not self.slots_w:
            import dataclasses
            w = dataclasses.replace(self, slots=self.slots_w, block_table=self.block_table_w, slots_w=None, block_table_w=None,
                                    cache=self.cache)
            self.cache["_windowed"] = w
        return w

    @property
    def B(self) -> int:
        return self.kv_lens.shape[0]

    @property
    def T(self) -> int:
        return self.tokens.shape[0]


def _k():
    from . import kernels
    return kernels


# --------------------------------------------------------------------------------------------
def embed(w: QuantWeight, ids: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    """Token embedding lookup with on-the-fly dequantisation -> f32 [T, D]."""
    if w.device.type == "cuda":
        return _k().gather_rows(w, ids.to(torch.int32), scale, torch.float32)
    return w.dequantize()[ids.long()] * scale


def norm(h: torch.Tensor, w: Optional[torch.Tensor], eps: float, *, delta: Optional[torch.Tensor] = None,
         want_q8: bool = False, want_bf16: bool = True, l2: bool = False) -> Act:
    """(h += delta, in place) then RMSNorm (or L2 norm) with optional weight."""
    if h.is_cuda:
        if delta is not None and delta.dtype != torch.bfloat16:
            h.add_(delta)
            delta = None
        yb, _, yq, yds = _k().rmsnorm(h, w, eps, delta=delta, want_bf16=want_bf16, want_q8=want_q8, l2=l2)
        return Act(yb, yq, yds)
    if delta is not None:
        h.add_(delta.float())
    return Act(ref.l2norm(h, eps) if l2 else ref.rmsnorm(h, w, eps))


def norm_add(x: torch.Tensor, w: Optional[torch.Tensor], eps: float, h: torch.Tensor) -> torch.Tensor:
    """Sandwich post-norm: returns h + RMSNorm(x) * w as a new f32 tensor."""
    if x.is_cuda:
        _, yf, _, _ = _k().rmsnorm(x.contiguous(), w, eps, want_bf16=False, add=h)
        return yf
    return h + ref.rmsnorm(x, w, eps)


def residual_layernorm(h: torch.Tensor, eps: float, n: int, *, y=None, post=None, add: Optional[torch.Tensor] = None, pre=None,
                       dtype: Optional[torch.dtype] = None) -> Optional[Act]:
    """The seam between two sublayers of a sandwich-normed decoder, one kernel on CUDA: ``h`` (f32 ``[T, D]``, in place)
    gains the layer norm ``post`` of the sublayer's output ``y`` (a tensor or :class:`MoeParts`) and then the vector
    ``add`` ``[D]``; returned is the layer norm ``pre`` of the new ``h`` as the next sublayer's input (None without
    ``pre``).  ``post`` / ``pre`` are (weight, bias); statistics run over the first ``n`` columns, the rest is padding."""
    if h.is_cuda:
        parts = y if isinstance(y, MoeParts) else None
        yt = parts.y if parts is not None else y
        out = _k().residual_layernorm(h, eps, n, y=yt, pos=parts.pos if parts else None, wts=parts.w if parts else None,
                                      parts=parts.k if parts else 1, post=post, add=add, pre=pre, out_dtype=dtype or torch.bfloat16)
        return Act(out) if out is not None else None
    if y is not None:
        h.add_(ref.layernorm_n(y.sum() if isinstance(y, MoeParts) else y.float(), post[0], post[1], eps, n))
    if add is not None:
        h.add_(add)
    return Act(ref.layernorm_n(h, pre[0], pre[1], eps, n)) if pre is not None else None


def parallel_seam(h: torch.Tensor, eps: float, n: int, *, y=(None, None), scale=(None, None), w=(None, None), out=(None, None),
                  outputs: int = 2, dtype: Optional[torch.dtype] = None, shift: Optional[torch.Tensor] = None,
                  state: Optional[torch.Tensor] = None, batch: Optional[Batch] = None):
    """The seam between two layers whose sublayers read the same residual (one kernel on CUDA): ``h`` (f32 ``[T, D]``) plus
    ``scale[0] * y[0] + scale[1] * y[1]`` (vectors ``[D]``; None: no such sublayer), and the next layer's inputs, the RMS
    norms of the sum with the weights ``w``.  The first input moves towards the previous token's by ``shift`` per channel;
    ``state`` (f32, a row per slot) holds that of the last token of each sequence between calls.  An output without a
    weight is the sum itself; ``out`` are buffers to write to, else the first ``outputs`` of them are made.  The norm runs
    over the first ``n`` columns, the rest is padding.  Returns (new h, first output, second output)."""
    out = list(out)
    if h.is_cuda:
        for i in range(outputs):
            if out[i] is None:
                out[i] = torch.empty(h.shape, dtype=dtype or torch.bfloat16, device=h.device)
        kw = dict(shift=shift, state=state, cu_q=batch.cu_q, seq_slots=batch.seq_slots) if shift is not None else {}
        return (_k().parallel_norm(h, eps, n, y=y, scale=scale, w=w, out=out, **kw),) + tuple(out)
    for t, s in zip(y, scale):
        if t is not None:
            h = h + s * t.float()
    rs = torch.rsqrt((h * h).sum(-1, keepdim=True) / n + eps)
    res = [h * rs * wi if wi is not None else h for wi in w]
    if shift is not None:
        v = res[0]
        before = torch.empty_like(v)
        before[1:] = v[:-1]
        for b, slot in enumerate(batch.seq_slots.tolist()):
            before[batch.h_cu_q[b]] = state[slot]
            state[slot] = v[batch.h_cu_q[b + 1] - 1]
        res[0] = v + (before - v) * shift
    for i in range(2):
        if out[i] is not None:
            out[i].copy_(res[i])
        elif i < outputs:
            out[i] = res[i]
    return h, out[0], out[1]


def post_norm_seam(h: torch.Tensor, eps: float, n: int, *, y=None, z: Optional[torch.Tensor] = None, branch=(None, None), mix: float = 1.0,
                   post: Optional[torch.Tensor] = None, pre: Optional[torch.Tensor] = None, dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """The seam of a decoder that normalises its sublayers' outputs, one kernel on CUDA: ``h`` (f32 ``[T, D]``, in place) gains
    the RMS norm of ``y`` (a tensor or :class:`MoeParts`) with the weight ``post``; with a second branch ``z`` it is the norm of
    ``mix`` times the sum of both branches' own norms (weights ``branch``).  Returns what the next product reads: ``h`` itself,
    or its RMS norm with the weight ``pre``.  Statistics run over the first ``n`` columns, the rest is padding."""
    parts = y if isinstance(y, MoeParts) else None
    if h.is_cuda:
        return _k().post_norm(h, eps, n, y=parts.y if parts else y, z=z, ids=parts.ids if parts else None, pos=parts.pos if parts else None,
                              wts=parts.w if parts else None, parts=parts.k if parts else 1, branch=branch, mix=mix, post=post, pre=pre,
                              out_dtype=dtype or torch.bfloat16)

    def rms(x):
        return x * torch.rsqrt((x * x).sum(-1, keepdim=True) / n + eps)
    if y is not None:
        x = parts.sum(h) if parts else y.float()
        if z is not None:
            x = mix * (rms(x) * branch[0] + rms(z.float()) * branch[1])
        h.add_(rms(x) * post)
    return rms(h) * pre if pre is not None else h.clone()


def conv_seam(h: torch.Tensor, eps: float, n: int, *, w: torch.Tensor, y: Optional[torch.Tensor] = None, parts: Optional["MoeParts"] = None,
              taps: Optional[torch.Tensor] = None, state: Optional[torch.Tensor] = None, batch: Optional[Batch] = None, plain: bool = True,
              dtype: Optional[torch.dtype] = None):
    """The seam of a decoder whose sublayers read one norm, one of them through a convolution over time.  ``h``
    (f32 ``[T, D]``) plus the sublayers' outputs ``y`` and the sum of ``parts``; v, the RMS norm of that with the weight ``w``; and
    v + conv(v), a causal convolution per channel with ``taps`` [K, D] (the last row is the current token's).  ``state`` (f32
    ``[slots, K - 1, D]``, oldest first) holds each sequence's last values of v between calls.  The norm runs over the first ``n``
    columns, the rest is padding.  Returns (new h, v or None without ``plain``, v + conv(v) or None without ``taps``)."""
    if h.is_cuda:
        return _k().conv_seam(h, eps, n, w=w, y=y, parts=parts, taps=taps, state=state, batch=batch, plain=plain, out_dtype=dtype or torch.bfloat16)
    if y is not None:
        h = h + y.float()
    if parts is not None:
        h = h + parts.sum()
    v = h * torch.rsqrt((h * h).sum(-1, keepdim=True) / n + eps) * w
    c = None
    if taps is not None:
        c = v + _conv_over_time(v, taps, None, state, batch)
    return h, v if plain else None, c


CONV_MAX_TAPS = 8          # of the convolutions over time below and of conv_seam


def _conv_over_time(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, batch: Batch) -> torch.Tensor:
    """CPU: causal convolution per channel over the packed rows, ``w`` [K, C]; ``state`` [slots, K - 1, C] is advanced."""
    outs = []
    for b, slot in enumerate(batch.seq_slots.tolist()):
        o, tail = ref.causal_conv1d(x[batch.h_cu_q[b]:batch.h_cu_q[b + 1]], w.t(), bias, state[slot], act_silu=False)
        state[slot] = tail
        outs.append(o)
    return torch.cat(outs, 0)


def short_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, batch: Batch, *, block: int = 0,
               dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """Causal convolution over time on every channel of a projection, no activation: ``x`` [T, C] (a view, rows may be strided),
    ``w`` [K, C] (the last row is the current token's); ``state`` f32 [slots, K - 1, C] holds each sequence's last inputs, oldest
    first.  Returns [T, C], or with ``block`` the columns in blocks of that size one below the other, [C / block * T, block]."""
    T, C = x.shape
    if x.is_cuda:
        return _k().short_conv(x, w, bias, state, batch, block=block, out_dtype=dtype or torch.float32)
    o = _conv_over_time(x, w, bias, state, batch)
    return o.view(T, C // block, block).transpose(0, 1).reshape(-1, block) if block else o


def conv_qkv_cache(y: torch.Tensor, w: torch.Tensor, state: torch.Tensor, batch: Batch, *, nq: int, dtype: torch.dtype,
                   k_cache: Optional[torch.Tensor] = None, v_cache: Optional[torch.Tensor] = None, q_temp: Optional[Tuple[float, float]] = None) -> torch.Tensor:
    """:func:`short_conv` on projection rows [q (nq) | k | v]: k and v go to the paged caches at ``batch.slots`` (without caches the
    rows are queries only), q times the position's temperature (coef, every) is returned, [T, nq] in ``dtype``, the caches' type."""
    if y.is_cuda:
        return _k().conv_qkv(y, w, state, batch, nq=nq, dtype=dtype, k_cache=k_cache, v_cache=v_cache, q_temp=q_temp)
    o = _conv_over_time(y, w, None, state, batch)
    if k_cache is not None:
        nk = k_cache.shape[1] * k_cache.shape[2]
        kv_scatter(k_cache, batch.slots, o[:, nq:nq + nk].unflatten(1, tuple(k_cache.shape[1:])))
        kv_scatter(v_cache, batch.slots, o[:, nq + nk:].unflatten(1, tuple(v_cache.shape[1:])))
    q = o[:, :nq]
    return q * ref.query_temperature(batch.positions, *q_temp).unsqueeze(1) if q_temp is not None else q


def embed_pairs(tok: QuantWeight, pair: QuantWeight, batch: Batch, prev: torch.Tensor, *, mul_prev: int, mul_cur: int,
                dtype: Optional[torch.dtype] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """Token embedding plus that of the pair (previous token, token): row (previous * mul_prev + token * mul_cur) mod buckets of
    ``pair`` [buckets + 1, D], the last row for a sequence's first token.  ``prev`` (int32 per slot, negative: none) is the token
    ahead of each sequence's new ones and is advanced.  Returns (f32 [T, D], the same as the next product reads it)."""
    if batch.tokens.is_cuda:
        return _k().pair_embed(tok, pair, batch.tokens, batch.cu_q, batch.seq_slots, prev, mul_prev=mul_prev, mul_cur=mul_cur,
                               out_dtype=dtype or torch.bfloat16)
    ids, buckets = batch.tokens.long(), pair.rows - 1
    before = torch.cat([ids[:1], ids[:-1]])
    for b, slot in enumerate(batch.seq_slots.tolist()):
        before[batch.h_cu_q[b]] = prev[slot]
        prev[slot] = ids[batch.h_cu_q[b + 1] - 1]
    rows = torch.where(before < 0, torch.full_like(ids, buckets), (before * mul_prev + ids * mul_cur) % buckets)
    h = tok.dequantize()[ids] + pair.dequantize()[rows]
    return h, h.clone()


def as_act(x, w: Optional[QuantWeight] = None) -> Act:
    """Wrap a plain activation tensor (an ``Act`` passes through)."""
    if isinstance(x, Act):
        return x
    if not x.is_cuda:
        return Act(x.float())
    a = Act(x if x.dtype == torch.bfloat16 else x.to(torch.bfloat16))
    return a


as_act_of = as_act


def _ensure_q8(a: Act) -> Act:
    if a.q is None:
        a.q, a.ds = _k().quantize_q8(a.b.contiguous())
    return a


FUSED_MAX_M = 4       # rows handled by the GEMV with the in-kernel norm / quantise prologue


def can_fuse(x: torch.Tensor, w: QuantWeight) -> bool:
    """Whether ``linear_fused`` should use the single-kernel path for this input (CUDA, at most
    FUSED_MAX_M rows, row length within the shared-memory staging limit).  Off unless
    TSB_FUSED_GEMV=1: on B200 the in-CTA prologue measured slower than the separate norm /
    quantise launches (Qwen3-4B decode 3.8 ms per step against 2.6 ms), because redoing the
    prologue per CTA costs more L2 traffic and occupancy than the two launches it removes."""
    return (os.environ.get("TSB_FUSED_GEMV", "0") == "1" and x.is_cuda and x.numel() // x.shape[-1] <= FUSED_MAX_M
            and w.K % 32 == 0 and w.K <= 10240 and w.experts == 1)


def linear_fused(x: torch.Tensor, w: QuantWeight, *, norm_w: Optional[torch.Tensor] = None, eps: float = 0.0,
                 do_norm: bool = False, bias: Optional[torch.Tensor] = None, residual: Optional[torch.Tensor] = None,
                 out_dtype=torch.float32, act: Optional[str] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(RMSNorm(x) * norm_w @ w^T + bias) + residual`` (the norm only with ``do_norm``) with
    ``x`` the f32 residual stream or a bf16 activation.  One kernel for small batches on CUDA
    (K-1 of the kernel list fused with K-5); the separate norm / linear ops otherwise."""
    if can_fuse(x, w):
        x = x.contiguous()
        kw = {"x_f32": x} if x.dtype == torch.float32 else {"x_bf16": x if x.dtype == torch.bfloat16 else x.to(torch.bfloat16)}
        return _k().fused_gemv(w, norm_w=norm_w, eps=eps, do_norm=do_norm, out_dtype=out_dtype, bias=bias,
                               residual=residual, act=act, out=out, **kw)
    T = x.numel() // x.shape[-1]
    a = norm(x, norm_w, eps, want_q8=T <= GEMV_MAX_M) if do_norm else as_act(x)
    y = linear(a, w, bias=bias, residual=residual, out_dtype=out_dtype, act=act)
    if out is not None:
        out.copy_(y)
        return out
    return y


_scratch = {}
_bf16_used = {}          # device index -> bytes of bf16 weight copies held
_bf16_auto = {}          # device index -> default budget


def _bf16_budget(device) -> int:
    """Bytes of spare HBM the prefill path may spend on bf16 copies of quantised weights.
    ``TSB_BF16_WEIGHT_CACHE_GB`` sets it (0 turns the copies off); the default is 35 % of the device's
    memory, at most 64 GB: a B200 holds a 4-bit 20 B-parameter model and its bf16 copy several times over."""
    env = os.environ.get("TSB_BF16_WEIGHT_CACHE_GB")
    if env is not None:
        return int(float(env) * (1 << 30))
    key = torch.device(device).index or 0
    if key not in _bf16_auto:
        _bf16_auto[key] = int(min(64 << 30, 0.35 * torch.cuda.get_device_properties(device).total_memory))
    return _bf16_auto[key]


def _release_bf16(dev_index: int, nbytes: int) -> None:
    _bf16_used[dev_index] = _bf16_used.get(dev_index, 0) - nbytes


def _dequant_scratch(w: QuantWeight, holder: Optional[QuantWeight] = None, slot: int = 0) -> torch.Tensor:
    """bf16 form of ``w`` for the tensor-core GEMM; bf16 weights are used in place.

    A quantised weight is decoded once and the copy is kept with the weight object (with ``holder`` and
    ``slot``: with the expert stack that ``w`` is a view of, so the copy outlives the temporary view) for
    as long as the budget of ``_bf16_budget`` lasts: prefill then reads weights the way a bf16 model would,
    while decode keeps streaming the GGUF blocks.  Past the budget the weight is decoded into a per-device
    scratch that every layer reuses (it stays L2-resident between the decode and the GEMM that follows)."""
    from ..gguf.constants import GGMLType
    if w.ggml_type == GGMLType.BF16:
        return w.planes[0].view(torch.bfloat16).view(w.rows, w.K)
    owner = holder if holder is not None else w
    cache = owner.__dict__.setdefault("_bf16_copies", {})
    hit = cache.get(slot)
    if hit is not None:
        return hit
    need = w.rows * w.K
    dev = w.device.index or 0
    if _bf16_used.get(dev, 0) + 2 * need <= _bf16_budget(w.device):
        import weakref
        out = torch.empty((w.rows, w.K), dtype=torch.bfloat16, device=w.device)
        _k().gather_rows(w, None, 1.0, out=out)
        cache[slot] = out
        _bf16_used[dev] = _bf16_used.get(dev, 0) + 2 * need
        weakref.finalize(out, _release_bf16, dev, 2 * need)
        return out
    key = (w.device.index, )
    buf = _scratch.get(key)
    if buf is None or buf.numel() < need:
        buf = torch.empty(max(need, 32 << 20), dtype=torch.bfloat16, device=w.device)
        _scratch[key] = buf
    out = buf[:need].view(w.rows, w.K)
    _k().gather_rows(w, None, 1.0, out=out)
    return out


def linear(a: Act, w: QuantWeight, *, bias: Optional[torch.Tensor] = None, residual: Optional[torch.Tensor] = None,
           out_dtype=torch.float32, act: Optional[str] = None) -> torch.Tensor:
    """y = a @ w^T (+ bias) (+ residual), optional GLU over the row halves of ``w``
    (rows [0, N/2) gate, [N/2, N) up).  ``residual`` is added in the output dtype."""
    T = a.T
    if w.device.type == "cuda" and a.b is not None and a.b.dtype == torch.float32:      # a model that runs in 32 bits
        y = _k().gemm_f32(w, a.b, bias=bias)
        if act is not None:
            half = w.N // 2
            y = _k().glu_f32(y, None, act) if act in ("relu2", "silu") else _k().glu_f32(y[:, :half], y[:, half:], act)
        return y if residual is None else y + residual
    if w.device.type != "cuda":
        y = a.b.float() @ w.dequantize().t()
        if bias is not None:
            y = y + bias.float()
        if act is not None:
            half = w.N // 2
            y = ref.glu(act, y[:, :half], y[:, half:]) if act not in ("relu2", "silu") else ref.glu(act, y, None)
        if residual is not None:
            y = y + residual.float()
        return y.to(out_dtype) if out_dtype != torch.float32 else y
    k = _k()
    if T <= DENSE_GEMV_MAX_M or (T <= GEMV_MAX_M and (a.b is None or w.experts != 1 or w.K % 8)):
        if w.uses_q8_activations:
            _ensure_q8(a)
            return k.gemv(w, xq=a.q, xds=a.ds, M=T, out_dtype=out_dtype, bias=bias, residual=residual, act=act)
        return k.gemv(w, xb=a.b.contiguous(), M=T, out_dtype=out_dtype, bias=bias, residual=residual, act=act)
    wb = _dequant_scratch(w)
    if act is None:
        return k.gemm_bf16(wb, a.b, out_dtype=out_dtype, bias=bias, residual=residual)
    y = k.gemm_bf16(wb, a.b, out_dtype=torch.bfloat16, bias=bias)
    half = w.N // 2
    if act in ("relu2", "silu"):
        out, _, _ = k.glu(y, None, act, w.N, w.N, 0, T)
    else:
        out, _, _ = k.glu(y, y[:, half:], act, half, w.N, w.N, T)
    if residual is not None:
        out = out.to(out_dtype) + residual
    return out if out.dtype == out_dtype else out.to(out_dtype)


def linear_multi(a: Act, ws, *, out_dtype=torch.float32):
    """``[a @ w^T for w in ws]`` for matrices that share the input.  Decode-sized CUDA batches run them
    as one launch (the separate Q / K / V projections of files whose tensors differ in quantisation
    type); anything else is the plain sequence of ``linear`` calls."""
    ws = list(ws)
    T = a.T
    if (ws[0].device.type == "cuda" and T <= DENSE_GEMV_MAX_M and 2 <= len(ws) <= 3 and all(w.experts == 1 and w.K == ws[0].K for w in ws)
            and len({w.uses_q8_activations for w in ws}) == 1):
        if ws[0].uses_q8_activations:
            _ensure_q8(a)
            y = _k().gemv_multi(ws, xq=a.q, xds=a.ds, M=T, out_dtype=out_dtype)
        else:
            y = _k().gemv_multi(ws, xb=a.b.contiguous(), M=T, out_dtype=out_dtype)
        outs, o = [], 0
        for w in ws:
            outs.append(y[:, o:o + w.N])
            o += w.N
        return outs
    return [linear(a, w, out_dtype=out_dtype) for w in ws]


def glu(act: str, gate: torch.Tensor, up: Optional[torch.Tensor]) -> torch.Tensor:
    """Standalone gated activation on two [T, F] tensors (row-strided views allowed)."""
    if not gate.is_cuda:
        return ref.glu(act, gate, up)
    T, F = gate.shape
    if up is not None and up.dtype != gate.dtype:      # the kernel reads both operands with one element type
        up = up.to(gate.dtype)
    out, _, _ = _k().glu(gate, up, act, F, gate.stride(0), up.stride(0) if up is not None else 0, T)
    return out


def qkv_rope_cache(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, Hq: int, Hkv: int, Dh: int,
                   batch: Batch, k_cache: torch.Tensor, v_cache: torch.Tensor, rope: Optional[RopeSpec],
                   qn: Optional[torch.Tensor] = None, kn: Optional[torch.Tensor] = None, v_norm: bool = False,
                   eps: float = 1e-6, q_scale: float = 1.0, write_kv: bool = True, Dv: Optional[int] = None,
                   norm_n: Optional[int] = None, q_temp: Optional[Tuple[float, float]] = None) -> torch.Tensor:
    """Per-head norm on Q / K (and optionally V), RoPE on Q / K, write K / V into the paged
    cache at ``batch.slots``; returns the rotated queries ``[T, Hq, Dh]``.
    ``q``, ``k``, ``v`` are ``[T, H*, Dh]`` views (any token / head stride, last dim dense).  ``Dv``: value head
    size where it differs; ``norm_n``: the norm's divisor where the head is padded with zeros; ``q_temp``
    (coef, every): position-dependent query factor (reference.py: query_temperature).  A float32 cache gets
    float32 rows and gives float32 queries."""
    T = batch.T
    Dv = Dv or Dh
    if q.is_cuda:
        kk = _k()
        rp = kk.RopeParams()
        if rope is not None:
            rp.theta_base, rp.freq_scale, rp.ext_factor = rope.theta_base, rope.freq_scale, rope.ext_factor
            rp.attn_factor, rp.corr_lo, rp.corr_hi = rope.attn_factor, rope.corr_lo, rope.corr_hi
            rp.rot_dim, rp.mode = rope.rot_dim, rope.mode
        else:
            rp.rot_dim, rp.mode, rp.theta_base, rp.freq_scale, rp.attn_factor = 0, 0, 10000.0, 1.0, 1.0
        table = None
        if rope is not None and rope.rot_dim > 0:
            key = ("rope", id(rope))
            table = batch.cache.get(key)
            if table is None:
                table = (kk.rotary_table(batch.positions, rope.freq, rope.attn_factor) if rope.freq is not None else
                         kk.rope_table(batch.positions, rp, rope.freq_factors))
                batch.cache[key] = table
        f32 = k_cache.dtype == torch.float32
        q_out = torch.empty((T, Hq, Dh), dtype=torch.float32 if f32 else torch.bfloat16, device=q.device)
        assert q.stride(-1) == 1 and k.stride(-1) == 1 and v.stride(-1) == 1 and q.dtype == k.dtype == v.dtype
        slots, kc, vc = batch.slots, k_cache, v_cache
        fp8 = write_kv and is_fp8(k_cache)
        if fp8 and Dv != Dh:
            raise ValueError("8-bit pages hold keys and values of one size")
        if fp8:
            # 8-bit pages: the kernel leaves the finished K / V rows in dense bf16 staging rows, which one more
            # kernel converts and scatters to their slots
            slots = batch.cache.get("arange_T")
            if slots is None:
                slots = batch.cache["arange_T"] = torch.arange(T, dtype=torch.int64, device=q.device)
            kc = torch.empty((T, Hkv, Dh), dtype=torch.bfloat16, device=q.device)
            vc = torch.empty_like(kc)
        kk.qkv_rope(q=q, k=k, v=v, q_strides=(q.stride(0), q.stride(1)), k_strides=(k.stride(0), k.stride(1)),
                    v_strides=(v.stride(0), v.stride(1)), Hq=Hq, Hkv=Hkv if write_kv else 0, Dh=Dh,
                    pos=batch.positions, slot=slots,
                    q_out=q_out, k_cache=kc, v_cache=vc, qn=qn, kn=kn, v_norm=v_norm, eps=eps, rope=rp,
                    freq_factors=rope.freq_factors if rope is not None else None, q_scale=q_scale,
                    cs_table=table, Dv=Dv, norm_n=norm_n or Dh, q_temp=q_temp, out_f32=f32)
        if fp8:
            kk.kv_store_fp8(kc, vc, k_cache, v_cache, batch.slots)
        return q_out
    qf, kf, vf = q.float(), k.float(), v.float()
    nn = norm_n or Dh
    if qn is not None:
        qf = torch.nn.functional.pad(ref.rmsnorm(qf[..., :nn], qn[:nn], eps), (0, Dh - nn))
    if kn is not None:
        kf = torch.nn.functional.pad(ref.rmsnorm(kf[..., :nn], kn[:nn], eps), (0, Dh - nn))
    if v_norm:
        vf = ref.rmsnorm(vf, None, eps)
    if rope is not None and rope.rot_dim > 0:
        if rope.freq is not None:
            ang = batch.positions.double().unsqueeze(1) * rope.freq
            cos, sin = (ang.cos() * rope.attn_factor).float(), (ang.sin() * rope.attn_factor).float()
        else:
            cos, sin = ref.rope_cos_sin(batch.positions, rope.rot_dim, rope.theta_base, rope.freq_scale,
                                        rope.ext_factor, rope.attn_factor, rope.corr_lo, rope.corr_hi,
                                        rope.freq_factors)
        qf = ref.apply_rope(qf, cos, sin, rope.rot_dim, rope.mode)
        kf = ref.apply_rope(kf, cos, sin, rope.rot_dim, rope.mode)
    if write_kv:
        kv_scatter(k_cache, batch.slots, kf)
        kv_scatter(v_cache, batch.slots, vf)
    if q_temp is not None:
        qf = qf * ref.query_temperature(batch.positions, *q_temp).view(-1, 1, 1)
    return qf * q_scale


FP8 = torch.float8_e4m3fn


def is_fp8(cache: torch.Tensor) -> bool:
    return cache.dtype == FP8


def kv_scatter(cache: torch.Tensor, slots: torch.Tensor, rows: torch.Tensor) -> None:
    """``cache[slots] = rows`` in the cache's element type (8-bit caches are indexed through their bytes)."""
    if is_fp8(cache):
        cache.view(torch.uint8)[slots] = rows.to(FP8).view(torch.uint8)
    else:
        cache[slots] = rows.to(cache.dtype)


def kv_gather(cache: torch.Tensor, idx: torch.Tensor) -> torch.Tensor:
    """``cache[idx]``; rows of an 8-bit cache come back as float32."""
    if is_fp8(cache):
        return cache.view(torch.uint8)[idx].view(FP8).float()
    return cache[idx]


def fp8_prefill_view(k_cache: torch.Tensor, v_cache: torch.Tensor, batch: Batch):
    """The cache rows of the batch's sequences as dense bf16 tensors, laid out as one page per sequence, with the
    block table that goes with them: (K, V, table, page size).  Converting a prompt's keys once per layer costs their
    bytes three times over; the flash kernel then reads them once per query tile as it does bf16 pages."""
    ps, B = batch.page_size, batch.B
    L = (batch.max_kv_len + 63) // 64 * 64
    key = ("fp8_idx", id(batch.block_table))
    cached = batch.cache.get(key)
    if cached is None:
        j = torch.arange(L, device=k_cache.device)
        width = batch.block_table.shape[1]
        pages = batch.block_table.long()[:, (j // ps).clamp_max(width - 1)]           # [B, L]; rows past a sequence's end are never read
        idx = (pages * ps + (j % ps)[None, :]).reshape(-1).contiguous()
        table = torch.arange(B, dtype=torch.int32, device=k_cache.device).view(B, 1)
        cached = batch.cache[key] = (idx, table)
    idx, table = cached
    kd, vd = _k().kv_load_fp8(k_cache, v_cache, idx)
    return kd, vd, table, L


def decode_split_len(batch: Batch, splits: int, window: int) -> int:
    """Positions per split fixed on the host from the reserved maximum length (0 with a sliding window, whose
    start depends on the actual length): the kernel then knows its range before it has read the length."""
    if window:
        return 0
    return ((batch.max_kv_len + splits - 1) // splits + 31) & ~31


def decode_splits(batch: Batch, Hkv: int, window: int) -> int:
    """Split-KV factor for decode attention: enough CTAs to cover the GPU's 148 SMs."""
    span = batch.max_kv_len if not window else min(batch.max_kv_len, window)
    # one sequence: about two CTAs per SM; batches: up to eight (a CTA is 128 threads and latency-bound, and with 16
    # sequences two splits per (sequence, KV head) left the kernel at a fifth of the memory rate)
    want = max(1, (148 * (2 if batch.B == 1 else 8)) // max(1, batch.B * Hkv))
    per = int(os.environ.get("TSB_ATTN_SPLIT_LEN", "128"))
    n = int(max(1, min(want, (span + per - 1) // per, 64)))
    # TSB_ATTN_CLUSTER=1: 8 or 16 splits are merged inside the attention kernel by a thread-block cluster (no combine
    # launch), so take those counts when the natural one is close (measured slower than the combine launch: off by default)
    if os.environ.get("TSB_ATTN_CLUSTER", "0") not in ("", "0"):
        if want >= 16 and 13 <= n <= 20:
            return 16
        if want >= 8 and 7 <= n <= 10:
            return 8
    return n


def attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, batch: Batch, *, scale: float,
              Hq: int, Hkv: int, Dh: int, window: int = 0, sinks: Optional[torch.Tensor] = None,
              softcap: float = 0.0, as_act: bool = False, Dv: Optional[int] = None, gate: Optional[torch.Tensor] = None, keep_first: int = 0,
              slopes: Optional[torch.Tensor] = None, own_values: bool = False, log_bias: Optional[Tuple[torch.Tensor, torch.Tensor]] = None,
              sigmoid_bias: Optional[torch.Tensor] = None):
    """Causal attention of the packed queries against the paged cache -> [T, Hq * Dh].  ``as_act`` returns an
    ``Act``; on the CUDA decode path it already carries the int8 form written by the combine kernel, so
    the quantised projection that follows needs no quantise launch.  ``Dv``: value head size where it differs from
    ``Dh`` (the result is then [T, Hq * Dv]); ``gate`` [T, Hq] (a view, last dim dense): head h's output is
    multiplied by sigmoid(gate[:, h]), with a gate [T, Hq * Dv] every column by its own; float32 caches run in 32 bits.
    ``keep_first``: with a window, so many positions at the start stay visible; ``slopes`` [Hq]: slopes[h] times the distance
    is taken off the score; ``own_values``: a row of ``k_cache`` (see :func:`joint_norm_cache`) is key and value at once;
    ``log_bias`` (r1, r2) [Hq] each: r1[h] ln(1 + r2[h] distance) is taken off the score (after the soft cap);
    ``sigmoid_bias`` [Hq]: no softmax, a visible key has the weight sigmoid(score + sigmoid_bias[h])."""
    T = q.shape[0]
    Dv = Dv or Dh
    if q.is_cuda and (Dv != Dh or gate is not None or k_cache.dtype == torch.float32 or keep_first or slopes is not None or own_values
                      or log_bias is not None or sigmoid_bias is not None):
        return _gated_attention(q, k_cache, v_cache, batch, scale=scale, Hq=Hq, Hkv=Hkv, Dh=Dh, Dv=Dv, window=window,
                                sinks=sinks, softcap=softcap, gate=gate, keep_first=keep_first, slopes=slopes,
                                kv_scale=Hkv * Dh if own_values else 0, log_bias=log_bias, sigmoid_bias=sigmoid_bias)
    if as_act:
        if q.is_cuda and batch.is_decode and Dh % 32 == 0:
            sp = decode_splits(batch, Hkv, window)
            out, oq, ods = _k().attn_decode(q, k_cache, v_cache, batch.block_table, batch.kv_lens, scale=scale, Hq=Hq, Hkv=Hkv,
                                            Dh=Dh, page_size=batch.page_size, splits=sp, split_len=decode_split_len(batch, sp, window),
                                            sinks=sinks, softcap=softcap, window=window, want_q8=True)
            return Act(out.view(T, Hq * Dh), oq, ods)
        return as_act_of(attention(q, k_cache, v_cache, batch, scale=scale, Hq=Hq, Hkv=Hkv, Dh=Dh, window=window, sinks=sinks,
                                   softcap=softcap))
    if q.is_cuda:
        kk = _k()
        if batch.is_decode:
            sp = decode_splits(batch, Hkv, window)
            out = kk.attn_decode(q, k_cache, v_cache, batch.block_table, batch.kv_lens, scale=scale, Hq=Hq, Hkv=Hkv,
                                 Dh=Dh, page_size=batch.page_size, splits=sp, split_len=decode_split_len(batch, sp, window),
                                 sinks=sinks, softcap=softcap, window=window)
        else:
            table, ps = batch.block_table, batch.page_size
            if is_fp8(k_cache):
                k_cache, v_cache, table, ps = fp8_prefill_view(k_cache, v_cache, batch)
            out = kk.attn_prefill(q, k_cache, v_cache, table, batch.kv_lens, batch.cu_q, batch.max_q_len,
                                  scale=scale, Hq=Hq, Hkv=Hkv, Dh=Dh, page_size=ps, sinks=sinks,
                                  softcap=softcap, window=window)
        return out.view(T, Hq * Dh)
    outs = []
    ps = batch.page_size
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        L = batch.h_kv_lens[b]
        pages = batch.block_table[b, :(L + ps - 1) // ps].long()
        idx = (pages.unsqueeze(1) * ps + torch.arange(ps)).reshape(-1)[:L]
        if own_values:
            rows = k_cache[idx].view(L, -1)
            if window:
                rows = rows.clone()
                rows[keep_first:max(keep_first, L - (q1 - q0) - window + 1)] = 0       # out of every query's sight; may be stale in a ring
            vb = rows[:, :Hkv * Dh].view(L, Hkv, Dh)
            kb = vb * rows[:, Hkv * Dh].view(L, 1, 1)
        else:
            kb, vb = kv_gather(k_cache, idx), kv_gather(v_cache, idx)
        outs.append(ref.attention(q[q0:q1], kb, vb, batch.positions[q0:q1], scale=scale, window=window, sinks=sinks,
                                  softcap=softcap, keep_first=keep_first, slopes=slopes, log_bias=log_bias, sigmoid_bias=sigmoid_bias))
    out = torch.cat(outs, 0)
    if gate is not None:
        out = out * torch.sigmoid(gate.float()).view(T, Hq, -1)
    return out.reshape(T, Hq * Dv)


def _gated_attention(q, k_cache, v_cache, batch: Batch, *, scale, Hq, Hkv, Dh, Dv, window, sinks, softcap, gate, keep_first=0, slopes=None,
                     kv_scale=0, log_bias=None, sigmoid_bias=None) -> torch.Tensor:
    """The CUDA side of :func:`attention` for the forms beyond one head size and bf16: keys and values of different
    sizes, sigmoid gates, kept first positions, distance biases, sigmoid weights, rows that are key and value at once, 32-bit caches."""
    kk = _k()
    T = q.shape[0]
    if is_fp8(k_cache):
        raise ValueError("8-bit pages have no gated attention")
    kw = dict(scale=scale, Hq=Hq, Hkv=Hkv, Dh=Dh, Dv=Dv, page_size=batch.page_size, sinks=sinks, softcap=softcap, window=window,
              gate=gate, keep_first=keep_first, slopes=slopes, kv_scale=kv_scale, log_bias=log_bias, sigmoid_bias=sigmoid_bias)
    if k_cache.dtype == torch.float32:
        return kk.attn_f32(q, k_cache, v_cache, batch.block_table, batch.kv_lens, batch.cu_q, **kw).view(T, Hq * Dv)
    if batch.is_decode:
        sp = decode_splits(batch, Hkv, window + keep_first if window else 0)
        out = kk.attn_decode(q, k_cache, v_cache, batch.block_table, batch.kv_lens, splits=sp,
                             split_len=decode_split_len(batch, sp, window), **kw)
    else:
        out = kk.attn_prefill(q, k_cache, v_cache, batch.block_table, batch.kv_lens, batch.cu_q, batch.max_q_len, **kw)
    return out.view(T, Hq * Dv)


def argmax(logits: torch.Tensor) -> torch.Tensor:
    if logits.is_cuda:
        return _k().argmax(logits.float().contiguous())
    return logits.argmax(-1).to(torch.int32)


# --------------------------------------------------------------------------------------------
# Latent attention: one cached row [latent | rotated key part] per token serves every head
# --------------------------------------------------------------------------------------------
@dataclass
class LatentSpec:
    """Sizes of a latent-attention mixer.  A cached row is [latent (rank) | rotated part (rot) | zeros] of ``row`` elements, a
    query head [unrotated (dim) | rotated (rot) | zeros] of ``Dk``, a value head ``Dv``; ``qp``, ``rank_p``: padded ranks."""
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    q_rank: int
    scale: float
    window: int                           # 0: the whole context
    base: float
    freq: torch.Tensor                    # float64 [rot / 2] on the compute device

    def __post_init__(self):
        self.Dk, self.Dv = (self.dim + self.rot + 15) // 16 * 16, (self.vdim + 15) // 16 * 16
        self.row = (self.rank + self.rot + 31) // 32 * 32
        self.qp, self.rank_p = (self.q_rank + 7) // 8 * 8, (self.rank + 7) // 8 * 8


def rotary_freqs(dims: int, base: float, device) -> torch.Tensor:
    """base^(-2 i / dims) of every pair, float64."""
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)


def yarn_freqs(dims: int, base: float, scaling: Optional[dict], device) -> Tuple[torch.Tensor, float]:
    """Frequencies of :func:`rotary_freqs` with YaRN scaling {factor, original, fast, slow} (None: as they are), and the factor
    on cos and sin: pairs that turn more than ``fast`` times over the original context keep their frequency, those that turn
    less than ``slow`` times have it divided by ``factor``, with a linear ramp over the pair's number in between."""
    f = rotary_freqs(dims, base, device)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair(turns: float) -> float:                  # twice the number of the pair that turns so often, as a real number
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(float(base)))
    lo, hi = max(math.floor(pair(float(scaling["fast"]))), 0), min(math.ceil(pair(float(scaling["slow"]))), dims - 1)
    i = torch.arange(dims // 2, dtype=torch.float64, device=device)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def alibi_slopes(heads: int, device) -> torch.Tensor:
    """Geometric slopes 2^(-8 (h + 1) / heads) of a distance bias."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float32, device=device)


def joint_norm_cache(y: torch.Tensor, w: torch.Tensor, cache: torch.Tensor, batch: Batch, *, nq: int, nk: int, q_n: int, k_n: int, eps: float) -> torch.Tensor:
    """Query and key norms over whole projections for attention whose values are the keys ahead of their norm.  Rows of ``y``:
    [q (nq) | k (nk)], padded heads.  A cached row holds k as it is and then 1 / rms(k); the keys' norm weight is part of ``w``
    (the query weight times that of the query head's key head), so q / rms(q) * w against k times the row's factor is the
    score.  ``q_n``, ``k_n``: sizes without padding.  Returns the queries [T, nq]."""
    if y.is_cuda:
        return _k().joint_norm(y, w, cache, batch.slots, nq=nq, nk=nk, q_n=q_n, k_n=k_n, eps=eps)
    y = y.float()
    q, k = y[:, :nq], y[:, nq:nq + nk]
    row = torch.zeros((y.shape[0], nk + 8))
    row[:, :nk] = k
    row[:, nk] = torch.rsqrt((k * k).sum(-1) / k_n + eps)
    kv_scatter(cache, batch.slots, row.unsqueeze(1))
    return q * torch.rsqrt((q * q).sum(-1, keepdim=True) / q_n + eps) * w


def rotary_table(batch: Batch, s: LatentSpec) -> torch.Tensor:
    """(cos, sin) [T, rot / 2, 2] of the batch's positions, made once per step for all layers with these frequencies."""
    key = ("rotary", s.base, s.rot)
    t = batch.cache.get(key)
    if t is None:
        if batch.positions.is_cuda:
            t = _k().rotary_table(batch.positions, s.freq)
        else:
            ang = batch.positions.double().unsqueeze(1) * s.freq
            t = torch.stack([ang.cos(), ang.sin()], -1).float()
        batch.cache[key] = t
    return t


def _rotate_half(x: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """x [T, ..., R] with the columns i and i + R / 2 as pairs."""
    half = x.shape[-1] // 2
    t = table.view(table.shape[0], *([1] * (x.dim() - 2)), half, 2)
    c, s = t[..., 0], t[..., 1]
    x0, x1 = x[..., :half], x[..., half:]
    return torch.cat([x0 * c - x1 * s, x1 * c + x0 * s], -1)


def latent_cache(y: torch.Tensor, s: LatentSpec, qn: torch.Tensor, kn: torch.Tensor, cache: torch.Tensor, batch: Batch, eps: float) -> Act:
    """Projection rows [query latent (qp) | latent (rank) | rotated part (rot)] -> the normed query latent; the normed latent
    and the rotated key part are written to the paged cache ``[slots, 1, row]`` at ``batch.slots``."""
    table = rotary_table(batch, s)
    if y.is_cuda:
        return Act(_k().latent_prep(y, s, qn, kn, table, cache, batch.slots, eps))
    T = y.shape[0]
    cq = torch.zeros((T, s.qp))
    cq[:, :s.q_rank] = ref.rmsnorm(y[:, :s.q_rank], qn, eps)
    row = torch.zeros((T, s.row))
    row[:, :s.rank] = ref.rmsnorm(y[:, s.qp:s.qp + s.rank], kn, eps)
    row[:, s.rank:s.rank + s.rot] = _rotate_half(y[:, s.qp + s.rank:s.qp + s.rank + s.rot].float(), table)
    kv_scatter(cache, batch.slots, row.unsqueeze(1))
    return Act(cq)


def visible_rows(batch: Batch, window: int):
    """The cache rows that some query of the batch can see, packed sequence after sequence: (cache slot of each packed row
    int32, block table of the packed rows in pages of 64).  A sequence's rows start at a multiple of 64 positions, and its
    last page is filled up with copies of its last row; memoised per step."""
    key = ("visible", id(batch.block_table), window)
    hit = batch.cache.get(key)
    if hit is not None:
        return hit
    seq, pos, table, n = [], [], [], 0
    width = max((L + 63) // 64 for L in batch.h_kv_lens)
    for b, L in enumerate(batch.h_kv_lens):
        first = L - (batch.h_cu_q[b + 1] - batch.h_cu_q[b])                 # position of the first query
        lo = max(0, first - window + 1) // 64 if window else 0
        hi = (L + 63) // 64
        table.append([0] * lo + list(range(n, n + hi - lo)) + [0] * (width - hi))
        p = torch.arange(lo * 64, hi * 64).clamp_(max=L - 1)
        pos.append(p)
        seq.append(torch.full_like(p, b))
        n += hi - lo
    dev, ps = batch.block_table.device, batch.page_size
    p, b = torch.cat(pos).to(dev), torch.cat(seq).to(dev)
    slots = (batch.block_table[b, p // ps].long() * ps + p % ps).to(torch.int32)
    hit = batch.cache[key] = (slots, torch.tensor(table, dtype=torch.int32).to(dev))
    return hit


def latent_splits(batch: Batch, s: LatentSpec) -> int:
    """Split-KV factor of the latent decode kernel: as many CTAs as the SMs hold at once (its tiles of 64 keys take up to
    most of an SM's shared memory), at least one tile each."""
    span = min(batch.max_kv_len, s.window) if s.window else batch.max_kv_len
    heads, smem = _k().latent_decode_shape(batch.B, s.heads, s.row)
    per_sm = max(1, min(4, (226 << 10) // smem))
    return max(1, min(148 * per_sm // max(1, batch.B * -(-s.heads // heads)), (span + 63) // 64, 64))


def latent_attention(q: torch.Tensor, cache: torch.Tensor, batch: Batch, s: LatentSpec, *, wuk: torch.Tensor, wuv: torch.Tensor,
                     expand: Optional[QuantWeight], sinks: Optional[torch.Tensor]) -> torch.Tensor:
    """Causal attention of the queries ``[T, heads * Dk]`` (not rotated yet) over the cached rows -> ``[T, heads * Dv]``.
    ``wuk`` [heads * dim, rank_p], ``wuv`` [heads * Dv, rank_p]: key and value maps; ``expand``: both as one matrix over
    whole rows, [heads * Dk + heads * Dv, row], the rotated part passed on to every head.

    CUDA, bf16: decode steps work on the rows themselves; prompts expand the rows in sight and take the ordinary prefill
    kernel.  CUDA, float32: on the rows themselves, prompts too."""
    T, H = q.shape[0], s.heads
    table = rotary_table(batch, s)
    if not q.is_cuda:
        qh = q.float().view(T, H, s.Dk)
        qh = torch.cat([qh[..., :s.dim], _rotate_half(qh[..., s.dim:s.dim + s.rot], table)], -1)
        uk, uv = wuk.float().view(H, s.dim, -1)[..., :s.rank], wuv.float().view(H, s.Dv, -1)[..., :s.rank]
        outs, ps = [], batch.page_size
        for b, L in enumerate(batch.h_kv_lens):
            q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
            p = torch.arange(L)
            rows = cache[batch.block_table[b].long()[p // ps] * ps + p % ps, 0].float()
            if s.window:
                rows[:max(0, L - (q1 - q0) - s.window + 1)] = 0                # out of every query's sight; may be stale
            k = torch.cat([torch.einsum("tr,hdr->thd", rows[:, :s.rank], uk),
                           rows[:, None, s.rank:s.rank + s.rot].expand(L, H, s.rot)], -1)
            v = torch.einsum("tr,hdr->thd", rows[:, :s.rank], uv)
            outs.append(ref.attention(qh[q0:q1], k, v, batch.positions[q0:q1], scale=s.scale, window=s.window, sinks=sinks))
        return torch.cat(outs).reshape(T, H * s.Dv)
    kk = _k()
    if cache.dtype == torch.float32:
        qa = kk.latent_absorb(q, s, wuk, table, cache)
        o = kk.attn_f32(qa, cache, cache[:, :, :s.rank], batch.block_table, batch.kv_lens, batch.cu_q, scale=s.scale, Hq=H, Hkv=1, Dh=s.row,
                        Dv=s.rank, page_size=batch.page_size, sinks=sinks, window=s.window)
        return kk.latent_out(o, None, s, wuv, None, table, cache)
    if batch.is_decode:
        qa = kk.latent_absorb(q, s, wuk, table, cache)
        part_o, part_ml = kk.latent_decode(qa, s, table, cache, batch.block_table, batch.kv_lens, batch.page_size,
                                           latent_splits(batch, s))
        return kk.latent_out(part_o, part_ml, s, wuv, sinks, table, cache)
    kk.latent_rotate(q, s, table, cache)
    slots, pages = visible_rows(batch, s.window)
    rows = kk.gather_bf16_rows(cache.view(-1, s.row), slots, 1)
    kv = kk.gemm_bf16(_dequant_scratch(expand), rows)
    k, v = kv[:, :H * s.Dk].unflatten(1, (H, s.Dk)), kv[:, H * s.Dk:].unflatten(1, (H, s.Dv))
    out = kk.attn_prefill(q.view(T, H, s.Dk), k, v, pages, batch.kv_lens, batch.cu_q, batch.max_q_len, scale=s.scale, Hq=H, Hkv=H, Dh=s.Dk,
                          Dv=s.Dv, page_size=64, sinks=sinks, window=s.window)
    return out.view(T, H * s.Dv)


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    if cap and cap > 0 and x.is_cuda and x.dtype == torch.float32 and x.is_contiguous():
        return _k().softcap(x, cap)
    return torch.tanh(x / cap) * cap if cap and cap > 0 else x


# --------------------------------------------------------------------------------------------
# Mixture of experts
# --------------------------------------------------------------------------------------------
MOE_TILE_MAX_PAIRS = int(os.environ.get("TSB_MOE_TILE_MAX_PAIRS", "1024"))


def route_topk_softmax(logits: torch.Tensor, k: int):
    """Top-k on the router logits, then softmax over the selected k (GPT-OSS, Qwen3.5 decode;
    GptOssModel.cs:814-865).  Equivalent to softmax over all -> top-k -> renormalise."""
    if logits.is_cuda and logits.dtype == torch.float32 and logits.shape[-1] <= 1024 and k <= 32:
        return _k().moe_route(logits.contiguous(), k, mode=0)
    vals, ids = torch.topk(logits.float(), k, dim=-1)
    return ids.to(torch.int32), torch.softmax(vals, -1)


def route_sigmoid(logits: torch.Tensor, k: int, bias: Optional[torch.Tensor], normalize: bool, scale: float):
    """Nemotron-H router: selection on sigmoid(logits) + bias, weights are the unbiased
    sigmoid values, optionally normalised (floor 6.1e-5) and scaled (NemotronModel.cs:822-856)."""
    if logits.is_cuda and logits.dtype == torch.float32 and logits.shape[-1] <= 1024 and k <= 16:
        return _k().moe_route(logits.contiguous(), k, mode=1, sel_bias=bias.float().contiguous() if bias is not None else None,
                              normalize=normalize, scale=scale)
    p = torch.sigmoid(logits.float())
    sel = p + bias.float() if bias is not None else p
    _, ids = torch.topk(sel, k, dim=-1)
    w = p.gather(-1, ids)
    if normalize:
        w = w / w.sum(-1, keepdim=True).clamp_min(6.103515625e-5)
    return ids.to(torch.int32), w * scale


def route_softmax_renorm(logits: torch.Tensor, E: int, k: int, scale: float, n_always: int = 0):
    """Softmax over the first ``E`` logits, the ``k`` largest, their scores divided by their sum (+ 1e-20) times
    ``scale``.  ``n_always`` > 0 appends the experts ``E .. E + n_always - 1`` (slices of a shared expert) to every
    token, each with the weight sigmoid(logits[:, E]).  -> (ids int32, weights f32), both [T, k + n_always]."""
    if logits.is_cuda:
        return _k().moe_route(logits, k, mode=2, scale=scale, n_experts=E, n_always=n_always)
    s = torch.softmax(logits[:, :E].float(), -1)
    val, ids = torch.topk(s, k, dim=-1)
    w = val / (val.sum(-1, keepdim=True) + 1e-20) * scale
    if n_always:
        T = logits.shape[0]
        ids = torch.cat([ids, torch.arange(E, E + n_always).expand(T, n_always)], 1)
        w = torch.cat([w, torch.sigmoid(logits[:, E:E + 1].float()).expand(T, n_always)], 1)
    return ids.to(torch.int32), w


def route_softmax_groups(logits: torch.Tensor, correction: Optional[torch.Tensor], k: int, *, groups: int, keep: int, n_real: int,
                         n_always: int = 0):
    """Softmax over all logits; the ``k`` largest of softmax + ``correction`` among the ``keep`` best of ``groups`` equal groups of
    neighbours (a group is as good as its best entry); the weights are the softmax values, not renormalised.  Entries from
    ``n_real`` on are identity experts: their id is -1.  The ids 0 .. n_always - 1 (slices of a shared expert) come first on every
    token with weight 1, the routed experts are numbered from ``n_always`` on.  -> (ids int32, weights f32), [T, n_always + k]."""
    if logits.is_cuda:
        return _k().moe_route_grouped(logits, k, correction=correction, groups=groups, keep=keep, n_real=n_real, n_always=n_always)
    s = torch.softmax(logits.float(), -1)
    choice = s + correction if correction is not None else s
    T, E = s.shape
    by_group = choice.view(T, groups, E // groups)
    best = torch.topk(by_group.max(-1).values, keep, dim=-1).indices
    shut = torch.ones((T, groups, 1), dtype=torch.bool).scatter_(1, best.unsqueeze(-1), False)
    ids = torch.topk(by_group.masked_fill(shut, float("-inf")).view(T, E), k, dim=-1).indices
    w = s.gather(-1, ids)
    ids = torch.where(ids < n_real, ids + n_always, torch.full_like(ids, -1))
    return (torch.cat([torch.arange(n_always).expand(T, n_always), ids], 1).to(torch.int32),
            torch.cat([torch.ones((T, n_always)), w], 1))


@dataclass
class MoeParts:
    """The experts' output rows before they are summed per token: token t's result is the sum over j < k of
    ``w[t * k + j] * y[pos[t * k + j]]`` (``w`` None: rows are weighted already; ``pos`` None: row t * k + j).  Where
    ``ids[t * k + j]`` is negative (an identity expert) the layer's input stands in place of the row."""
    y: torch.Tensor
    k: int
    pos: Optional[torch.Tensor] = None
    w: Optional[torch.Tensor] = None
    ids: Optional[torch.Tensor] = None

    def sum(self, x: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``x`` [T, D]: the layer's input (with ``ids``)."""
        y = self.y.float()
        if self.ids is not None:
            ids = self.ids.view(-1, self.k)
            own = (self.w.view(-1, self.k) * (ids < 0)).sum(1, keepdim=True)
            return own * x + y
        if self.pos is not None:
            y = y[self.pos.long()]
        if self.w is not None:
            y = y * self.w.reshape(-1, 1)
        return y.view(-1, self.k, y.shape[-1]).sum(1)


def moe_expert_parts(a: Act, ids: torch.Tensor, weights: torch.Tensor, gate_up: QuantWeight, down: QuantWeight, *, act: str,
                     clamp: Optional[Tuple[float, float, int]] = None, identity: bool = False) -> MoeParts:
    """:func:`moe_experts` without its last step, for a consumer that sums the rows itself (``residual_layernorm``,
    ``post_norm_seam``): every expert is local, there are no biases, and ``act`` is gated.  ``clamp`` (limit, limit of the first
    experts, how many): the clamp of "swiglu_oai"; ids below that number are on every token and come first in ``ids``'
    rows.  ``identity``: negative ids stand for the layer's input itself."""
    T, k = ids.shape
    if ids.device.type != "cuda":
        if clamp is None:
            return MoeParts(moe_experts(a, ids, weights, gate_up, down, act=act), 1)
        y = torch.zeros((T, down.N))
        half = gate_up.N // 2
        for e in range(gate_up.experts):
            tok, slot = (ids == e).nonzero(as_tuple=True)
            if tok.numel():
                u = linear(Act(a.b[tok]), gate_up.expert(e))
                u = ref.glu(act, u[:, :half], u[:, half:], clamp[1] if e < clamp[2] else clamp[0])
                y.index_add_(0, tok, linear(Act(u), down.expert(e)) * weights[tok, slot].unsqueeze(1))
        return MoeParts(y, k, None, weights, ids) if identity else MoeParts(y, 1)
    kk = _k()
    flat_ids = ids if identity else None
    row_clamp = (clamp[0], clamp[1], T * clamp[2]) if clamp else None          # sorted by expert, the first experts' rows come first
    P, E, F_out, D = T * k, gate_up.experts, gate_up.N // 2, down.N
    wts = weights.reshape(-1)
    if a.b.dtype == torch.float32:
        bn = 64
        order, tiles, pos = kk.moe_sort(ids, E, bn)
        y1 = kk.gemm_f32(gate_up, a.b, tiles=tiles, rows=order, row_div=k)
        h = kk.glu_f32(y1[:, :F_out], y1[:, F_out:], act, row_clamp)
        return MoeParts(kk.gemm_f32(down, h, tiles=tiles), k, pos, wts, flat_ids)
    if P <= 4 * GEMV_MAX_M:
        flat = ids.reshape(-1)
        gu = torch.empty((P, F_out), dtype=torch.bfloat16, device=ids.device)
        kk.gemv(gate_up, xb=a.b, M=1, ids=flat, x_div=k, act=act, out=gu, clamp=clamp)
        y = torch.empty((P, D), dtype=torch.float32, device=ids.device)
        kk.gemv(down, xb=gu, M=1, ids=flat, x_div=1, out=y)
        return MoeParts(y, k, None, wts, flat_ids)
    avg = max(1, P // E)
    bn = 32 if avg <= 32 else 64 if avg <= 64 else 128 if avg <= 128 else 256
    order, tiles, pos = kk.moe_sort(ids, E, bn)
    xs = kk.gather_bf16_rows(a.b, order, k)
    y1 = kk.gemm_bf16_grouped(_dequant_scratch(gate_up), E, xs, tiles, bn, out_dtype=torch.bfloat16, zero=False)
    h, _, _ = kk.glu(y1, y1[:, F_out:], act, F_out, gate_up.N, gate_up.N, P, clamp=row_clamp)
    y2 = kk.gemm_bf16_grouped(_dequant_scratch(down), E, h, tiles, bn, out_dtype=torch.bfloat16, zero=False)
    return MoeParts(y2, k, pos, wts, flat_ids)


def moe_experts(a: Act, ids: torch.Tensor, weights: torch.Tensor, gate_up: QuantWeight, down: QuantWeight, *,
                act: str, gate_up_bias: Optional[torch.Tensor] = None, down_bias: Optional[torch.Tensor] = None,
                expert_offset: int = 0, down_scale: Optional[torch.Tensor] = None, push=None) -> Optional[torch.Tensor]:
    """sum_k weights[t, k] * down_e(act(gate_up_e(x_t)))  with e = ids[t, k]  -> f32 [T, D].

    ``gate_up`` / ``down`` are expert stacks; when they hold only experts
    ``[expert_offset, expert_offset + E_local)`` (expert parallelism) the other selections are
    skipped and the caller sums the partial results over ranks.  For non-gated activations
    (relu2) ``gate_up`` is the plain up projection.  ``push`` (a ``TpExchange``; small CUDA batches
    only) makes the down projection store its weighted slot rows straight into every rank's
    mailbox - the expert-parallel combine happens in the consumer of the exchange, which adds
    ``k`` parts per source (``reduce_norm(parts=k)``), and nothing is returned."""
    T, k = ids.shape
    D = down.N
    E_local = gate_up.experts
    glu_act = act not in ("relu2", "silu")
    F_out = gate_up.N // 2 if glu_act else gate_up.N
    dev = ids.device
    local = ids - expert_offset
    if expert_offset != 0 or E_local != int(1e9):
        local = torch.where((local >= 0) & (local < E_local), local, torch.full_like(local, -1))
    if dev.type == "cuda" and T * k <= 4 * GEMV_MAX_M:
        kk = _k()
        flat = local.reshape(-1).contiguous()
        if gate_up.uses_q8_activations:
            _ensure_q8(a)
            gu = torch.zeros((T * k, F_out), dtype=torch.bfloat16, device=dev)
            kk.gemv(gate_up, xq=a.q, xds=a.ds, M=1, ids=flat, x_div=k, act=act if glu_act or act == "relu2" else None,
                    bias=gate_up_bias, out=gu)
        else:
            gu = torch.zeros((T * k, F_out), dtype=torch.bfloat16, device=dev)
            kk.gemv(gate_up, xb=a.b.contiguous(), M=1, ids=flat, x_div=k,
                    act=act if glu_act or act == "relu2" else None, bias=gate_up_bias, out=gu)
        if act == "silu":
            gu, _, _ = kk.glu(gu, None, "silu", F_out, F_out, 0, T * k)
        w = weights.reshape(-1).float().contiguous()
        if down_scale is not None:
            w = w * down_scale[ids.reshape(-1).long()]
        pk = dict(push=push.struct.data_ptr()) if push is not None else dict(out=torch.zeros((T * k, D), dtype=torch.float32, device=dev))
        if down.uses_q8_activations:
            gq, gds = kk.quantize_q8(gu)
            y = kk.gemv(down, xq=gq, xds=gds, M=1, ids=flat, x_div=1, bias=down_bias, row_scale=w, **pk)
        else:
            y = kk.gemv(down, xb=gu, M=1, ids=flat, x_div=1, bias=down_bias, row_scale=w, **pk)
        return y.view(T, k, D).sum(1) if push is None else None
    if push is not None:
        raise ValueError("moe_experts(push=...) needs a CUDA batch of at most 4 * GEMV_MAX_M slots")
    if dev.type == "cuda" and T * k <= MOE_TILE_MAX_PAIRS:
        # medium batches (batched decode): routing stays on the device, each expert's rows are streamed
        # once per tile of 8 pairs; the launch sequence is fixed, so the step can be graph-captured
        kk = _k()
        wts = weights.reshape(-1).float()
        if down_scale is not None:
            wts = wts * down_scale[ids.reshape(-1).long()]
        if gate_up.uses_q8_activations:
            _ensure_q8(a)
            return kk.moe_grouped(xq=a.q, xds=a.ds, ids=ids, weights=wts, gate_up=gate_up, down=down, act=act,
                                  gate_up_bias=gate_up_bias, down_bias=down_bias, expert_offset=expert_offset)
        return kk.moe_grouped(xb=a.b.contiguous(), ids=ids, weights=wts, gate_up=gate_up, down=down, act=act,
                              gate_up_bias=gate_up_bias, down_bias=down_bias, expert_offset=expert_offset)
    if dev.type == "cuda" and os.environ.get("TSB_MOE_GROUPED_GEMM", "1") != "0" and gate_up.K % 8 == 0 and down.K % 8 == 0:
        return _moe_grouped_gemm(a, ids, local, weights, gate_up, down, act, gate_up_bias, down_bias, down_scale)
    # per-expert path (CPU oracle, and CUDA with TSB_MOE_GROUPED_GEMM=0): sort the (token, slot) pairs by expert on the
    # host and run each expert on its rows
    out = torch.zeros((T, D), dtype=torch.float32, device=dev)
    flat = local.reshape(-1)
    order = torch.argsort(flat, stable=True)
    counts = torch.bincount((flat[order] + 1).long(), minlength=E_local + 1).tolist()
    x = a.b
    off = counts[0]                      # skipped (non-local) selections sort first (-1)
    wflat = weights.reshape(-1).float()
    if down_scale is not None:
        wflat = wflat * down_scale[ids.reshape(-1).long()]
    for e in range(E_local):
        n = counts[e + 1]
        if n == 0:
            continue
        rows = order[off:off + n]
        off += n
        tok = torch.div(rows, k, rounding_mode="floor")
        xe = Act(x[tok].contiguous())
        gb = gate_up_bias[e] if gate_up_bias is not None else None
        y1 = linear(xe, gate_up.expert(e), bias=gb, act=act, out_dtype=torch.bfloat16 if dev.type == "cuda" else torch.float32)
        db = down_bias[e] if down_bias is not None else None
        y2 = linear(as_act(y1), down.expert(e), bias=db, out_dtype=torch.float32)
        out.index_add_(0, tok, y2 * wflat[rows].unsqueeze(1))
    return out


def moe_tile_list(flat: torch.Tensor, n_groups: int, bn: int):
    """Device-side work list of a grouped GEMM.  ``flat`` [P]: group of every row, -1 = skipped.  Returns ``(order,
    tiles)``: ``order`` sorts the rows by group (skipped rows first), ``tiles`` int32 [ceil(P / bn) + n_groups, 3] holds
    (group or -1, first sorted row, end sorted row) per tile of at most ``bn`` rows.  Nothing is read back to the host:
    the list has a fixed upper-bound length and unused entries are marked -1."""
    P = flat.numel()
    order = torch.argsort(flat, stable=True)
    counts = torch.bincount((flat + 1).long(), minlength=n_groups + 1)
    starts = torch.cumsum(counts, 0) - counts
    cnt, st = counts[1:], starts[1:]
    per = (cnt + bn - 1) // bn
    cum = torch.cumsum(per, 0)
    n_tiles = (P + bn - 1) // bn + n_groups
    t = torch.arange(n_tiles, device=flat.device)
    e = torch.searchsorted(cum, t, right=True)
    valid = e < n_groups
    ec = e.clamp(max=n_groups - 1)
    first = st[ec] + (t - (cum[ec] - per[ec])) * bn
    tiles = torch.stack([torch.where(valid, e, torch.full_like(e, -1)), first, st[ec] + cnt[ec]], 1).to(torch.int32)
    return order, tiles.contiguous()


def _moe_grouped_gemm(a: Act, ids, local, weights, gate_up: QuantWeight, down: QuantWeight, act, gate_up_bias, down_bias,
                      down_scale) -> torch.Tensor:
    """Large batches (prefill): the (token, slot) pairs are sorted by expert on the device, both projections run as one
    grouped tensor-core GEMM each over a device-built tile list (no host read-back, two GEMM launches whatever the
    number of experts), and the weighted rows are added back to their tokens."""
    kk = _k()
    T, k = ids.shape
    D, E = down.N, gate_up.experts
    P = T * k
    avg = max(1, P // max(1, E))
    bn = 32 if avg <= 32 else 64 if avg <= 64 else 128 if avg <= 128 else 256
    flat = local.reshape(-1)
    order, tiles = moe_tile_list(flat, E, bn)
    tok = torch.div(order, k, rounding_mode="floor")
    x = a.b if a.b.dtype == torch.bfloat16 else a.b.to(torch.bfloat16)
    xs = x[tok].contiguous()                                         # rows in expert order
    glu_act = act not in ("relu2", "silu")
    y1 = kk.gemm_bf16_grouped(_dequant_scratch(gate_up), E, xs, tiles, bn, out_dtype=torch.bfloat16,
                              bias=gate_up_bias.float().contiguous() if gate_up_bias is not None else None)
    if glu_act:
        half = gate_up.N // 2
        h, _, _ = kk.glu(y1, y1[:, half:], act, half, gate_up.N, gate_up.N, P)
    else:
        h, _, _ = kk.glu(y1, None, act, gate_up.N, gate_up.N, 0, P)
    y2 = kk.gemm_bf16_grouped(_dequant_scratch(down), E, h, tiles, bn, out_dtype=torch.float32,
                              bias=down_bias.float().contiguous() if down_bias is not None else None)
    w = weights.reshape(-1).float()
    if down_scale is not None:
        w = w * down_scale[ids.reshape(-1).long()]
    if D % 4 == 0:
        # every token gathers its own k rows (fixed summation order, no atomics): pos = where each pair went
        pos = torch.empty(P, dtype=torch.int32, device=ids.device)
        pos[order] = torch.arange(P, dtype=torch.int32, device=ids.device)
        pos = torch.where(flat >= 0, pos, torch.full_like(pos, -1))          # skipped pairs contribute nothing
        return kk.moe_combine_weighted(y2, pos, w, T, k)
    w = torch.where(flat >= 0, w, torch.zeros_like(w))[order]
    out = torch.zeros((T, D), dtype=torch.float32, device=ids.device)
    out.index_add_(0, tok, y2 * w.unsqueeze(1))
    return out


# --------------------------------------------------------------------------------------------
# Recurrent layers (state tensors are indexed by ``batch.seq_slots``)
# --------------------------------------------------------------------------------------------
def causal_conv1d(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, batch: Batch,
                  act_silu: bool = True) -> torch.Tensor:
    """Depth-wise causal conv over the packed tokens; ``state`` [slots, K-1, C] carries each
    sequence's last K-1 inputs between calls.  Returns f32 [T, C]."""
    if x.is_cuda:
        return _k().causal_conv1d(x, w, bias, state, batch.cu_q, batch.seq_slots, batch.max_q_len, act_silu)
    outs = []
    slots = batch.seq_slots.tolist()
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        o, tail = ref.causal_conv1d(x[q0:q1], w, bias, state[slots[b]], act_silu)
        state[slots[b]] = tail
        outs.append(o)
    return torch.cat(outs, 0)


def _gdn_chunk_min() -> int:
    """Prompts of at least this many tokens take the chunked form of the recurrence (the reference's
    GDN_CHUNK_PREFILL_MIN_SEQ_LEN, default 64; GDN_DISABLE_CHUNKED_PREFILL=1 keeps the token-by-token scan)."""
    if os.environ.get("GDN_DISABLE_CHUNKED_PREFILL", "0") not in ("", "0"):
        return 1 << 62
    return max(2, int(os.environ.get("GDN_CHUNK_PREFILL_MIN_SEQ_LEN", "64") or 64))


CUDA_CHUNKED_MIN_TOKENS = 1024


def _use_chunked_scan(batch: Batch, on_cuda: bool, switch: str) -> bool:
    """Whether a recurrent layer runs its chunked form for this batch.  CPU: prompts of ``_gdn_chunk_min()`` tokens or
    more.  CUDA: prompts of ``CUDA_CHUNKED_MIN_TOKENS`` or more (one B200, 2048 tokens: GatedDeltaNet 5.9 ms as a scan,
    3.6 ms chunked; Mamba2 3.3 against 2.9 ms; at 8192 tokens 23.8 / 12.9 and 18.8 / 8.1 ms; at 512 the scan wins);
    ``<switch>=1`` lowers the bar to the CPU's, ``=0`` keeps the scan kernel."""
    if not on_cuda:
        return batch.max_q_len >= _gdn_chunk_min()
    mode = os.environ.get(switch, "")
    if mode == "0":
        return False
    return batch.max_q_len >= (_gdn_chunk_min() if mode == "1" else max(CUDA_CHUNKED_MIN_TOKENS, _gdn_chunk_min()))


def gdn(qkv: torch.Tensor, z: torch.Tensor, beta: torch.Tensor, alpha: torch.Tensor, dt_bias, a_log, norm_w,
        state: torch.Tensor, batch: Batch, *, Hk: int, Hv: int, Dk: int, Dv: int, eps: float) -> torch.Tensor:
    """GatedDeltaNet recurrence over the packed tokens -> gated output [T, Hv*Dv].  Decode steps and short prompts
    run the token-by-token scan (one kernel on CUDA); longer prompts run the chunked form (matrix products over heads x
    chunks; thresholds in :func:`_use_chunked_scan`)."""
    chunked = _use_chunked_scan(batch, qkv.is_cuda, "TSB_GDN_CHUNKED")
    if qkv.is_cuda and not chunked:
        return _k().gdn_recurrent(qkv, z, beta, alpha, dt_bias, a_log, norm_w, state, batch.cu_q, batch.seq_slots,
                                  Hk=Hk, Hv=Hv, Dk=Dk, Dv=Dv, eps=eps)
    slots = batch.seq_slots.tolist()
    if chunked and qkv.is_cuda and os.environ.get("TSB_GDN_CHUNK_KERNELS", "1") != "0" and _k().gdn_chunked_supported(Dk, Dv) \
            and qkv.dtype == torch.float32 and beta.dtype == alpha.dtype and beta.stride(0) == alpha.stride(0):
        return _k().gdn_chunked(qkv, z, beta, alpha, dt_bias, a_log, norm_w, state, batch.cu_q, list(batch.h_cu_q), slots,
                                Hk=Hk, Hv=Hv, Dk=Dk, Dv=Dv, eps=eps)
    if chunked:                                 # every sequence of a batch that took this route, short ones included
        carry = None
        if qkv.is_cuda and os.environ.get("TSB_GDN_CARRY_KERNEL", "1") != "0" and _k().gdn_chunk_carry_supported(Dk, Dv, 64):
            carry = _k().gdn_chunk_carry
        out = ref.gdn_chunked_batch(qkv, z, beta, alpha, dt_bias, a_log, norm_w, [state[sl] for sl in slots], list(batch.h_cu_q),
                                    Hk=Hk, Hv=Hv, Dk=Dk, Dv=Dv, eps=eps, carry=carry)
        return out.to(torch.bfloat16 if qkv.is_cuda else torch.float32)
    outs = []
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        outs.append(ref.gdn_recurrent(qkv[q0:q1], z[q0:q1], beta[q0:q1], alpha[q0:q1], dt_bias, a_log, norm_w, state[slots[b]],
                                      Hk=Hk, Hv=Hv, Dk=Dk, Dv=Dv, eps=eps))
    return torch.cat(outs, 0).to(torch.bfloat16 if qkv.is_cuda else torch.float32)     # the kernel's output types


GENERAL_DELTA_SCAN_MIN = 8          # tokens of the longest portion from which the prompt kernels beat the one-kernel step


def general_delta(y: torch.Tensor, w2: QuantWeight, w0: torch.Tensor, ab: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor, batch: Batch,
                  *, H: int, D: int, n: int, rank: int, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """Generalized delta rule with a decay and a removal rate per key channel over the packed tokens -> gated output
    [T, H * D].  ``y`` rows: r | k | v | removal | gate (H * D each) | low-rank part of the decay (``rank``); ``w2``
    [H * D, rank up to 8], ``w0``: the decay's second map and offset; ``ab``: the removal's offset.  ``state`` f32
    [slots, H, values, keys].  Heads of ``n`` channels are padded with zeros to ``D``."""
    HD = H * D
    if y.is_cuda:
        kk = _k()
        kw = dict(H=H, D=D, n=n, eps=eps, out_dtype=dtype)
        if batch.max_q_len < GENERAL_DELTA_SCAN_MIN:
            return kk.general_delta_short(y, _weight_matrix(w2), w0, ab, norm_w, state, batch.cu_q, batch.seq_slots, rank=w2.K, **kw)
        t = kk.tanh_rows(y, 5 * HD, rank, w2.K, dtype)
        z = linear(Act(t), w2, out_dtype=torch.float32)
        if dtype == torch.bfloat16:
            return kk.general_delta_chunk(y, z, w0, ab, norm_w, state, batch.cu_q, batch.seq_slots, max_q=batch.max_q_len, **kw)
        return kk.general_delta_prompt(y, z, w0, ab, norm_w, state, batch.cu_q, batch.seq_slots, wide=batch.B * HD >= 2048, **kw)
    T, y = y.shape[0], y.float()
    z = torch.tanh(y[:, 5 * HD:5 * HD + rank]) @ w2.dequantize()[:, :rank].t() + w0
    r, k, v, a = (y[:, i * HD:(i + 1) * HD].view(T, H, D) for i in range(4))
    o, slots = torch.empty((T, H, D)), batch.seq_slots.tolist()
    decay, a = ref.delta_decay(z).view(T, H, D), torch.sigmoid(a + ab.view(H, D))
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        o[q0:q1] = ref.general_delta(r[q0:q1], k[q0:q1], v[q0:q1], decay[q0:q1], a[q0:q1], state[slots[b]])
    o = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / n + eps)
    return o.reshape(T, HD) * norm_w * torch.sigmoid(y[:, 4 * HD:5 * HD])


@dataclass
class GatedLinearSpec:
    """Sizes of a gated linear attention mixer (``D``, ``E``: padded key and value head sizes)."""
    H: int
    dim: int
    vdim: int
    tau: float

    def __post_init__(self):
        self.D = (self.dim + 31) // 32 * 32
        pad = 16 if self.vdim <= 128 else 32
        self.E = (self.vdim + pad - 1) // pad * pad
        self.q_scale = self.dim ** -0.5


GATED_LINEAR_CHUNK_MIN = 12          # tokens of the longest portion from which the chunk kernel is used


def gated_linear_segments(batch: Batch, s: GatedLinearSpec) -> int:
    """Pieces in which the chunk kernel takes the batch's sequences: about sixteen warps per SM (one per 16 value columns), no
    fewer than 64 tokens each."""
    warps = batch.B * s.H * s.E // 16
    return max(1, min(round(16 * 148 / warps), batch.max_q_len // 64))


def gated_linear(y: torch.Tensor, s: GatedLinearSpec, cols: Tuple[int, ...], w2: QuantWeight, zb: torch.Tensor, norm_w: torch.Tensor,
                 state: torch.Tensor, batch: Batch, *, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """Gated linear attention with a decay per key channel over the packed tokens -> normed and gated output [T, H * E].  Columns
    ``cols`` of ``y``: queries, keys (H * D each), values, gate (H * E each), low rank part of the decay; ``w2`` [H * D, rank up to
    8], ``zb``: its second map and offset.  ``state`` f32 [slots, H, values, keys].  Heads are padded with zeros."""
    if y.is_cuda:
        kk = _k()
        if y.dtype != torch.bfloat16 or batch.max_q_len < GATED_LINEAR_CHUNK_MIN:
            return kk.gla_step(y, s, cols, _weight_matrix(w2), zb, norm_w, state, batch.cu_q, batch.seq_slots, eps=eps, out_dtype=dtype)
        z = linear(Act(y[:, cols[4]:cols[4] + w2.K]), w2, out_dtype=torch.float32)
        return kk.gla_prompt(y, s, cols, z, zb, norm_w, state, batch.cu_q, batch.seq_slots, eps=eps, max_q=batch.max_q_len,
                             segs=gated_linear_segments(batch, s))
    T, y = y.shape[0], y.float()
    H, D, E = s.H, s.D, s.E
    q, k = (y[:, c:c + H * D].view(T, H, D) for c in cols[:2])
    v = y[:, cols[2]:cols[2] + H * E].view(T, H, E)
    z = y[:, cols[4]:cols[4] + w2.K] @ w2.dequantize().t() + zb
    decay = torch.exp(torch.nn.functional.logsigmoid(z) / s.tau).view(T, H, D)
    o, slots = torch.empty((T, H, E)), batch.seq_slots.tolist()
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        o[q0:q1] = ref.gated_linear(q[q0:q1] * s.q_scale, k[q0:q1], v[q0:q1], decay[q0:q1], state[slots[b]])
    o = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / s.vdim + eps) * norm_w
    return o.reshape(T, H * E) * torch.nn.functional.silu(y[:, cols[3]:cols[3] + H * E])


@dataclass
class RglruSpec:
    """Sizes of a recurrent block with real-gated linear recurrent units: ``blocks`` of ``size`` channels, padded to ``block``."""
    width: int
    blocks: int

    def __post_init__(self):
        self.size = self.width // self.blocks
        self.block = (self.size + 7) // 8 * 8
        self.W = self.blocks * self.block


RGLRU_SCAN_MIN = 5          # tokens of the longest portion from which batches of more than GEMV_MAX_M rows take the scan


def rglru_segments(batch: Batch, s: RglruSpec) -> int:
    """Pieces in which the scan takes the batch's sequences: about 1024 threads per SM, no fewer than 32 tokens each."""
    return max(1, min(round(1024 * 148 / (batch.B * s.W)), batch.max_q_len // 32, 128))


def rglru(y: torch.Tensor, s: RglruSpec, conv_w: torch.Tensor, conv_b: torch.Tensor, gates: QuantWeight, gate_b: torch.Tensor, rate: torch.Tensor,
          conv_state: torch.Tensor, state: torch.Tensor, batch: Batch, *, dtype: torch.dtype) -> torch.Tensor:
    """Recurrent block with real-gated linear recurrent units over the packed tokens -> [T, W].  Rows of ``y``: [output branch (W) |
    input branch (W)]; u = the short convolution of the input branch (``conv_w`` [K, W], ``conv_b``); gates r and i per block:
    sigmoid(``gates`` u + ``gate_b``), ``gates`` a stack of [2 block, block] (r's rows, then i's), ``gate_b`` [2, W]; ``rate`` [W] <= 0
    per channel.  log a = rate r; S <- a S + sqrt(1 - a^2) i u; the result is S gelu(output branch).  ``state`` f32 [slots, W]."""
    W, T = s.W, batch.T
    x = y[:, W:2 * W]
    if y.is_cuda:
        kk = _k()
        if T <= GEMV_MAX_M or batch.max_q_len < RGLRU_SCAN_MIN:
            u = kk.short_conv(x, conv_w, conv_b, conv_state, batch, out_dtype=torch.float32)
            return kk.rglru_step(y, u, s, _weight_matrix(gates), gate_b, rate, state, batch, out_dtype=dtype)
        f32 = y.dtype == torch.float32 and dtype == torch.float32
        u = kk.short_conv(x, conv_w, conv_b, conv_state, batch, block=s.block, out_dtype=dtype)
        tiles = block_tiles(batch, s.blocks, 64 if f32 else 256)
        z = (kk.gemm_f32(gates, u, tiles=tiles) if f32 else
             kk.gemm_bf16_grouped(_dequant_scratch(gates), s.blocks, u, tiles, 256, out_dtype=torch.float32, zero=False))
        return kk.rglru_scan(y, u, z, s, gate_b, rate, state, batch, out_dtype=dtype, segs=rglru_segments(batch, s))
    y = y.float()
    u = _conv_over_time(y[:, W:2 * W], conv_w, conv_b, conv_state, batch)
    z = torch.einsum("tbi,boi->tbo", u.view(T, s.blocks, s.block), gates.dequantize().view(s.blocks, 2 * s.block, s.block))
    r, i = (torch.sigmoid(z[..., p * s.block:(p + 1) * s.block].reshape(T, W) + gate_b[p]) for p in (0, 1))
    out = torch.empty((T, W))
    for b, slot in enumerate(batch.seq_slots.tolist()):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        out[q0:q1] = ref.real_gated_recurrence(u[q0:q1], r[q0:q1], i[q0:q1], rate, state[slot])
    return out * torch.nn.functional.gelu(y[:, :W], approximate="tanh")


def block_tiles(batch: Batch, blocks: int, bn: int) -> torch.Tensor:
    """Work list of a grouped product over ``blocks`` matrices, each with the T rows of the batch (rows block after block): int32
    [n, 3] (matrix, first row, end row), at most ``bn`` rows each; memoised per step."""
    key = ("block_tiles", blocks, bn)
    t = batch.cache.get(key)
    if t is None:
        T = batch.T
        rows = [(b, b * T + r, b * T + min(r + bn, T)) for b in range(blocks) for r in range(0, T, bn)]
        t = batch.cache[key] = torch.tensor(rows, dtype=torch.int32).to(batch.tokens.device)
    return t


@dataclass
class MlstmSpec:
    """Sizes of an mLSTM mixer (``D``, ``E``: padded key and value head sizes); ``cap`` bounds the gates' logarithms."""
    H: int
    dim: int
    vdim: int
    cap: float

    def __post_init__(self):
        self.D = (self.dim + 31) // 32 * 32
        pad = 16 if self.vdim <= 128 else 32
        self.E = (self.vdim + pad - 1) // pad * pad
        self.q_scale = self.dim ** -0.5


MLSTM_CHUNK_MIN = 16          # tokens of the longest portion from which the chunk kernel is used


def mlstm_segments(batch: Batch, s: MlstmSpec) -> int:
    """Pieces in which the chunk kernel takes the batch's sequences: about eight warps per SM (one per 16 value columns), no
    fewer than 128 tokens each."""
    warps = batch.B * s.H * s.E // 16
    return max(1, min(round(8 * 148 / warps), batch.max_q_len // 128))


def mlstm(y: torch.Tensor, s: MlstmSpec, cols: Tuple[int, int, int, int], z: torch.Tensor, zb: torch.Tensor, norm_w: torch.Tensor, S: torch.Tensor,
          n: torch.Tensor, m: torch.Tensor, batch: Batch, *, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """Matrix memory with exponential gates over the packed tokens -> normed and gated output [T, H * E].  Columns ``cols`` of ``y``:
    queries, keys (H * D each), values, output gate (H * E each); ``z`` [T, 2 H] f32 and ``zb``: the input and forget gates'
    projections and offsets, i = cap tanh(z / cap), f = log sigmoid(cap tanh(z / cap)).  The heads' outputs are divided by their
    root mean square, times ``norm_w`` [H * E], times sigmoid of the output gate.  State, f32 with a row per slot: ``S`` [slots, H,
    values, keys], ``n`` [slots, H, keys], ``m`` [slots, H].  Heads are padded with zeros."""
    if y.is_cuda:
        kk = _k()
        kw = dict(eps=eps, out_dtype=dtype)
        if y.dtype != torch.bfloat16 or batch.max_q_len < MLSTM_CHUNK_MIN:
            return kk.mlstm_step(y, s, cols, z, zb, norm_w, S, n, m, batch, **kw)
        return kk.mlstm_prompt(y, s, cols, z, zb, norm_w, S, n, m, batch, segs=mlstm_segments(batch, s), **kw)
    T, y = y.shape[0], y.float()
    H, D, E = s.H, s.D, s.E
    q, k = (y[:, c:c + H * D].view(T, H, D) for c in cols[:2])
    v = y[:, cols[2]:cols[2] + H * E].view(T, H, E)
    z = s.cap * torch.tanh((z.float() + zb) / s.cap)
    i, f = z[:, :H], torch.nn.functional.logsigmoid(z[:, H:])
    o = torch.empty((T, H, E))
    for b, slot in enumerate(batch.seq_slots.tolist()):
        a = slice(batch.h_cu_q[b], batch.h_cu_q[b + 1])
        o[a] = ref.mlstm(q[a] * s.q_scale, k[a], v[a], i[a], f[a], S[slot], n[slot], m[slot])
    o = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / s.vdim + eps)
    return o.reshape(T, H * E) * norm_w * torch.sigmoid(y[:, cols[3]:cols[3] + H * E])


def _weight_matrix(w: QuantWeight) -> torch.Tensor:
    """The [N, K] tensor of a bf16 or f32 weight."""
    from ..gguf.constants import GGMLType
    return w.planes[0].view(torch.bfloat16 if w.ggml_type == GGMLType.BF16 else torch.float32).view(w.rows, w.K)


def mamba2(xbc: torch.Tensor, dt: torch.Tensor, dt_bias, A, D, state: torch.Tensor, batch: Batch, *, H: int, P: int,
           G: int, N: int) -> torch.Tensor:
    """Mamba2 selective scan over the packed tokens -> y f32 [T, H*P] (before gating).  Long prompts take
    the chunked form (thresholds in :func:`_use_chunked_scan`)."""
    chunked = _use_chunked_scan(batch, xbc.is_cuda, "TSB_MAMBA_CHUNKED")
    if xbc.is_cuda and not chunked:
        return _k().mamba2_recurrent(xbc, dt, dt_bias, A, D, state, batch.cu_q, batch.seq_slots, H=H, P=P, G=G, N=N)
    outs = []
    slots = batch.seq_slots.tolist()
    if (chunked and xbc.is_cuda and os.environ.get("TSB_MAMBA_CHUNK_KERNELS", "1") != "0"
            and os.environ.get("TSB_MAMBA_CARRY_KERNEL", "1") != "0" and _k().mamba2_chunked_supported(N, P)
            and _k().gdn_chunk_carry_supported(N, P, 64) and state.dtype == torch.float32 and xbc.dtype == torch.float32
            and batch.B * H <= 65535):
        # the whole batch in two kernels: the chunk-parallel algebra, then the chunk-carry kernel of the delta rule
        return _k().mamba2_chunked(xbc, dt, dt_bias, A, D, state, batch.cu_q, batch.h_cu_q, slots, H=H, P=P, G=G, N=N)
    scan = ref.mamba2_chunked if chunked else ref.mamba2_recurrent
    kw = {}
    if chunked and xbc.is_cuda and os.environ.get("TSB_MAMBA_CARRY_KERNEL", "1") != "0" and _k().gdn_chunk_carry_supported(N, P, 64) \
            and state.dtype == torch.float32:
        kw["carry"] = _k().gdn_chunk_carry          # the state update has the delta rule's shape with nothing to correct
    for b in range(batch.B):
        q0, q1 = batch.h_cu_q[b], batch.h_cu_q[b + 1]
        outs.append(scan(xbc[q0:q1], dt[q0:q1], dt_bias, A, D, state[slots[b]], H=H, P=P, G=G, N=N, **kw))
    return torch.cat(outs, 0)
