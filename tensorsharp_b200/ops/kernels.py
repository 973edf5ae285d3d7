"""ctypes bindings for the sm_100a kernels in ``libtsb200.so``.

Each function takes torch CUDA tensors, passes their raw pointers and the current
stream, and raises on a non-zero status.  There is no fallback here: if the library
is missing the call fails loudly.
"""
from __future__ import annotations

import ctypes as C
import math
import os
from typing import Optional

import torch

from ..quant.qweight import QuantWeight
from . import native

ACT = {None: 0, "none": 0, "swiglu": 1, "geglu": 2, "geglu_tanh": 2, "geglu_erf": 3, "swiglu_oai": 4,
       "relu2": 5, "silu": 6, "sigmoid_mul": 7}

_vp = C.c_void_p


def _p(t: Optional[torch.Tensor]):
    return _vp(t.data_ptr()) if t is not None else _vp(0)


def _stream():
    return _vp(torch.cuda.current_stream().cuda_stream)


# Debug mode TSB_CHECK_INDICES=1: before a launch, every index tensor that the kernel will use to address memory (token
# ids, KV slots, block-table pages, cache lengths, expert ids, state slots) is checked on the host against the size of
# what it indexes, and an IndexError names the kernel and the offending value instead of the kernel reading or writing out
# of bounds.  Each check synchronises the stream, so the mode is for debugging only (and cannot be used while a CUDA
# graph is being captured).  The kernels themselves index unchecked.
CHECK_INDICES = os.environ.get("TSB_CHECK_INDICES", "0") not in ("", "0")


def check_index(kernel: str, what: str, t: Optional[torch.Tensor], limit: int, low: int = 0) -> None:
    """Raise IndexError unless every element of ``t`` lies in ``[low, limit)``.  No-op unless TSB_CHECK_INDICES=1."""
    if not CHECK_INDICES or t is None or t.numel() == 0:
        return
    if t.is_cuda and torch.cuda.is_current_stream_capturing():
        return
    lo, hi = int(t.min().item()), int(t.max().item())
    if lo < low or hi >= limit:
        raise IndexError(f"{kernel}: {what} out of range: values span [{lo}, {hi}], allowed [{low}, {limit})")


def _planes(w: QuantWeight):
    ps = [_vp(p.data_ptr()) for p in w.planes]
    while len(ps) < 4:
        ps.append(_vp(0))
    return ps


class RopeParams(C.Structure):
    _fields_ = [("theta_base", C.c_float), ("freq_scale", C.c_float), ("ext_factor", C.c_float),
                ("attn_factor", C.c_float), ("corr_lo", C.c_float), ("corr_hi", C.c_float),
                ("rot_dim", C.c_int), ("mode", C.c_int)]


class QkvArgs(C.Structure):
    _fields_ = [("q", _vp), ("k", _vp), ("v", _vp),
                ("q_tok", C.c_long), ("q_head", C.c_long), ("k_tok", C.c_long), ("k_head", C.c_long),
                ("v_tok", C.c_long), ("v_head", C.c_long),
                ("in_f32", C.c_int), ("qn", _vp), ("kn", _vp), ("v_norm", C.c_int), ("eps", C.c_float),
                ("pos", _vp), ("slot", _vp), ("freq_factors", _vp), ("cs_table", _vp), ("q_out", _vp), ("k_cache", _vp),
                ("v_cache", _vp), ("q_scale", C.c_float),
                ("T", C.c_int), ("Hq", C.c_int), ("Hkv", C.c_int), ("Dh", C.c_int), ("rp", RopeParams),
                ("Dv", C.c_int), ("norm_n", C.c_int), ("qt_coef", C.c_float), ("qt_every", C.c_float), ("out_f32", C.c_int)]


class AttnArgs(C.Structure):
    _fields_ = [("q", _vp), ("k_cache", _vp), ("v_cache", _vp), ("out", _vp), ("block_table", _vp),
                ("kv_lens", _vp), ("cu_q", _vp), ("sinks", _vp), ("part_o", _vp), ("part_ml", _vp),
                ("scale", C.c_float), ("softcap", C.c_float), ("window", C.c_int),
                ("B", C.c_int), ("Hq", C.c_int), ("Hkv", C.c_int), ("Dh", C.c_int), ("page_size", C.c_int),
                ("max_pages", C.c_int), ("splits", C.c_int), ("q_pos0", _vp), ("lse_out", _vp),
                ("out_q", _vp), ("out_ds", _vp), ("ticket", _vp), ("split_len", C.c_int),
                ("gate", _vp), ("gate_tok", C.c_long), ("gate_f32", C.c_int), ("Dv", C.c_int),
                ("k_ld", C.c_long), ("v_ld", C.c_long), ("keep_first", C.c_int), ("slopes", _vp), ("gate_cols", C.c_int),
                ("kv_scale", C.c_int), ("log_r1", _vp), ("log_r2", _vp), ("sig_bias", _vp)]


_configured = False
LAUNCHES = 0          # kernels launched through this module (eager mode; graph replays add theirs)


def _count(n: int = 1) -> None:
    global LAUNCHES
    LAUNCHES += n


def _lib():
    global _configured
    lib = native.lib()
    if not _configured:
        for name in ("tsb_quantize_q8", "tsb_gemv", "tsb_rmsnorm", "tsb_qkv_rope", "tsb_glu", "tsb_gather_rows",
                     "tsb_argmax", "tsb_rope_table", "tsb_fused_gemv", "tsb_gemv_push", "tsb_tp_reduce_norm", "tsb_tpseq_push_rows", "tsb_decode_advance", "tsb_attn_decode", "tsb_attn_prefill", "tsb_gemm_bf16", "tsb_causal_conv1d", "tsb_gdn_recurrent",
                     "tsb_mamba2_recurrent"):
            fn = getattr(lib, name, None)             # a library linked from a selection of sources lacks some
            if fn is not None:
                fn.restype = C.c_int
        _configured = True
    return lib


# --------------------------------------------------------------------------------------------
def quantize_q8(x: torch.Tensor):
    """x [rows, K] (bf16 or f32) -> (int8 [rows, K], float32 [rows, K/32, 2])."""
    assert x.is_cuda and x.is_contiguous()
    rows, K = x.shape
    xq = torch.empty((rows, K), dtype=torch.int8, device=x.device)
    xds = torch.empty((rows, K // 32, 2), dtype=torch.float32, device=x.device)
    native.check(_lib().tsb_quantize_q8(_p(x), C.c_int(x.dtype == torch.float32), _p(xq), _p(xds), C.c_long(rows),
                                        C.c_int(K), _stream()), "quantize_q8")
    _count(1)
    return xq, xds


def gemv(w: QuantWeight, *, xq=None, xds=None, xb=None, M: int, out_dtype=torch.float32, bias=None, residual=None,
         act=None, ids=None, row_scale=None, x_div: int = 1, out: Optional[torch.Tensor] = None,
         push: Optional[int] = None, clamp=None) -> Optional[torch.Tensor]:
    """Small-batch matvec over quantised weights.  With ``ids`` ([P] int32) each problem p
    uses expert ids[p], activation row p // x_div and output row p.  ``push`` (device address of a
    tensor-parallel exchange descriptor) sends the f32 result to every rank's mailbox instead of
    ``out``.  ``clamp`` (limit, limit of the first experts, how many): the clamp of "swiglu_oai" (default 7)."""
    a = ACT[act]
    glu = 1 <= a <= 4
    lim, lim_first, n_first = clamp or (7.0, 7.0, 0)
    n_out = w.N // 2 if glu else w.N
    problems = int(ids.numel()) if ids is not None else 1
    rows = problems if ids is not None else M
    dev = w.device
    if out is None and push is None:
        out = torch.empty((rows, n_out), dtype=out_dtype, device=dev)
    ps = _planes(w)
    native.check(_lib().tsb_gemv_clamped(ps[0], ps[1], ps[2], ps[3], C.c_int(int(w.ggml_type)), C.c_int(w.N), C.c_int(w.K),
                                         _p(xq), _p(xds), _p(xb), _p(out), _p(bias), _p(residual), _p(ids), _p(row_scale),
                                         C.c_int(M), C.c_int(problems), C.c_int(x_div),
                                         C.c_int(1 if (out is None or out.dtype == torch.float32) else 0), C.c_int(a),
                                         C.c_void_p(push) if push else None, C.c_float(lim), C.c_float(lim_first), C.c_int(n_first),
                                         _stream()), "gemv")
    _count(1)
    return out


def gemv_multi(ws, *, xq=None, xds=None, xb=None, M: int, out_dtype=torch.float32) -> torch.Tensor:
    """Two or three weight matrices over the same activations in one launch -> [M, sum of rows]."""
    n = len(ws)
    planes = (C.c_void_p * (4 * n))()
    for i, w in enumerate(ws):
        for j, p in enumerate(_planes(w)):
            planes[4 * i + j] = p.value if hasattr(p, "value") else p
    types = (C.c_int * n)(*[int(w.ggml_type) for w in ws])
    rows = (C.c_int * n)(*[w.N for w in ws])
    total = sum(w.N for w in ws)
    out = torch.empty((M, total), dtype=out_dtype, device=ws[0].device)
    native.check(_lib().tsb_gemv_multi(planes, types, rows, C.c_int(n), C.c_int(ws[0].K), _p(xq), _p(xds), _p(xb), _p(out),
                                       C.c_int(M), C.c_int(1 if out_dtype == torch.float32 else 0), _stream()), "gemv_multi")
    _count(1)
    return out


def moe_route(logits: torch.Tensor, k: int, *, mode: int = 0, sel_bias=None, normalize: bool = False, scale: float = 1.0,
              n_experts: Optional[int] = None, n_always: int = 0):
    """Router on the device: f32 logits [T, E] -> (ids int32 [T, k], weights f32 [T, k]).  mode 0: top-k
    then softmax over the selected; mode 1: sigmoid, selection on p + sel_bias, optional renormalise, scale;
    mode 2: softmax over all, top-k, divided by the selected's sum (+ 1e-20), scale.  ``n_experts``: only the
    first of the columns are routed experts; ``n_always``: that many further ids follow on every token,
    weighted sigmoid(logits[:, n_experts])."""
    assert logits.is_cuda and logits.dtype == torch.float32 and logits.is_contiguous()
    T, ld = logits.shape
    E, ko = n_experts or ld, k + n_always
    ids = torch.empty((T, ko), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, ko), dtype=torch.float32, device=logits.device)
    native.check(_lib().tsb_moe_route_ex(_p(logits), _p(sel_bias), C.c_int(T), C.c_int(E), C.c_int(k), C.c_int(mode),
                                         C.c_int(1 if normalize else 0), C.c_float(scale), C.c_int(ld), C.c_int(n_always), _p(ids), _p(w),
                                         _stream()), "moe_route")
    _count(1)
    return ids, w


def moe_route_grouped(logits: torch.Tensor, k: int, *, correction, groups: int, keep: int, n_real: int, n_always: int = 0, scale: float = 1.0):
    """Router with groups of neighbours and identity experts (functional.py: route_softmax_groups): f32 logits [T, E] ->
    (ids int32, weights f32), both [T, n_always + k]."""
    assert logits.is_cuda and logits.dtype == torch.float32 and logits.is_contiguous()
    T, E = logits.shape
    ids = torch.empty((T, n_always + k), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, n_always + k), dtype=torch.float32, device=logits.device)
    native.check(_lib().tsb_moe_route_grouped(_p(logits), _p(correction), C.c_int(T), C.c_int(E), C.c_int(n_real), C.c_int(k), C.c_int(groups),
                                              C.c_int(keep), C.c_float(scale), C.c_int(n_always), _p(ids), _p(w), _stream()), "moe_route")
    _count(1)
    return ids, w


def moe_sort(ids: torch.Tensor, E: int, bn: int):
    """Sort the (token, slot) pairs of ``ids`` (int32, every value in [0, E) or negative) by expert on the device.  Returns
    ``order`` (the pair at each sorted place; -1 at the end, for the pairs with a negative id), ``tiles`` int32
    [ceil(P / bn) + E, 3] (expert or -1, first, end place; at most bn places each) and ``pos`` (the sorted place of each pair, -1
    for a negative id)."""
    assert ids.dtype == torch.int32 and ids.is_contiguous()
    check_index("moe_sort", "expert id", ids, E, low=-1)
    P, dev = ids.numel(), ids.device
    n_tiles = (P + bn - 1) // bn + E
    order, pos = torch.empty(P, dtype=torch.int32, device=dev), torch.empty(P, dtype=torch.int32, device=dev)
    tiles = torch.empty((n_tiles, 3), dtype=torch.int32, device=dev)
    counts = torch.empty(((P + 1023) // 1024, E), dtype=torch.int32, device=dev) if P > 4096 else None
    native.check(_lib().tsb_moe_sort(_p(ids), C.c_int(P), C.c_int(E), C.c_int(bn), _p(order), _p(pos), _p(tiles), C.c_int(n_tiles), _p(counts),
                                     _stream()), "moe_sort")
    _count(1 if counts is None else 3)
    return order, tiles, pos


def gather_bf16_rows(x: torch.Tensor, order: torch.Tensor, div: int) -> torch.Tensor:
    """x[order // div] for bf16 rows (what stands in rows with a negative order is undefined)."""
    assert x.dtype == torch.bfloat16 and x.is_contiguous() and order.dtype == torch.int32
    out = torch.empty((order.numel(), x.shape[1]), dtype=torch.bfloat16, device=x.device)
    native.check(_lib().tsb_gather_bf16_rows(_p(x), _p(order), C.c_int(order.numel()), C.c_int(div), C.c_int(x.shape[1]), _p(out), _stream()),
                 "gather_bf16_rows")
    _count(1)
    return out


def moe_grouped(*, xq=None, xds=None, xb=None, ids: torch.Tensor, weights: torch.Tensor, gate_up: QuantWeight,
                down: QuantWeight, act, gate_up_bias=None, down_bias=None, expert_offset: int = 0) -> torch.Tensor:
    """Grouped expert projections with the routing kept on the device (no host read-back, fixed launch
    sequence): group the (token, slot) pairs by local expert, gather activations into that order, run
    gate/up and down as tile GEMVs (each tile streams its expert's rows once for up to 8 pairs), and
    sum every token's slots.  ``ids`` are global expert ids [T, k]; pairs whose expert is not in
    ``[expert_offset, expert_offset + gate_up.experts)`` contribute nothing.  Returns f32 [T, D]."""
    lib = _lib()
    T, k = ids.shape
    P = T * k
    dev = ids.device
    E_local = gate_up.experts
    a = ACT[act]
    glu = 1 <= a <= 4
    F_out = gate_up.N // 2 if glu else gate_up.N
    D, K = down.N, gate_up.K
    ids = ids.contiguous()
    pos = torch.empty((P,), dtype=torch.int32, device=dev)
    max_tiles = int(lib.tsb_moe_max_tiles(C.c_int(P), C.c_int(E_local)))
    tiles = torch.empty((max_tiles, 4), dtype=torch.int32, device=dev)
    meta = torch.empty((2,), dtype=torch.int32, device=dev)
    native.check(lib.tsb_moe_group(_p(ids), C.c_int(P), C.c_int(expert_offset), C.c_int(E_local), _p(pos), _p(tiles), _p(meta),
                                   _stream()), "moe_group")
    sq = sds = sb = None
    if xq is not None:
        sq = torch.zeros((P, K), dtype=torch.int8, device=dev)
        sds = torch.zeros((P, K // 32, 2), dtype=torch.float32, device=dev)
    else:
        sb = torch.zeros((P, K), dtype=torch.bfloat16, device=dev)
    sw = torch.zeros((P,), dtype=torch.float32, device=dev)
    wflat = weights.reshape(-1).float().contiguous()
    native.check(lib.tsb_moe_gather(_p(pos), C.c_int(P), C.c_int(k), C.c_int(K), _p(xq), _p(xds), _p(xb), _p(wflat), _p(sq),
                                    _p(sds), _p(sb), _p(sw), _stream()), "moe_gather")
    gu = torch.zeros((P, F_out), dtype=torch.bfloat16, device=dev)
    ps = _planes(gate_up)
    native.check(lib.tsb_moe_gemv_tiles(ps[0], ps[1], ps[2], ps[3], C.c_int(int(gate_up.ggml_type)), C.c_int(gate_up.N), C.c_int(K),
                                        _p(sq), _p(sds), _p(sb), _p(gu), _p(gate_up_bias), None, _p(tiles), _p(meta),
                                        C.c_int(max_tiles), C.c_int(0), C.c_int(a), _stream()), "moe_gemv_tiles(gate_up)")
    y = torch.empty((P, D), dtype=torch.float32, device=dev)
    ps = _planes(down)
    if down.uses_q8_activations:
        gq, gds = quantize_q8(gu)
        gb = None
    else:
        gq = gds = None
        gb = gu
    native.check(lib.tsb_moe_gemv_tiles(ps[0], ps[1], ps[2], ps[3], C.c_int(int(down.ggml_type)), C.c_int(D), C.c_int(F_out),
                                        _p(gq), _p(gds), _p(gb), _p(y), _p(down_bias), _p(sw), _p(tiles), _p(meta),
                                        C.c_int(max_tiles), C.c_int(1), C.c_int(0), _stream()), "moe_gemv_tiles(down)")
    out = torch.empty((T, D), dtype=torch.float32, device=dev)
    native.check(lib.tsb_moe_combine(_p(y), _p(pos), C.c_int(T), C.c_int(k), C.c_int(D), _p(out), _stream()), "moe_combine")
    _count(5)
    return out


def moe_combine_weighted(y: torch.Tensor, pos: torch.Tensor, w: torch.Tensor, T: int, k: int) -> torch.Tensor:
    """out[t] = sum_j w[t, j] * y[pos[t * k + j]] (f32 rows; pos < 0 = no row): each token gathers its own rows, so the
    sum has a fixed order and needs no atomics."""
    D = y.shape[1]
    assert y.dtype == torch.float32 and y.is_contiguous() and pos.dtype == torch.int32 and w.dtype == torch.float32
    out = torch.empty((T, D), dtype=torch.float32, device=y.device)
    lib = _lib()
    lib.tsb_moe_combine_weighted.restype = C.c_int
    native.check(lib.tsb_moe_combine_weighted(_p(y), _p(pos.contiguous()), _p(w.contiguous()), C.c_int(T), C.c_int(k), C.c_int(D),
                                              _p(out), _stream()), "moe_combine_weighted")
    _count(1)
    return out


def sample(logits: torch.Tensor, ngen: torch.Tensor, *, temperature: float, top_k: int, top_p: float, min_p: float,
           repetition_penalty: float = 1.0, presence_penalty: float = 0.0, frequency_penalty: float = 0.0, seed: int = 0,
           counts: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Draw one token per row of f32 logits [B, V] on the device (reference order of transformations).
    ``ngen`` [B] int32 counts the tokens drawn so far per row and keys the random stream; ``counts``
    [B, V] int32 holds the occurrences of each id for the penalties.  Both are advanced by the kernel."""
    assert logits.is_cuda and logits.dtype == torch.float32 and logits.is_contiguous()
    B, V = logits.shape
    if out is None:
        out = torch.empty((B,), dtype=torch.int32, device=logits.device)
    native.check(_lib().tsb_sample(_p(logits), _p(counts), _p(ngen), _p(out), C.c_int(B), C.c_int(V), C.c_float(temperature),
                                   C.c_int(top_k), C.c_float(top_p), C.c_float(min_p), C.c_float(repetition_penalty),
                                   C.c_float(presence_penalty), C.c_float(frequency_penalty),
                                   C.c_ulonglong(seed & 0xFFFFFFFFFFFFFFFF), _stream()), "sample")
    _count(1)
    return out


def device_sampler_supports(cfg) -> bool:
    """Settings the device sampler reproduces exactly (the rest stay with the host sampler)."""
    if cfg.temperature <= 0:
        return True
    return (1 <= cfg.top_k <= 1024) or (cfg.top_k <= 0 and cfg.top_p >= 1.0)


def fused_gemv(w: QuantWeight, *, x_f32=None, x_bf16=None, norm_w=None, eps: float = 0.0, do_norm: bool = False,
               out_dtype=torch.float32, bias=None, residual=None, act=None, out: Optional[torch.Tensor] = None,
               push: Optional[int] = None) -> Optional[torch.Tensor]:
    """Decode GEMV (at most 4 rows) with RMSNorm / cast + int8 quantisation of the input done
    inside the kernel.  ``push`` is the device address of a tensor-parallel exchange descriptor:
    the result then goes to the mailboxes and nothing is returned."""
    x = x_f32 if x_f32 is not None else x_bf16
    assert x.is_cuda and x.is_contiguous() and x.shape[-1] == w.K
    M = x.numel() // w.K
    a = ACT[act]
    glu = 1 <= a <= 4
    n_out = w.N // 2 if glu else w.N
    if push is None and out is None:
        out = torch.empty((M, n_out), dtype=out_dtype, device=w.device)
    ps = _planes(w)
    lib = _lib()
    native.check(lib.tsb_fused_gemv(ps[0], ps[1], ps[2], ps[3], C.c_int(int(w.ggml_type)), C.c_int(w.N), C.c_int(w.K),
                                    _p(x_f32), _p(x_bf16), _p(norm_w), C.c_float(eps), C.c_int(1 if do_norm else 0),
                                    _p(out), _p(bias), _p(residual), C.c_int(M),
                                    C.c_int(1 if (out is None or out.dtype == torch.float32) else 0), C.c_int(a),
                                    C.c_void_p(push) if push else None, _stream()), "fused_gemv")
    _count(1)
    return out


def rmsnorm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float, *, delta=None, want_bf16=True, want_q8=False,
            want_f32=False, add=None, l2=False):
    """Fused (x += delta) -> RMSNorm -> {bf16, f32 (+add), q8}.  Returns (y_bf16, y_f32, yq, yds)."""
    assert x.is_cuda and x.is_contiguous()
    D = x.shape[-1]
    rows = x.numel() // D
    dev = x.device
    yb = torch.empty(x.shape, dtype=torch.bfloat16, device=dev) if want_bf16 else None
    yf = torch.empty(x.shape, dtype=torch.float32, device=dev) if (want_f32 or add is not None) else None
    yq = yds = None
    if want_q8:
        yq = torch.empty((rows, D), dtype=torch.int8, device=dev)
        yds = torch.empty((rows, D // 32, 2), dtype=torch.float32, device=dev)
    native.check(_lib().tsb_rmsnorm(_p(x), C.c_int(x.dtype == torch.float32), _p(delta), _p(w), C.c_float(eps),
                                    C.c_long(rows), C.c_int(D), _p(yb), _p(yf), _p(add), _p(yq), _p(yds),
                                    C.c_int(1 if l2 else 0), _stream()), "rmsnorm")
    _count(1)
    return yb, yf, yq, yds


def yarn_corr_dims(n_dims: int, n_ctx_orig: int, freq_base: float, beta_fast: float, beta_slow: float):
    """ggml's rope_yarn_corr_dims: the pair-index range over which YaRN blends."""
    def corr(n_rot):
        return n_dims * math.log(n_ctx_orig / (n_rot * 2 * math.pi)) / (2 * math.log(freq_base))
    lo = max(0.0, math.floor(corr(beta_fast)))
    hi = min(n_dims - 1.0, math.ceil(corr(beta_slow)))
    return lo, hi


def qkv_rope(*, q, k, v, q_strides, k_strides, v_strides, Hq, Hkv, Dh, pos, slot, q_out, k_cache, v_cache,
             qn=None, kn=None, v_norm=False, eps=1e-6, rope: RopeParams, freq_factors=None, q_scale=1.0,
             cs_table=None, Dv=None, norm_n=None, q_temp=None, out_f32=False):
    T = int(pos.numel())
    check_index("qkv_rope", "KV slot", slot, k_cache.shape[0] if k_cache is not None else 1 << 62)
    check_index("qkv_rope", "position", pos, 1 << 31)
    a = QkvArgs()
    a.q, a.k, a.v = _p(q), _p(k), _p(v)
    a.q_tok, a.q_head = q_strides
    a.k_tok, a.k_head = k_strides
    a.v_tok, a.v_head = v_strides
    a.in_f32 = int(q.dtype == torch.float32)
    a.qn, a.kn = _p(qn), _p(kn)
    a.v_norm = int(v_norm)
    a.eps = eps
    a.pos, a.slot, a.freq_factors = _p(pos), _p(slot), _p(freq_factors)
    a.cs_table = _p(cs_table)
    a.q_out, a.k_cache, a.v_cache = _p(q_out), _p(k_cache), _p(v_cache)
    a.q_scale = q_scale
    a.T, a.Hq, a.Hkv, a.Dh = T, Hq, Hkv, Dh
    a.rp = rope
    a.Dv, a.norm_n, a.out_f32 = Dv or Dh, norm_n or Dh, int(out_f32)
    a.qt_coef, a.qt_every = q_temp or (0.0, 0.0)
    native.check(_lib().tsb_qkv_rope(C.byref(a), _stream()), "qkv_rope")
    _count(1)


def rope_table(pos: torch.Tensor, rope: RopeParams, freq_factors=None) -> torch.Tensor:
    """(cos, sin) for every (token, rotary pair): float32 [T, rot_dim / 2, 2]."""
    T = int(pos.numel())
    out = torch.empty((T, rope.rot_dim // 2, 2), dtype=torch.float32, device=pos.device)
    native.check(_lib().tsb_rope_table(_p(pos), C.byref(rope), _p(freq_factors), _p(out), C.c_int(T), _stream()),
                 "rope_table")
    _count(1)
    return out


def glu(gate: torch.Tensor, up: Optional[torch.Tensor], act: str, F: int, g_stride: int, u_stride: int, rows: int,
        want_bf16=True, want_q8=False, clamp=None):
    """``clamp`` (limit, limit of the first rows, how many): the clamp of "swiglu_oai" (default 7)."""
    dev = gate.device
    lim, lim_first, rows_first = clamp or (7.0, 7.0, 0)
    out = torch.empty((rows, F), dtype=torch.bfloat16, device=dev) if want_bf16 else None
    yq = yds = None
    if want_q8:
        yq = torch.empty((rows, F), dtype=torch.int8, device=dev)
        yds = torch.empty((rows, F // 32, 2), dtype=torch.float32, device=dev)
    native.check(_lib().tsb_glu(_p(gate), _p(up), C.c_int(gate.dtype == torch.float32), C.c_long(g_stride),
                                C.c_long(u_stride), C.c_long(rows), C.c_int(F), C.c_int(ACT[act]), _p(out), _p(yq),
                                _p(yds), C.c_float(lim), C.c_float(lim_first), C.c_long(rows_first), _stream()), "glu")
    _count(1)
    return out, yq, yds


def gather_rows(w: QuantWeight, ids: Optional[torch.Tensor], scale: float = 1.0, out_dtype=torch.bfloat16,
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Embedding lookup (ids given) or whole-matrix decode to ``out_dtype`` (ids None)."""
    n = int(ids.numel()) if ids is not None else w.rows
    check_index("gather_rows", "row id", ids, w.rows)
    if out is None:
        out = torch.empty((n, w.K), dtype=out_dtype, device=w.device)
    ps = _planes(w)
    native.check(_lib().tsb_gather_rows(ps[0], ps[1], ps[2], ps[3], C.c_int(int(w.ggml_type)), C.c_int(w.rows),
                                        C.c_int(w.K), _p(ids), C.c_long(n), C.c_float(scale), _p(out),
                                        C.c_int(out.dtype == torch.float32), _stream()), "gather_rows")
    _count(1)
    return out


def argmax(logits: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    assert logits.dtype == torch.float32 and logits.stride(-1) == 1
    rows, V = logits.shape
    if out is None:
        out = torch.empty((rows,), dtype=torch.int32, device=logits.device)
    native.check(_lib().tsb_argmax(_p(logits), C.c_long(logits.stride(0)), C.c_long(rows), C.c_int(V), _p(out), _vp(0),
                                   _stream()), "argmax")
    _count(1)
    return out


def decode_advance(sampled, batch) -> None:
    """In-place, on the device: next tokens = sampled, positions / kv_lens += 1, new KV slots."""
    B = batch.tokens.shape[0]
    native.check(_lib().tsb_decode_advance(_p(sampled), _p(batch.tokens), _p(batch.positions), _p(batch.kv_lens),
                                           _p(batch.slots), _p(batch.block_table), C.c_int(batch.block_table.shape[1]),
                                           C.c_int(batch.page_size), C.c_int(B), _stream()), "decode_advance")
    _count(1)


def _attn_args(q, k_cache, v_cache, out, block_table, kv_lens, cu_q, sinks, scale, softcap, window, Hq, Hkv, Dh,
               page_size, B, Dv=None, gate=None, keep_first=0, slopes=None, kv_scale=0, log_bias=None, sigmoid_bias=None):
    check_index("attention", "block-table page", block_table, k_cache.shape[0] // page_size)
    check_index("attention", "cache length", kv_lens, block_table.shape[1] * page_size + 1)
    a = AttnArgs()
    a.q, a.k_cache, a.v_cache, a.out = _p(q), _p(k_cache), _p(v_cache), _p(out)
    a.block_table, a.kv_lens, a.cu_q, a.sinks = _p(block_table), _p(kv_lens), _p(cu_q), _p(sinks)
    a.scale, a.softcap, a.window = scale, softcap or 0.0, int(window or 0)
    a.B, a.Hq, a.Hkv, a.Dh, a.page_size = B, Hq, Hkv, Dh, page_size
    a.max_pages = block_table.shape[1]
    a.splits = 1
    a.Dv = Dv or Dh
    assert slopes is None or (slopes.dtype == torch.float32 and slopes.is_contiguous() and slopes.numel() == Hq)
    a.keep_first, a.slopes, a.kv_scale = int(keep_first) if window else 0, _p(slopes), int(kv_scale)
    for t in (*(log_bias or ()), sigmoid_bias):
        assert t is None or (t.dtype == torch.float32 and t.is_contiguous() and t.numel() == Hq)
    if log_bias is not None:
        a.log_r1, a.log_r2 = _p(log_bias[0]), _p(log_bias[1])
    a.sig_bias = _p(sigmoid_bias)
    if kv_scale:                          # rows that are key and value at once, with the factor of the key behind them
        assert k_cache.dim() == 3 and k_cache.stride(2) == 1 and k_cache.shape[-1] >= kv_scale + 1 and kv_scale >= Hkv * Dh
        a.k_ld = a.v_ld = k_cache.stride(0)
        k_cache = v_cache = None
    # a slot's rows may be a slice of a wider row (no gaps between the heads)
    for c, heads, d, ld in ((k_cache, Hkv, Dh, "k_ld"), (v_cache, Hkv, Dv or Dh, "v_ld")):
        if c is not None and c.dim() == 3 and c.stride(0) != heads * d:
            assert c.stride(2) == 1 and (heads == 1 or c.stride(1) == d)
            setattr(a, ld, c.stride(0))
    if gate is not None:
        assert gate.stride(1) == 1 and gate.shape[0] == q.shape[0] and gate.shape[1] in (Hq, Hq * a.Dv)
        a.gate_cols = int(gate.shape[1] != Hq)
        a.gate, a.gate_tok, a.gate_f32 = gate.data_ptr(), gate.stride(0), int(gate.dtype == torch.float32)
    return a


def attn_decode(q, k_cache, v_cache, block_table, kv_lens, *, scale, Hq, Hkv, Dh, page_size, splits, sinks=None,
                softcap=0.0, window=0, out=None, want_q8=False, split_len=0, Dv=None, gate=None, **forms):
    """q [B, Hq, Dh] bf16; one query per sequence against the paged cache.  ``want_q8`` also returns the
    output as int8 groups of 32 with (scale, sum) written by the combine kernel: (out, q, ds).  ``forms``: keep_first,
    slopes, kv_scale, log_bias, sigmoid_bias (see AttnArgs)."""
    B = q.shape[0]
    Dv = Dv or Dh
    if out is None:
        out = torch.empty((B, Hq, Dv), dtype=q.dtype, device=q.device)
    a = _attn_args(q, k_cache, v_cache, out, block_table, kv_lens, None, sinks, scale, softcap, window, Hq, Hkv, Dh,
                   page_size, B, Dv, gate, **forms)
    a.splits = splits
    a.split_len = split_len
    part_o = torch.empty((B, Hq, splits, Dv), dtype=torch.float32, device=q.device)
    part_ml = torch.empty((B, Hq, splits, 2), dtype=torch.float32, device=q.device)
    a.part_o, a.part_ml = _p(part_o), _p(part_ml)
    oq = ods = None
    if want_q8 and Dh % 32 == 0:
        oq = torch.empty((B, Hq * Dh), dtype=torch.int8, device=q.device)
        ods = torch.empty((B, Hq * Dh // 32, 2), dtype=torch.float32, device=q.device)
        a.out_q, a.out_ds = oq.data_ptr(), ods.data_ptr()
    if k_cache.dtype in FP8_DTYPES:           # e4m3 pages: the split kernel that reads bytes, the same merge kernel
        lib = _lib()
        lib.tsb_attn_decode_fp8.restype = C.c_int
        native.check(lib.tsb_attn_decode_fp8(C.byref(a), _stream()), "attn_decode_fp8")
    else:
        native.check(_lib().tsb_attn_decode(C.byref(a), _stream()), "attn_decode")
    _count(2)
    return (out, oq, ods) if want_q8 else out


FP8_DTYPES = (torch.float8_e4m3fn,)


def kv_store_fp8(k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, slots: torch.Tensor) -> None:
    """Dense bf16 rows ``k`` / ``v`` ``[T, Hkv, Dh]`` -> e4m3 bytes at ``slots`` (int64 ``[T]``) of the paged caches."""
    assert k.dtype == v.dtype == torch.bfloat16 and k.is_contiguous() and v.is_contiguous() and slots.dtype == torch.int64
    assert k_cache.dtype in FP8_DTYPES and v_cache.dtype in FP8_DTYPES and k_cache.is_contiguous() and v_cache.is_contiguous()
    T, Hkv, Dh = k.shape
    check_index("kv_store_fp8", "cache slot", slots, k_cache.shape[0])
    lib = _lib()
    lib.tsb_kv_store_fp8.restype = C.c_int
    native.check(lib.tsb_kv_store_fp8(_p(k), _p(v), _p(k_cache), _p(v_cache), _p(slots), C.c_long(T), C.c_int(Hkv), C.c_int(Dh),
                                      _stream()), "kv_store_fp8")
    _count(1)


def kv_load_fp8(k_cache: torch.Tensor, v_cache: torch.Tensor, idx: torch.Tensor):
    """Rows ``idx`` (int64 ``[n]``) of the e4m3 caches as dense bf16 ``[n, Hkv, Dh]`` tensors (K, V)."""
    assert k_cache.dtype in FP8_DTYPES and v_cache.dtype in FP8_DTYPES and idx.dtype == torch.int64 and idx.is_contiguous()
    n, (_, Hkv, Dh) = idx.numel(), k_cache.shape
    check_index("kv_load_fp8", "cache slot", idx, k_cache.shape[0])
    ko = torch.empty((n, Hkv, Dh), dtype=torch.bfloat16, device=idx.device)
    vo = torch.empty_like(ko)
    lib = _lib()
    lib.tsb_kv_load_fp8.restype = C.c_int
    native.check(lib.tsb_kv_load_fp8(_p(k_cache), _p(v_cache), _p(idx), _p(ko), _p(vo), C.c_long(n), C.c_int(Hkv), C.c_int(Dh),
                                     _stream()), "kv_load_fp8")
    _count(1)
    return ko, vo


def attn_prefill(q, k_cache, v_cache, block_table, kv_lens, cu_q, max_q_len, *, scale, Hq, Hkv, Dh, page_size,
                 sinks=None, softcap=0.0, window=0, out=None, q_pos0=None, lse_out=None, Dv=None, gate=None, **forms):
    """q [T, Hq, Dh] bf16 packed over sequences (cu_q [B+1]).  ``q_pos0`` [B] int32 overrides the cache
    position of each sequence's first query (default kv_len - q_len); ``lse_out`` [T, Hq] f32 receives the
    log-sum-exp of the scores, for merging partial results over KV shards."""
    B = kv_lens.shape[0]
    if out is None:
        out = torch.empty((q.shape[0], Hq, Dv or Dh), dtype=q.dtype, device=q.device)
    a = _attn_args(q, k_cache, v_cache, out, block_table, kv_lens, cu_q, sinks, scale, softcap, window, Hq, Hkv, Dh,
                   page_size, B, Dv, gate, **forms)
    a.q_pos0 = q_pos0.data_ptr() if q_pos0 is not None else None
    a.lse_out = lse_out.data_ptr() if lse_out is not None else None
    native.check(_lib().tsb_attn_prefill(C.byref(a), C.c_int(max_q_len), _stream()), "attn_prefill")
    _count(1)
    return out


def attn_f32(q, k_cache, v_cache, block_table, kv_lens, cu_q, *, scale, Hq, Hkv, Dh, page_size, Dv=None, sinks=None, softcap=0.0,
             window=0, gate=None, **forms):
    """Attention in 32 bits over a float32 cache, prompts and decode alike: q [T, Hq, Dh] -> [T, Hq, Dv]."""
    assert q.dtype == k_cache.dtype == v_cache.dtype == torch.float32 and (gate is None or gate.dtype == torch.float32)
    out = torch.empty((q.shape[0], Hq, Dv or Dh), dtype=torch.float32, device=q.device)
    a = _attn_args(q, k_cache, v_cache, out, block_table, kv_lens, cu_q, sinks, scale, softcap, window, Hq, Hkv, Dh, page_size,
                   kv_lens.shape[0], Dv, gate, **forms)
    native.check(_lib().tsb_attn_f32(C.byref(a), C.c_int(q.shape[0]), _stream()), "attn_f32")
    _count(1)
    return out


class SandwichArgs(C.Structure):
    _fields_ = [("h", _vp), ("y", _vp), ("pos", _vp), ("wts", _vp), ("post_w", _vp), ("post_b", _vp), ("add", _vp), ("pre_w", _vp),
                ("pre_b", _vp), ("out", _vp), ("rows", C.c_long), ("D", C.c_int), ("n", C.c_int), ("parts", C.c_int),
                ("y_f32", C.c_int), ("out_f32", C.c_int), ("eps", C.c_float)]


def residual_layernorm(h: torch.Tensor, eps: float, n: int, *, y=None, pos=None, wts=None, parts: int = 1, post=None, add=None, pre=None,
                       out_dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """h (f32 [T, D], in place) += layernorm(sum of y's parts; post) (+ add); returns layernorm(h; pre) or None."""
    assert h.dtype == torch.float32 and h.is_contiguous()
    T, D = h.shape
    a = SandwichArgs()
    a.h, a.rows, a.D, a.n, a.parts, a.eps = _p(h), T, D, n, parts, eps
    if y is not None:
        assert y.is_contiguous() and y.shape[-1] == D and y.dtype in (torch.float32, torch.bfloat16)
        assert (y.shape[0] == T * parts or pos is not None) and (pos is None or (pos.dtype == torch.int32 and pos.numel() == T * parts))
        assert wts is None or (wts.dtype == torch.float32 and wts.is_contiguous() and wts.numel() == T * parts)
        check_index("residual_layernorm", "part row", pos, y.shape[0], low=-1)
        a.y, a.pos, a.wts, a.y_f32 = _p(y), _p(pos), _p(wts), int(y.dtype == torch.float32)
        a.post_w, a.post_b = _p(post[0]), _p(post[1])
    a.add = _p(add)
    out = None
    if pre is not None:
        out = torch.empty((T, D), dtype=out_dtype, device=h.device)
        a.pre_w, a.pre_b, a.out, a.out_f32 = _p(pre[0]), _p(pre[1]), _p(out), int(out_dtype == torch.float32)
    native.check(_lib().tsb_sandwich_norm(C.byref(a), _stream()), "residual_layernorm")
    _count(1)
    return out


class ParallelNormArgs(C.Structure):
    _fields_ = [("h", _vp), ("h_out", _vp), ("y1", _vp), ("y2", _vp), ("s1", _vp), ("s2", _vp), ("w1", _vp), ("w2", _vp),
                ("out1", _vp), ("out2", _vp), ("shift", _vp), ("state", _vp), ("cu_q", _vp), ("seq_slots", _vp),
                ("rows", C.c_long), ("ld1", C.c_long), ("ld2", C.c_long), ("state_s", C.c_long),
                ("D", C.c_int), ("n", C.c_int), ("B", C.c_int), ("y_f32", C.c_int), ("out1_f32", C.c_int), ("out2_f32", C.c_int),
                ("span", C.c_int), ("eps", C.c_float)]


def parallel_norm(h, eps: float, n: int, *, y=(None, None), scale=(None, None), w=(None, None), out=(None, None), shift=None, state=None,
                  cu_q=None, seq_slots=None) -> torch.Tensor:
    """The seam of csrc/parallel_norm.cu: returns the new residual (``h`` itself when there is nothing to add) and fills the
    ``out`` tensors (rows may be strided)."""
    assert h.dtype == torch.float32 and h.is_contiguous()
    T, D = h.shape
    a = ParallelNormArgs()
    a.h, a.rows, a.D, a.n, a.eps = _p(h), T, D, n, eps
    res = h
    if y[0] is not None:
        res = torch.empty_like(h)
        a.h_out, a.y_f32 = _p(res), int(y[0].dtype == torch.float32)
        for t in y:
            assert t is None or (t.shape == h.shape and t.is_contiguous() and t.dtype == y[0].dtype and t.dtype in (torch.float32, torch.bfloat16))
        a.y1, a.y2, a.s1, a.s2 = _p(y[0]), _p(y[1]), _p(scale[0]), _p(scale[1])
    a.w1, a.w2 = _p(w[0]), _p(w[1])
    for i, o in enumerate(out, 1):
        if o is not None:
            assert o.shape == h.shape and o.stride(1) == 1 and o.dtype in (torch.float32, torch.bfloat16)
            setattr(a, f"out{i}", _p(o))
            setattr(a, f"ld{i}", o.stride(0))
            setattr(a, f"out{i}_f32", int(o.dtype == torch.float32))
    if shift is not None:
        check_index("parallel_norm", "state slot", seq_slots, state.shape[0])
        check_index("parallel_norm", "row offset", cu_q, T + 1)
        assert state.dtype == torch.float32 and state.stride(1) == 1 and seq_slots.dtype == torch.int64 and cu_q.dtype == torch.int32
        a.shift, a.state, a.state_s, a.cu_q, a.seq_slots, a.B = _p(shift), _p(state), state.stride(0), _p(cu_q), _p(seq_slots), cu_q.numel() - 1
    native.check(_lib().tsb_parallel_norm(C.byref(a), _stream()), "parallel_norm")
    _count(1)
    return res


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """cap tanh(x / cap) (f32)."""
    assert x.dtype == torch.float32 and x.is_contiguous()
    out = torch.empty_like(x)
    native.check(_lib().tsb_softcap(_p(x), _p(out), C.c_long(x.numel()), C.c_float(cap), _stream()), "softcap")
    _count(1)
    return out


class PostNormArgs(C.Structure):
    _fields_ = [("h", _vp), ("y", _vp), ("z", _vp), ("ids", _vp), ("pos", _vp), ("wts", _vp), ("b1", _vp), ("b2", _vp), ("post", _vp),
                ("pre", _vp), ("out", _vp), ("rows", C.c_long), ("D", C.c_int), ("n", C.c_int), ("parts", C.c_int), ("y_f32", C.c_int),
                ("out_f32", C.c_int), ("eps", C.c_float), ("mix", C.c_float)]


def post_norm(h: torch.Tensor, eps: float, n: int, *, y=None, z=None, ids=None, pos=None, wts=None, parts: int = 1, branch=(None, None),
              mix: float = 1.0, post=None, pre=None, out_dtype=torch.bfloat16) -> torch.Tensor:
    """The seam of csrc/post_norm.cu: h (f32 [T, D], in place) gains the norm of the sublayer's output; returns h, or its norm
    with the weight ``pre``, in ``out_dtype``."""
    assert h.dtype == torch.float32 and h.is_contiguous()
    T, D = h.shape
    a = PostNormArgs()
    a.h, a.rows, a.D, a.n, a.parts, a.eps, a.mix = _p(h), T, D, n, parts, eps, mix
    if y is not None:
        assert y.is_contiguous() and y.shape[-1] == D and y.dtype in (torch.float32, torch.bfloat16)
        assert (y.shape[0] == T * parts or pos is not None) and (pos is None or (pos.dtype == torch.int32 and pos.numel() == T * parts))
        assert z is None or (z.shape == y.shape == h.shape and z.dtype == y.dtype and z.is_contiguous())
        assert wts is None or (wts.dtype == torch.float32 and wts.is_contiguous() and wts.numel() == T * parts)
        assert ids is None or (ids.dtype == torch.int32 and ids.is_contiguous() and ids.numel() == T * parts)
        check_index("post_norm", "part row", pos, y.shape[0], low=-1)
        a.y, a.z, a.ids, a.pos, a.wts, a.y_f32 = _p(y), _p(z), _p(ids), _p(pos), _p(wts), int(y.dtype == torch.float32)
        a.b1, a.b2, a.post = _p(branch[0]), _p(branch[1]), _p(post)
    out = torch.empty((T, D), dtype=out_dtype, device=h.device)
    a.pre, a.out, a.out_f32 = _p(pre), _p(out), int(out_dtype == torch.float32)
    native.check(_lib().tsb_post_norm(C.byref(a), _stream()), "post_norm")
    _count(1)
    return out


def pair_embed(tok: QuantWeight, pair: QuantWeight, ids, cu_q, seq_slots, prev, *, mul_prev: int, mul_cur: int, out_dtype):
    """Token rows plus bigram rows: (f32 [T, D], the same in ``out_dtype``); ``prev`` int32 per slot is read and advanced."""
    T, D, dev = ids.numel(), tok.K, ids.device
    check_index("pair_embed", "state slot", seq_slots, prev.shape[0])
    check_index("pair_embed", "row offset", cu_q, T + 1)
    check_index("pair_embed", "token", ids, tok.rows)
    assert ids.dtype == cu_q.dtype == prev.dtype == torch.int32 and seq_slots.dtype == torch.int64 and prev.is_contiguous()
    assert tok.ggml_type == pair.ggml_type and pair.K == D
    h, out = torch.empty((T, D), dtype=torch.float32, device=dev), torch.empty((T, D), dtype=out_dtype, device=dev)
    native.check(_lib().tsb_pair_embed(_p(tok.planes[0]), _p(pair.planes[0]), C.c_int(int(tok.ggml_type)), C.c_int(tok.rows), C.c_int(D), _p(ids),
                                       _p(cu_q), _p(seq_slots), _p(prev), _p(h), _p(out), C.c_int(out_dtype == torch.float32), C.c_int(T),
                                       C.c_int(cu_q.numel() - 1), C.c_long(pair.rows - 1), C.c_long(mul_prev), C.c_long(mul_cur), _stream()), "pair_embed")
    _count(1)
    return h, out


class JointNormArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("w", _vp), ("slot", _vp), ("q", _vp), ("cache", _vp), ("ld", C.c_long),
                ("T", C.c_int), ("nq", C.c_int), ("nk", C.c_int), ("q_n", C.c_int), ("k_n", C.c_int), ("out_f32", C.c_int), ("eps", C.c_float)]


def joint_norm(y: torch.Tensor, w: torch.Tensor, cache: torch.Tensor, slots: torch.Tensor, *, nq: int, nk: int, q_n: int, k_n: int, eps: float) -> torch.Tensor:
    """Rows [q (nq) | k (nk)]: q over its root mean square times ``w`` -> [T, nq]; k and 1 / its root mean square to the cache rows."""
    T = y.shape[0]
    check_index("joint_norm", "cache slot", slots, cache.shape[0])
    assert y.stride(1) == 1 and y.shape[1] >= nq + nk and cache.is_contiguous() and cache.shape[-1] == nk + 8 and w.numel() == nq
    a = JointNormArgs()
    q = torch.empty((T, nq), dtype=cache.dtype, device=y.device)
    a.y, a.y_s, a.y_f32, a.w, a.slot, a.q, a.cache, a.ld = _p(y), y.stride(0), int(y.dtype == torch.float32), _p(w), _p(slots), _p(q), _p(cache), nk + 8
    a.T, a.nq, a.nk, a.q_n, a.k_n, a.out_f32, a.eps = T, nq, nk, q_n, k_n, int(cache.dtype == torch.float32), eps
    native.check(_lib().tsb_joint_norm(C.byref(a), _stream()), "joint_norm")
    _count(1)
    return q


class GlaArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("q", C.c_long), ("k", C.c_long), ("v", C.c_long), ("g", C.c_long), ("t", C.c_long),
                ("z", _vp), ("z_s", C.c_long), ("w2", _vp), ("w2_f32", C.c_int), ("zb", _vp), ("norm_w", _vp), ("state", _vp), ("state_s", C.c_long),
                ("cu_q", _vp), ("seq_slots", _vp), ("seg", _vp), ("seg_w", _vp), ("core", _vp), ("out", _vp), ("out_s", C.c_long),
                ("out_f32", C.c_int), ("T", C.c_int), ("B", C.c_int), ("H", C.c_int), ("D", C.c_int), ("E", C.c_int), ("e_n", C.c_int),
                ("rank", C.c_int), ("segs", C.c_int), ("seg_len", C.c_int), ("eps", C.c_float), ("q_scale", C.c_float), ("inv_tau", C.c_float)]


def _gla_args(y, s, cols, zb, norm_w, state, cu_q, seq_slots, eps: float, out_dtype):
    T = y.shape[0]
    check_index("gated_linear", "state slot", seq_slots, state.shape[0])
    check_index("gated_linear", "row offset", cu_q, T + 1)
    assert y.stride(1) == 1 and state.dtype == torch.float32 and state.shape[1:] == (s.H, s.E, s.D) and seq_slots.dtype == torch.int64
    assert state.stride(1) == s.E * s.D and state.stride(2) == s.D and state.stride(3) == 1
    a = GlaArgs()
    a.y, a.y_s, a.y_f32 = _p(y), y.stride(0), int(y.dtype == torch.float32)
    a.q, a.k, a.v, a.g, a.t = cols
    a.zb, a.norm_w, a.state, a.state_s, a.cu_q, a.seq_slots = _p(zb), _p(norm_w), _p(state), state.stride(0), _p(cu_q), _p(seq_slots)
    out = torch.empty((T, s.H * s.E), dtype=out_dtype, device=y.device)
    a.out, a.out_s, a.out_f32 = _p(out), s.H * s.E, int(out_dtype == torch.float32)
    a.T, a.B, a.H, a.D, a.E, a.e_n, a.eps, a.q_scale, a.inv_tau = T, cu_q.numel() - 1, s.H, s.D, s.E, s.vdim, eps, s.q_scale, 1.0 / s.tau
    return a, out


def gla_step(y, s, cols, w2: torch.Tensor, zb, norm_w, state, cu_q, seq_slots, *, eps: float, out_dtype) -> torch.Tensor:
    """Gated linear attention token by token (csrc/gated_linear.cu), decay map, norm and gate included."""
    a, out = _gla_args(y, s, cols, zb, norm_w, state, cu_q, seq_slots, eps, out_dtype)
    assert w2.is_contiguous() and w2.shape[0] == s.H * s.D and y.shape[1] >= cols[4] + w2.shape[1]
    a.w2, a.w2_f32, a.rank = _p(w2), int(w2.dtype == torch.float32), w2.shape[1]
    native.check(_lib().tsb_gla_step(C.byref(a), _stream()), "gla_step")
    _count(1)
    return out


def gla_prompt(y, s, cols, z: torch.Tensor, zb, norm_w, state, cu_q, seq_slots, *, eps: float, max_q: int, segs: int) -> torch.Tensor:
    """The same for prompts of bf16 models, 16 tokens at a time on the tensor cores, in ``segs`` segments per sequence (the
    longest has ``max_q`` tokens); ``z`` f32 [T, H * D]: the decay's projection."""
    assert y.dtype == torch.bfloat16 and z.dtype == torch.float32 and z.shape == (y.shape[0], s.H * s.D) and z.stride(1) == 1
    a, out = _gla_args(y, s, cols, zb, norm_w, state, cu_q, seq_slots, eps, torch.bfloat16)
    seg_len = (-(-max_q // segs) + 15) // 16 * 16
    segs = -(-max_q // seg_len)
    f32 = dict(dtype=torch.float32, device=y.device)
    if segs > 1:
        seg, seg_w = torch.empty((a.B, segs, s.H, s.E, s.D), **f32), torch.empty((a.B, segs, s.H, s.D), **f32)
        a.seg, a.seg_w = _p(seg), _p(seg_w)
    core = torch.empty((y.shape[0], s.H, s.E), **f32) if s.E > 128 else None
    a.z, a.z_s, a.core, a.segs, a.seg_len = _p(z), z.stride(0), _p(core), segs, seg_len
    native.check(_lib().tsb_gla_prompt(C.byref(a), C.c_int(max_q), _stream()), "gla_prompt")
    _count(1 + 2 * (segs > 1) + (core is not None))
    return out


SEAM_FUSED_ROWS = 64          # rows up to which the seam and its convolution are one kernel


class ConvSeamArgs(C.Structure):
    _fields_ = [("h", _vp), ("h_out", _vp), ("y", _vp), ("p", _vp), ("pos", _vp), ("wts", _vp), ("w", _vp), ("taps", _vp), ("state", _vp),
                ("cu_q", _vp), ("seq_slots", _vp), ("out", _vp), ("conv", _vp), ("rs", _vp), ("rows", C.c_long), ("state_s", C.c_long),
                ("D", C.c_int), ("n", C.c_int), ("B", C.c_int), ("K", C.c_int), ("parts", C.c_int), ("y_f32", C.c_int), ("p_f32", C.c_int),
                ("out_f32", C.c_int), ("span", C.c_int), ("eps", C.c_float)]


def _carried(what: str, state: torch.Tensor, rest: tuple, cu_q, seq_slots, T: int) -> int:
    """Checks a per-slot f32 state of rows ``rest`` (a view whose slots are strided, dense inside) and returns the slot stride."""
    check_index(what, "state slot", seq_slots, state.shape[0])
    check_index(what, "row offset", cu_q, T + 1)
    assert state.dtype == torch.float32 and tuple(state.shape[1:]) == tuple(rest) and seq_slots.dtype == torch.int64 and cu_q.dtype == torch.int32
    want = 1
    for d in range(state.dim() - 1, 0, -1):
        assert state.shape[d] <= 1 or state.stride(d) == want
        want *= state.shape[d]
    return state.stride(0) if state.shape[0] > 1 else 0          # (torch may give a dimension of one slot any stride)


def conv_seam(h: torch.Tensor, eps: float, n: int, *, w, y=None, parts=None, taps=None, state=None, batch=None, plain: bool = True,
              out_dtype=torch.bfloat16):
    """The seam of csrc/conv_seam.cu: (new residual, ``h`` itself when there is nothing to add; norm or None; norm plus its
    convolution over time, or None)."""
    assert h.dtype == torch.float32 and h.is_contiguous() and w.numel() == h.shape[1]
    T, D = h.shape
    a = ConvSeamArgs()
    a.h, a.w, a.rows, a.D, a.n, a.eps, a.out_f32 = _p(h), _p(w), T, D, n, eps, int(out_dtype == torch.float32)
    res = h
    if y is not None or parts is not None:
        res = torch.empty_like(h)
        a.h_out = _p(res)
    if y is not None:
        assert y.shape == h.shape and y.is_contiguous() and y.dtype in (torch.float32, torch.bfloat16)
        a.y, a.y_f32 = _p(y), int(y.dtype == torch.float32)
    if parts is not None:
        k, p = parts.k, parts.y
        assert p.is_contiguous() and p.shape[1] == D and p.dtype in (torch.float32, torch.bfloat16) and parts.ids is None
        assert (p.shape[0] == T * k or parts.pos is not None) and (parts.pos is None or (parts.pos.dtype == torch.int32 and parts.pos.numel() == T * k))
        assert parts.w is None or (parts.w.dtype == torch.float32 and parts.w.is_contiguous() and parts.w.numel() == T * k)
        check_index("conv_seam", "part row", parts.pos, p.shape[0], low=-1)
        a.p, a.p_f32, a.pos, a.wts, a.parts = _p(p), int(p.dtype == torch.float32), _p(parts.pos), _p(parts.w), k
    out = conv = None
    if plain:
        out = torch.empty((T, D), dtype=out_dtype, device=h.device)
        a.out = _p(out)
    if taps is not None:
        conv = torch.empty((T, D), dtype=out_dtype, device=h.device)
        K = taps.shape[0]
        assert taps.dtype == torch.float32 and taps.is_contiguous() and taps.shape[1] == D
        a.state_s = _carried("conv_seam", state, (K - 1, D), batch.cu_q, batch.seq_slots, T)
        a.conv, a.taps, a.K, a.state, a.cu_q, a.seq_slots, a.B = _p(conv), _p(taps), K, _p(state), _p(batch.cu_q), _p(batch.seq_slots), batch.B
        if T > SEAM_FUSED_ROWS:
            rs = torch.empty(T, dtype=torch.float32, device=h.device)
            a.rs = _p(rs)
    native.check(_lib().tsb_conv_seam(C.byref(a), _stream()), "conv_seam")
    _count(2 if a.rs else 1)
    return res, out, conv


class ShortConvArgs(C.Structure):
    _fields_ = [("x", _vp), ("x_s", C.c_long), ("x_f32", C.c_int), ("w", _vp), ("bias", _vp), ("state", _vp), ("state_s", C.c_long),
                ("cu_q", _vp), ("seq_slots", _vp), ("out", _vp), ("out_s", C.c_long), ("out_f32", C.c_int), ("block", C.c_int),
                ("pos", _vp), ("slot", _vp), ("k_cache", _vp), ("v_cache", _vp), ("nq", C.c_int), ("nk", C.c_int), ("qt_coef", C.c_float),
                ("qt_every", C.c_float), ("T", C.c_int), ("C", C.c_int), ("K", C.c_int), ("B", C.c_int), ("span", C.c_int)]


def _short_conv_args(x, w, bias, state, batch) -> ShortConvArgs:
    T, Cc = x.shape
    K = w.shape[0]
    assert x.stride(1) == 1 and x.dtype in (torch.float32, torch.bfloat16) and w.dtype == torch.float32 and w.is_contiguous() and w.shape[1] == Cc
    assert x.data_ptr() % (16 if x.dtype == torch.float32 else 8) == 0
    a = ShortConvArgs()
    a.state_s = _carried("short_conv", state, (K - 1, Cc), batch.cu_q, batch.seq_slots, T)
    a.x, a.x_s, a.x_f32, a.w, a.bias, a.state = _p(x), x.stride(0), int(x.dtype == torch.float32), _p(w), _p(bias), _p(state)
    a.cu_q, a.seq_slots, a.T, a.C, a.K, a.B = _p(batch.cu_q), _p(batch.seq_slots), T, Cc, K, batch.B
    return a


def short_conv(x, w, bias, state, batch, *, block: int = 0, out_dtype=torch.float32) -> torch.Tensor:
    """Causal convolution per channel (csrc/short_conv.cu) -> [T, C], or [C / block * T, block]."""
    T, Cc = x.shape
    a = _short_conv_args(x, w, bias, state, batch)
    out = torch.empty((Cc // block * T, block) if block else (T, Cc), dtype=out_dtype, device=x.device)
    a.out, a.out_s, a.out_f32, a.block = _p(out), Cc, int(out_dtype == torch.float32), block
    native.check(_lib().tsb_short_conv(C.byref(a), _stream()), "short_conv")
    _count(1)
    return out


def conv_qkv(y, w, state, batch, *, nq: int, dtype, k_cache=None, v_cache=None, q_temp=None) -> torch.Tensor:
    """The same on projection rows [q | k | v] of attention: keys and values to their cache slots, returns the queries [T, nq]."""
    T, Cc = y.shape
    a = _short_conv_args(y, w, None, state, batch)
    if k_cache is not None:
        check_index("short_conv", "cache slot", batch.slots, k_cache.shape[0])
        a.nk = k_cache.shape[1] * k_cache.shape[2]
        assert k_cache.dtype == dtype and k_cache.is_contiguous() and v_cache.is_contiguous() and v_cache.dtype == dtype and nq + a.nk + v_cache.shape[1] * v_cache.shape[2] == Cc
        a.k_cache, a.v_cache = _p(k_cache), _p(v_cache)
    else:
        assert nq == Cc
    q = torch.empty((y.shape[0], nq), dtype=dtype, device=y.device)
    assert dtype in (torch.float32, torch.bfloat16) and batch.positions.dtype == torch.int32 and batch.slots.dtype == torch.int64
    a.out, a.out_s, a.out_f32, a.nq, a.pos, a.slot = _p(q), nq, int(dtype == torch.float32), nq, _p(batch.positions), _p(batch.slots)
    a.qt_coef, a.qt_every = q_temp or (0.0, 0.0)
    native.check(_lib().tsb_short_conv(C.byref(a), _stream()), "short_conv")
    _count(1)
    return q


class RglruArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("u", _vp), ("u_f32", C.c_int), ("w", _vp), ("w_f32", C.c_int), ("z", _vp),
                ("gate_b", _vp), ("rate", _vp), ("state", _vp), ("state_s", C.c_long), ("cu_q", _vp), ("seq_slots", _vp), ("seg_a", _vp),
                ("seg_s", _vp), ("out", _vp), ("out_f32", C.c_int), ("T", C.c_int), ("B", C.c_int), ("W", C.c_int), ("block", C.c_int),
                ("segs", C.c_int), ("seg_len", C.c_int)]


def _rglru_args(y, u, s, gate_b, rate, state, batch, out_dtype):
    T = y.shape[0]
    assert y.stride(1) == 1 and y.shape[1] >= s.W and u.is_contiguous() and u.numel() == T * s.W and gate_b.shape == (2, s.W) and gate_b.is_contiguous()
    a = RglruArgs()
    a.state_s = _carried("rglru", state, (s.W,), batch.cu_q, batch.seq_slots, T)
    a.y, a.y_s, a.y_f32, a.u, a.u_f32 = _p(y), y.stride(0), int(y.dtype == torch.float32), _p(u), int(u.dtype == torch.float32)
    a.gate_b, a.rate, a.state, a.cu_q, a.seq_slots = _p(gate_b), _p(rate), _p(state), _p(batch.cu_q), _p(batch.seq_slots)
    out = torch.empty((T, s.W), dtype=out_dtype, device=y.device)
    a.out, a.out_f32, a.T, a.B, a.W, a.block = _p(out), int(out_dtype == torch.float32), T, batch.B, s.W, s.block
    return a, out


def rglru_step(y, u, s, w: torch.Tensor, gate_b, rate, state, batch, *, out_dtype) -> torch.Tensor:
    """Real-gated linear recurrent units token by token (csrc/rglru.cu), gates and output branch included; ``u`` f32 [T, W]."""
    a, out = _rglru_args(y, u, s, gate_b, rate, state, batch, out_dtype)
    assert u.dtype == torch.float32 and w.is_contiguous() and w.numel() == 2 * s.W * s.block
    a.w, a.w_f32 = _p(w), int(w.dtype == torch.float32)
    native.check(_lib().tsb_rglru_step(C.byref(a), _stream()), "rglru_step")
    _count(1)
    return out


def rglru_scan(y, u, z, s, gate_b, rate, state, batch, *, out_dtype, segs: int) -> torch.Tensor:
    """The same for prompts, from the gates' products ``z`` f32 [blocks * T, 2 block], in ``segs`` segments per sequence."""
    a, out = _rglru_args(y, u, s, gate_b, rate, state, batch, out_dtype)
    assert z.dtype == torch.float32 and z.is_contiguous() and z.shape == (s.blocks * y.shape[0], 2 * s.block)
    max_q = batch.max_q_len
    a.seg_len = -(-max_q // segs)
    a.segs = -(-max_q // a.seg_len)
    a.z = _p(z)
    if a.segs > 1:
        seg = torch.empty((2, a.B, a.segs, s.W), dtype=torch.float32, device=y.device)
        a.seg_a, a.seg_s = _p(seg[0]), _p(seg[1])
    native.check(_lib().tsb_rglru_scan(C.byref(a), C.c_int(max_q), _stream()), "rglru_scan")
    _count(1 + (a.segs > 1))
    return out


class MlstmArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("q", C.c_long), ("k", C.c_long), ("v", C.c_long), ("g", C.c_long),
                ("z", _vp), ("z_s", C.c_long), ("zb", _vp), ("norm_w", _vp), ("S", _vp), ("n", _vp), ("m", _vp), ("state_s", C.c_long),
                ("cu_q", _vp), ("seq_slots", _vp), ("fim", _vp), ("m0", _vp), ("seg", _vp), ("seg_n", _vp), ("seg_w", _vp), ("core", _vp),
                ("out", _vp), ("out_s", C.c_long), ("out_f32", C.c_int), ("T", C.c_int), ("B", C.c_int), ("H", C.c_int), ("D", C.c_int),
                ("E", C.c_int), ("e_n", C.c_int), ("segs", C.c_int), ("seg_len", C.c_int), ("eps", C.c_float), ("q_scale", C.c_float),
                ("cap", C.c_float)]


def _mlstm_args(y, s, cols, z, zb, norm_w, S, n, m, batch, eps: float, out_dtype):
    T = y.shape[0]
    assert y.stride(1) == 1 and z.dtype == torch.float32 and z.shape == (T, 2 * s.H) and z.stride(1) == 1 and zb.numel() == 2 * s.H
    assert norm_w.numel() == s.H * s.E
    a = MlstmArgs()
    strides = {_carried("mlstm", t, rest, batch.cu_q, batch.seq_slots, T) for t, rest in ((S, (s.H, s.E, s.D)), (n, (s.H, s.D)), (m, (s.H,)))}
    assert len(strides) == 1                              # all three are parts of one row per slot
    a.state_s = strides.pop()
    a.y, a.y_s, a.y_f32 = _p(y), y.stride(0), int(y.dtype == torch.float32)
    a.q, a.k, a.v, a.g = cols
    a.z, a.z_s, a.zb, a.norm_w, a.S, a.n, a.m = _p(z), z.stride(0), _p(zb), _p(norm_w), _p(S), _p(n), _p(m)
    a.cu_q, a.seq_slots = _p(batch.cu_q), _p(batch.seq_slots)
    out = torch.empty((T, s.H * s.E), dtype=out_dtype, device=y.device)
    a.out, a.out_s, a.out_f32 = _p(out), s.H * s.E, int(out_dtype == torch.float32)
    a.T, a.B, a.H, a.D, a.E, a.e_n, a.eps, a.q_scale, a.cap = T, batch.B, s.H, s.D, s.E, s.vdim, eps, s.q_scale, s.cap
    return a, out


def mlstm_step(y, s, cols, z, zb, norm_w, S, n, m, batch, *, eps: float, out_dtype) -> torch.Tensor:
    """mLSTM token by token (csrc/mlstm.cu), gates, norm and output gate included."""
    a, out = _mlstm_args(y, s, cols, z, zb, norm_w, S, n, m, batch, eps, out_dtype)
    native.check(_lib().tsb_mlstm_step(C.byref(a), _stream()), "mlstm_step")
    _count(1)
    return out


def mlstm_prompt(y, s, cols, z, zb, norm_w, S, n, m, batch, *, eps: float, out_dtype, segs: int) -> torch.Tensor:
    """The same for prompts of bf16 models, 64 tokens at a time on the tensor cores, in ``segs`` segments per sequence."""
    assert y.dtype == out_dtype == torch.bfloat16
    a, out = _mlstm_args(y, s, cols, z, zb, norm_w, S, n, m, batch, eps, out_dtype)
    max_q, T = batch.max_q_len, y.shape[0]
    a.seg_len = (-(-max_q // segs) + 63) // 64 * 64
    a.segs = segs = -(-max_q // a.seg_len)
    f32 = dict(dtype=torch.float32, device=y.device)
    fim, m0, seg_n = torch.empty((3, s.H, T), **f32), torch.empty((a.B, s.H), **f32), torch.empty((a.B, segs, s.H, s.D), **f32)
    seg = seg_w = None
    if segs > 1:
        seg, seg_w = torch.empty((a.B, segs, s.H, s.E, s.D), **f32), torch.empty((a.B, segs, s.H), **f32)
    core = torch.empty((T, s.H, s.E), **f32) if s.E > 128 else None
    a.fim, a.m0, a.seg_n, a.seg, a.seg_w, a.core = _p(fim), _p(m0), _p(seg_n), _p(seg), _p(seg_w), _p(core)
    native.check(_lib().tsb_mlstm_prompt(C.byref(a), C.c_int(max_q), _stream()), "mlstm_prompt")
    _count(2 + 2 * (segs > 1) + (core is not None))
    return out


class LatentArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("qn", _vp), ("kn", _vp), ("cs", _vp), ("slots", _vp), ("cache", _vp),
                ("cq", _vp), ("f32", C.c_int), ("T", C.c_int), ("qr", C.c_int), ("qp", C.c_int), ("R", C.c_int), ("rot", C.c_int),
                ("Lp", C.c_int), ("eps", C.c_float),
                ("q", _vp), ("q_f32", C.c_int), ("wuk", _vp), ("wuv", _vp), ("w_f32", C.c_int), ("qa", _vp),
                ("H", C.c_int), ("dim", C.c_int), ("Dk", C.c_int), ("Rp", C.c_int), ("Dv", C.c_int),
                ("block_table", _vp), ("kv_lens", _vp), ("part_o", _vp), ("part_ml", _vp), ("sinks", _vp), ("out", _vp),
                ("scale", C.c_float), ("window", C.c_int), ("page_size", C.c_int), ("max_pages", C.c_int), ("splits", C.c_int),
                ("Ro", C.c_int)]


def rotary_table(pos: torch.Tensor, freq: torch.Tensor, gain: float = 1.0) -> torch.Tensor:
    """(cos, sin) of pos * freq, times ``gain``: float32 [T, pairs, 2]; ``freq`` float64 on the device."""
    assert pos.dtype == torch.int32 and freq.dtype == torch.float64
    out = torch.empty((pos.numel(), freq.numel(), 2), dtype=torch.float32, device=pos.device)
    native.check(_lib().tsb_rotary_table(_p(pos), _p(freq), _p(out), C.c_int(pos.numel()), C.c_int(freq.numel()),
                                         C.c_float(gain), _stream()), "rotary_table")
    _count(1)
    return out


def _latent_args(s, T: int, cs: torch.Tensor, cache: torch.Tensor) -> LatentArgs:
    a = LatentArgs()
    a.T, a.qr, a.qp, a.R, a.rot, a.Lp, a.cs = T, s.q_rank, s.qp, s.rank, s.rot, s.row, _p(cs)
    a.H, a.dim, a.Dk, a.Rp, a.Dv, a.scale, a.window = s.heads, s.dim, s.Dk, s.rank_p, s.Dv, s.scale, s.window
    assert cache.shape[-1] == s.row and cache.is_contiguous() and cache.dtype in (torch.float32, torch.bfloat16)
    a.cache, a.f32 = _p(cache), int(cache.dtype == torch.float32)
    return a


def latent_prep(y: torch.Tensor, s, qn, kn, cs, cache, slots, eps: float) -> torch.Tensor:
    """Rows [query latent | key / value latent | rotated part] -> the normed query latent [T, qp]; the normed latent and the
    rotated key part go to the cache rows ``slots``."""
    T = y.shape[0]
    check_index("latent_prep", "cache slot", slots, cache.shape[0])
    assert y.stride(1) == 1 and y.shape[1] >= s.qp + s.rank + s.rot and slots.dtype == torch.int64
    a = _latent_args(s, T, cs, cache)
    cq = torch.empty((T, s.qp), dtype=cache.dtype, device=y.device)
    a.y, a.y_s, a.y_f32, a.qn, a.kn, a.slots, a.cq, a.eps = _p(y), y.stride(0), int(y.dtype == torch.float32), _p(qn), _p(kn), _p(slots), _p(cq), eps
    native.check(_lib().tsb_latent_prep(C.byref(a), _stream()), "latent_prep")
    _count(1)
    return cq


def latent_rotate(q: torch.Tensor, s, cs, cache) -> torch.Tensor:
    """Rotate the rotated parts of queries [T, H * Dk] in place."""
    a = _latent_args(s, q.shape[0], cs, cache)
    assert q.is_contiguous() and q.shape[1] == s.heads * s.Dk
    a.q, a.q_f32 = _p(q), int(q.dtype == torch.float32)
    native.check(_lib().tsb_latent_rotate(C.byref(a), _stream()), "latent_rotate")
    _count(1)
    return q


def latent_absorb(q: torch.Tensor, s, wuk: torch.Tensor, cs, cache) -> torch.Tensor:
    """Queries [T, H * Dk] (not rotated) in the space of the cached rows: [T, H, row]."""
    T = q.shape[0]
    a = _latent_args(s, T, cs, cache)
    assert q.is_contiguous() and q.shape[1] == s.heads * s.Dk and wuk.is_contiguous() and wuk.shape == (s.heads * s.dim, s.rank_p)
    qa = torch.empty((T, s.heads, s.row), dtype=cache.dtype, device=q.device)
    a.q, a.q_f32, a.wuk, a.w_f32, a.qa = _p(q), int(q.dtype == torch.float32), _p(wuk), int(wuk.dtype == torch.float32), _p(qa)
    native.check(_lib().tsb_latent_absorb(C.byref(a), _stream()), "latent_absorb")
    _count(1)
    return qa


def latent_decode_shape(B: int, heads: int, row: int):
    """(query heads per CTA, bytes of shared memory) of the latent decode kernel."""
    lib = _lib()
    lib.tsb_latent_decode_smem.restype = C.c_long
    n = (C.c_int(B), C.c_int(heads), C.c_int(row))
    return int(lib.tsb_latent_heads_per_cta(*n)), int(lib.tsb_latent_decode_smem(*n))


def latent_decode(qa: torch.Tensor, s, cs, cache, block_table, kv_lens, page_size: int, splits: int):
    """One query per sequence against the cached bf16 rows -> split partials (o [B, H, splits, Ro], (max, sum))."""
    B = qa.shape[0]
    check_index("latent_decode", "block-table page", block_table, cache.shape[0] // page_size)
    check_index("latent_decode", "cache length", kv_lens, block_table.shape[1] * page_size + 1)
    a = _latent_args(s, B, cs, cache)
    Ro = (s.rank + 7) // 8 * 8
    part_o = torch.empty((B, s.heads, splits, Ro), dtype=torch.float32, device=qa.device)
    part_ml = torch.empty((B, s.heads, splits, 2), dtype=torch.float32, device=qa.device)
    a.qa, a.block_table, a.kv_lens, a.part_o, a.part_ml = _p(qa), _p(block_table), _p(kv_lens), _p(part_o), _p(part_ml)
    a.page_size, a.max_pages, a.splits, a.Ro = page_size, block_table.shape[1], splits, Ro
    native.check(_lib().tsb_latent_decode(C.byref(a), _stream()), "latent_decode")
    _count(1)
    return part_o, part_ml


def latent_out(part_o: torch.Tensor, part_ml: Optional[torch.Tensor], s, wuv: torch.Tensor, sinks, cs, cache) -> torch.Tensor:
    """Merge split partials (``part_ml`` None: finished rows [T, H, rank]) and apply the value map -> [T, H * Dv]."""
    T = part_o.shape[0]
    a = _latent_args(s, T, cs, cache)
    assert wuv.is_contiguous() and wuv.shape == (s.heads * s.Dv, s.rank_p) and part_o.dtype == torch.float32 and part_o.is_contiguous()
    out = torch.empty((T, s.heads * s.Dv), dtype=cache.dtype, device=part_o.device)
    a.part_o, a.part_ml, a.wuv, a.w_f32, a.sinks, a.out = _p(part_o), _p(part_ml), _p(wuv), int(wuv.dtype == torch.float32), _p(sinks), _p(out)
    a.splits, a.Ro = part_o.shape[2] if part_ml is not None else 1, part_o.shape[-1]
    native.check(_lib().tsb_latent_out(C.byref(a), _stream()), "latent_out")
    _count(1)
    return out


class GdrArgs(C.Structure):
    _fields_ = [("y", _vp), ("y_s", C.c_long), ("y_f32", C.c_int), ("z", _vp), ("z_s", C.c_long), ("w2", _vp), ("w2_f32", C.c_int),
                ("w0", _vp), ("ab", _vp), ("norm_w", _vp), ("state", _vp), ("state_s", C.c_long), ("cu_q", _vp), ("seq_slots", _vp),
                ("pack", _vp), ("link", _vp), ("core", _vp), ("out", _vp), ("out_s", C.c_long), ("out_f32", C.c_int),
                ("T", C.c_int), ("B", C.c_int), ("H", C.c_int), ("D", C.c_int), ("n", C.c_int), ("rank", C.c_int), ("eps", C.c_float)]


def _gdr_args(y, w0, ab, norm_w, state, cu_q, seq_slots, *, H, D, n, rank, eps, out_dtype):
    T = y.shape[0]
    check_index("general_delta", "state slot", seq_slots, state.shape[0])
    check_index("general_delta", "row offset", cu_q, T + 1)
    assert y.stride(1) == 1 and y.shape[1] >= 5 * H * D + rank and state.dtype == torch.float32 and state.shape[1:] == (H, D, D)
    assert state.stride(1) == D * D and state.stride(2) == D and seq_slots.dtype == torch.int64
    a = GdrArgs()
    a.y, a.y_s, a.y_f32, a.w0, a.ab, a.norm_w = _p(y), y.stride(0), int(y.dtype == torch.float32), _p(w0), _p(ab), _p(norm_w)
    a.state, a.state_s, a.cu_q, a.seq_slots = _p(state), state.stride(0), _p(cu_q), _p(seq_slots)
    out = torch.empty((T, H * D), dtype=out_dtype, device=y.device)
    a.out, a.out_s, a.out_f32 = _p(out), H * D, int(out_dtype == torch.float32)
    a.T, a.B, a.H, a.D, a.n, a.rank, a.eps = T, cu_q.numel() - 1, H, D, n, rank, eps
    return a, out


def general_delta_short(y, w2: torch.Tensor, w0, ab, norm_w, state, cu_q, seq_slots, *, H, D, n, rank, eps, out_dtype) -> torch.Tensor:
    """Decode steps and short portions of the generalized delta rule (csrc/general_delta.cu), everything in one kernel."""
    assert w2.is_contiguous() and w2.shape == (H * D, rank)
    a, out = _gdr_args(y, w0, ab, norm_w, state, cu_q, seq_slots, H=H, D=D, n=n, rank=rank, eps=eps, out_dtype=out_dtype)
    a.w2, a.w2_f32 = _p(w2), int(w2.dtype == torch.float32)
    native.check(_lib().tsb_general_delta_short(C.byref(a), _stream()), "general_delta_short")
    _count(1)
    return out


def general_delta_prompt(y, z: torch.Tensor, w0, ab, norm_w, state, cu_q, seq_slots, *, H, D, n, eps, out_dtype, wide: bool = True) -> torch.Tensor:
    """Prompts: per-token vectors, recurrence, norm and gate in three kernels; ``z`` f32 [T, H * D] is the decay's projection.
    ``wide``: twice the value channels per warp."""
    T = y.shape[0]
    assert z.dtype == torch.float32 and z.shape == (T, H * D) and z.stride(1) == 1
    a, out = _gdr_args(y, w0, ab, norm_w, state, cu_q, seq_slots, H=H, D=D, n=n, rank=0, eps=eps, out_dtype=out_dtype)
    pack = torch.empty((T + 1, H, 5, D), dtype=torch.float32, device=y.device)
    core = torch.empty((T, H, D), dtype=torch.float32, device=y.device)
    link = torch.empty((T + 1, H, 4), dtype=torch.float32, device=y.device)
    a.z, a.z_s, a.pack, a.link, a.core = _p(z), z.stride(0), _p(pack), _p(link), _p(core)
    native.check(_lib().tsb_general_delta_prompt(C.byref(a), C.c_int(wide), _stream()), "general_delta_prompt")
    _count(3)
    return out


def general_delta_chunk(y, z: torch.Tensor, w0, ab, norm_w, state, cu_q, seq_slots, *, H, D, n, eps, max_q: int, out_dtype) -> torch.Tensor:
    """:func:`general_delta_prompt` in chunks of eight tokens on the tensor cores (csrc/general_delta_chunk.cu: split tf32
    operands, f32 accuracy); ``max_q``: the longest portion of the batch."""
    T = y.shape[0]
    assert z.dtype == torch.float32 and z.shape == (T, H * D) and z.stride(1) == 1
    a, out = _gdr_args(y, w0, ab, norm_w, state, cu_q, seq_slots, H=H, D=D, n=n, rank=0, eps=eps, out_dtype=out_dtype)
    lib = _lib()
    lib.tsb_general_delta_chunk_floats.restype = C.c_long
    pack = torch.empty((T // 8 + a.B + 1) * H * int(lib.tsb_general_delta_chunk_floats(C.c_int(D))), dtype=torch.float32, device=y.device)
    core = torch.empty((T, H, D), dtype=torch.float32, device=y.device)
    a.z, a.z_s, a.pack, a.core = _p(z), z.stride(0), _p(pack), _p(core)
    native.check(lib.tsb_general_delta_chunk(C.byref(a), C.c_int(max_q), _stream()), "general_delta_chunk")
    _count(3)
    return out


def tanh_rows(y: torch.Tensor, off: int, cols: int, ld: int, out_dtype) -> torch.Tensor:
    """tanh of ``cols`` columns of y from ``off`` on as dense rows [T, ld], zero past the columns."""
    assert y.stride(1) == 1 and off + cols <= y.shape[1]
    out = torch.empty((y.shape[0], ld), dtype=out_dtype, device=y.device)
    native.check(_lib().tsb_tanh_rows(_p(y), C.c_long(y.stride(0)), C.c_int(y.dtype == torch.float32), C.c_long(off), C.c_int(y.shape[0]),
                                      C.c_int(cols), C.c_int(ld), _p(out), C.c_int(out_dtype == torch.float32), _stream()), "tanh_rows")
    _count(1)
    return out


class GemmF32Args(C.Structure):
    _fields_ = [("W", _vp), ("X", _vp), ("out", _vp), ("bias", _vp), ("tiles", _vp), ("rows", _vp), ("ldx", C.c_long), ("ldo", C.c_long),
                ("T", C.c_int), ("N", C.c_int), ("K", C.c_int), ("row_div", C.c_int)]


def gemm_f32(w: QuantWeight, x: torch.Tensor, *, bias=None, tiles=None, rows=None, row_div: int = 1) -> torch.Tensor:
    """x [T, K] float32 @ w^T in 32-bit arithmetic (weights as stored, bf16 or f32).  With ``tiles`` (int32 [n, 3] on the
    device, pieces of at most 64 rows, see :func:`moe_sort`) ``w`` is a stack and row i of the result uses the matrix of its
    tile; ``rows`` int32: result row i reads x row rows[i] // row_div."""
    from ..gguf.constants import GGMLType
    assert x.dtype == torch.float32 and x.stride(1) == 1 and x.shape[1] == w.K and w.ggml_type in (GGMLType.BF16, GGMLType.F32)
    T = rows.numel() if rows is not None else x.shape[0]
    out = torch.empty((T, w.N), dtype=torch.float32, device=x.device)
    a = GemmF32Args()
    a.W, a.X, a.out, a.bias, a.tiles, a.rows = _p(w.planes[0]), _p(x), _p(out), _p(bias), _p(tiles), _p(rows)
    a.ldx, a.ldo, a.T, a.N, a.K, a.row_div = x.stride(0), w.N, T, w.N, w.K, row_div
    native.check(_lib().tsb_gemm_f32(C.byref(a), C.c_int(w.ggml_type == GGMLType.BF16), C.c_int(tiles.shape[0] if tiles is not None else 0),
                                     _stream()), "gemm_f32")
    _count(1)
    return out


def glu_f32(gate: torch.Tensor, up: Optional[torch.Tensor], act: str, clamp=None) -> torch.Tensor:
    """Gated activation of two float32 [T, F] views in 32 bits (``clamp`` as for :func:`glu`)."""
    lim, lim_first, rows_first = clamp or (7.0, 7.0, 0)
    T, F = gate.shape
    assert gate.dtype == torch.float32 and gate.stride(1) == 1 and (up is None or (up.dtype == torch.float32 and up.stride(1) == 1))
    out = torch.empty((T, F), dtype=torch.float32, device=gate.device)
    native.check(_lib().tsb_glu_f32(_p(gate), _p(up), C.c_long(gate.stride(0)), C.c_long(up.stride(0) if up is not None else 0), C.c_long(T),
                                    C.c_int(F), C.c_int(ACT[act]), _p(out), C.c_float(lim), C.c_float(lim_first), C.c_long(rows_first),
                                    _stream()), "glu_f32")
    _count(1)
    return out


_status_words = {}


def gemm_status(device) -> torch.Tensor:
    key = torch.device(device).index or 0
    if key not in _status_words:
        _status_words[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status_words[key]


_SPLITK_WS: dict = {}


def _splitk_workspace(device) -> Optional[torch.Tensor]:
    """Per-device float32 scratch (16 MB) for the partial tiles of split-K GEMMs; launches on one stream reuse it in order."""
    if os.environ.get("TSB_GEMM_SPLITK", "1") == "0":
        return None
    key = torch.device(device).index or 0
    ws = _SPLITK_WS.get(key)
    if ws is None:
        ws = _SPLITK_WS[key] = torch.empty(4 << 20, dtype=torch.float32, device=device)
    return ws


def gemm_bf16(W: torch.Tensor, X: torch.Tensor, *, out_dtype=torch.bfloat16, bias=None, residual=None,
              out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[T, N] = X[T, K] @ W[N, K]^T on tcgen05 tensor cores (bf16 in, f32 accumulate)."""
    assert W.dtype == torch.bfloat16 and X.dtype == torch.bfloat16
    assert W.stride(1) == 1 and X.stride(1) == 1
    N, K = W.shape
    T = X.shape[0]
    if out is None:
        out = torch.empty((T, N), dtype=out_dtype, device=X.device)
    ws = _splitk_workspace(X.device) if T <= 64 else None       # few tiles, long K: the library may split K over CTAs
    lib = _lib()
    lib.tsb_gemm_bf16_ws.restype = C.c_int
    native.check(lib.tsb_gemm_bf16_ws(_p(W), C.c_long(W.stride(0)), _p(X), C.c_long(X.stride(0)), _p(out),
                                      C.c_long(out.stride(0)), C.c_int(out.dtype == torch.float32), _p(bias),
                                      _p(residual), C.c_int(T), C.c_int(N), C.c_int(K), _p(gemm_status(X.device)),
                                      _stream(), _p(ws), C.c_long(ws.numel() * 4 if ws is not None else 0)), "gemm_bf16")
    _count(1)
    return out


def gemm_bf16_grouped(W: torch.Tensor, E: int, X: torch.Tensor, tiles: torch.Tensor, bn: int, *, out_dtype=torch.bfloat16,
                      bias=None, zero: bool = True) -> torch.Tensor:
    """Grouped GEMM over a stack of ``E`` matrices: W [E * N, K] bf16, X [P, K] bf16 with each group's rows contiguous,
    ``tiles`` int32 [n_tiles, 3] on the device = (matrix index or -1, first row, end row) with at most ``bn`` rows per
    tile -> out [P, N], zero where no tile covers a row (``zero=False``: every row is covered)."""
    assert W.dtype == torch.bfloat16 and X.dtype == torch.bfloat16 and W.stride(1) == 1 and X.stride(1) == 1
    assert tiles.dtype == torch.int32 and tiles.is_contiguous() and tiles.shape[1] == 3
    N, K = W.shape[0] // E, W.shape[1]
    P = X.shape[0]
    out = (torch.zeros if zero else torch.empty)((P, N), dtype=out_dtype, device=X.device)
    lib = _lib()
    lib.tsb_gemm_bf16_grouped.restype = C.c_int
    native.check(lib.tsb_gemm_bf16_grouped(_p(W), C.c_long(W.stride(0)), C.c_int(E), _p(X), C.c_long(X.stride(0)), _p(out),
                                           C.c_long(out.stride(0)), C.c_int(out.dtype == torch.float32), _p(bias), C.c_int(P),
                                           C.c_int(N), C.c_int(K), _p(tiles), C.c_int(tiles.shape[0]), C.c_int(bn),
                                           _p(gemm_status(X.device)), _stream()), "gemm_bf16_grouped")
    _count(1)
    return out


# --------------------------------------------------------------------------------------------
class ConvArgs(C.Structure):
    _fields_ = [("x", _vp), ("xs", C.c_long), ("x_f32", C.c_int), ("w", _vp), ("bias", _vp), ("state", _vp),
                ("cu_q", _vp), ("seq_slots", _vp), ("out", _vp), ("os", C.c_long),
                ("C", C.c_int), ("K", C.c_int), ("B", C.c_int), ("act", C.c_int)]


class GdnArgs(C.Structure):
    _fields_ = [("qkv", _vp), ("qkv_s", C.c_long), ("z", _vp), ("z_s", C.c_long), ("z_f32", C.c_int),
                ("beta", _vp), ("alpha", _vp), ("ba_s", C.c_long), ("ba_f32", C.c_int),
                ("dt_bias", _vp), ("a", _vp), ("norm_w", _vp), ("state", _vp), ("cu_q", _vp), ("seq_slots", _vp),
                ("out", _vp), ("out_s", C.c_long), ("eps", C.c_float),
                ("Hk", C.c_int), ("Hv", C.c_int), ("Dk", C.c_int), ("Dv", C.c_int), ("B", C.c_int)]


class GdnCarryArgs(C.Structure):
    _fields_ = [("U0", _vp), ("W", _vp), ("Qd", _vp), ("Kd", _vp), ("P", _vp), ("gamma", _vp), ("state", _vp), ("out", _vp),
                ("Hv", C.c_int), ("nc", C.c_int), ("Dk", C.c_int), ("Dv", C.c_int)]


class GdnPrepArgs(C.Structure):
    _fields_ = [("qkv", _vp), ("qkv_s", C.c_long), ("beta", _vp), ("alpha", _vp), ("ba_s", C.c_long), ("ba_f32", C.c_int),
                ("dt_bias", _vp), ("a_log", _vp), ("cu_q", _vp),
                ("U0", _vp), ("W", _vp), ("Qd", _vp), ("Kd", _vp), ("P", _vp), ("gamma", _vp),
                ("Hk", C.c_int), ("Hv", C.c_int), ("Dk", C.c_int), ("Dv", C.c_int), ("B", C.c_int), ("nc", C.c_int),
                ("eps", C.c_float)]


class GdnFinishArgs(C.Structure):
    _fields_ = [("core", _vp), ("z", _vp), ("z_s", C.c_long), ("z_f32", C.c_int), ("norm_w", _vp), ("cu_q", _vp),
                ("out", _vp), ("out_s", C.c_long), ("Hv", C.c_int), ("Dv", C.c_int), ("B", C.c_int), ("nc", C.c_int),
                ("eps", C.c_float)]


class MambaArgs(C.Structure):
    _fields_ = [("xbc", _vp), ("xbc_s", C.c_long), ("dt", _vp), ("dt_s", C.c_long), ("dt_f32", C.c_int),
                ("dt_bias", _vp), ("A", _vp), ("D", _vp), ("state", _vp), ("cu_q", _vp), ("seq_slots", _vp),
                ("y", _vp), ("y_s", C.c_long),
                ("H", C.c_int), ("P", C.c_int), ("G", C.c_int), ("N", C.c_int), ("B", C.c_int)]


def causal_conv1d(x, w, bias, state, cu_q, seq_slots, max_q, act_silu=True) -> torch.Tensor:
    """x [T, C] view (row stride allowed) -> f32 [T, C]; the per-slot tail ``state`` is updated."""
    T, Cc = x.shape
    check_index("causal_conv1d", "state slot", seq_slots, state.shape[0])
    out = torch.empty((T, Cc), dtype=torch.float32, device=x.device)
    a = ConvArgs()
    a.x, a.xs, a.x_f32 = _p(x), x.stride(0), int(x.dtype == torch.float32)
    a.w, a.bias, a.state = _p(w), _p(bias), _p(state)
    a.cu_q, a.seq_slots, a.out, a.os = _p(cu_q), _p(seq_slots), _p(out), Cc
    a.C, a.K, a.B, a.act = Cc, w.shape[1], cu_q.numel() - 1, 1 if act_silu else 0
    native.check(_lib().tsb_causal_conv1d(C.byref(a), C.c_int(max_q), _stream()), "causal_conv1d")
    _count(2)
    return out


def gdn_recurrent(qkv, z, beta, alpha, dt_bias, a_log, norm_w, state, cu_q, seq_slots, *, Hk, Hv, Dk, Dv, eps):
    T = qkv.shape[0]
    check_index("gdn_recurrent", "state slot", seq_slots, state.shape[0])
    check_index("gdn_recurrent", "row offset", cu_q, T + 1)
    out = torch.empty((T, Hv * Dv), dtype=torch.bfloat16, device=qkv.device)
    assert qkv.dtype == torch.float32 and beta.dtype == alpha.dtype and beta.stride(0) == alpha.stride(0)
    a = GdnArgs()
    a.qkv, a.qkv_s = _p(qkv), qkv.stride(0)
    a.z, a.z_s, a.z_f32 = _p(z), z.stride(0), int(z.dtype == torch.float32)
    a.beta, a.alpha, a.ba_s, a.ba_f32 = _p(beta), _p(alpha), beta.stride(0), int(beta.dtype == torch.float32)
    a.dt_bias, a.a, a.norm_w, a.state = _p(dt_bias), _p(a_log), _p(norm_w), _p(state)
    a.cu_q, a.seq_slots, a.out, a.out_s, a.eps = _p(cu_q), _p(seq_slots), _p(out), Hv * Dv, eps
    a.Hk, a.Hv, a.Dk, a.Dv, a.B = Hk, Hv, Dk, Dv, cu_q.numel() - 1
    native.check(_lib().tsb_gdn_recurrent(C.byref(a), _stream()), "gdn_recurrent")
    _count(1)
    return out


def gdn_chunk_carry_supported(Dk: int, Dv: int, chunk: int) -> bool:
    return chunk == 64 and Dk in (64, 128) and Dv % 32 == 0


def gdn_chunked_supported(Dk: int, Dv: int) -> bool:
    return Dk in (64, 128) and Dv % 32 == 0 and Dv <= 128


def gdn_chunked(qkv, z, beta, alpha, dt_bias, a_log, norm_w, state, cu_q, h_cu_q, slots, *, Hk, Hv, Dk, Dv, eps) -> torch.Tensor:
    """Chunked GatedDeltaNet prefill of a packed batch in three kernels (csrc/gdn_chunk.cu): the chunk-parallel algebra
    (normalisation, decay, Gram products, the triangular solve) per (sequence, head, chunk); the state carried chunk
    after chunk per (sequence, head, value slice); the gated output norm.  ``state`` [slots, Hv, Dv, Dk] f32 is updated
    for the sequences' slots (host list ``slots``); ``cu_q`` int32 [B + 1] on the device, ``h_cu_q`` its host copy.
    Returns bf16 [T, Hv * Dv]."""
    T = qkv.shape[0]
    B = len(h_cu_q) - 1
    nc = (max(h_cu_q[i + 1] - h_cu_q[i] for i in range(B)) + 63) // 64
    dev = qkv.device
    assert qkv.dtype == torch.float32 and qkv.stride(1) == 1 and beta.dtype == alpha.dtype and beta.stride(0) == alpha.stride(0)
    BH = B * Hv
    f32 = dict(dtype=torch.float32, device=dev)
    U0, W = torch.empty((BH, nc, 64, Dv), **f32), torch.empty((BH, nc, 64, Dk), **f32)
    Qd, Kd = torch.empty((BH, nc, 64, Dk), **f32), torch.empty((BH, nc, 64, Dk), **f32)
    P, gamma = torch.empty((BH, nc, 64, 64), **f32), torch.empty((BH, nc), **f32)
    a = GdnPrepArgs()
    a.qkv, a.qkv_s = _p(qkv), qkv.stride(0)
    a.beta, a.alpha, a.ba_s, a.ba_f32 = _p(beta), _p(alpha), beta.stride(0), int(beta.dtype == torch.float32)
    a.dt_bias, a.a_log, a.cu_q = _p(dt_bias), _p(a_log), _p(cu_q)
    a.U0, a.W, a.Qd, a.Kd, a.P, a.gamma = _p(U0), _p(W), _p(Qd), _p(Kd), _p(P), _p(gamma)
    a.Hk, a.Hv, a.Dk, a.Dv, a.B, a.nc, a.eps = Hk, Hv, Dk, Dv, B, nc, eps
    lib = _lib()
    native.check(lib.tsb_gdn_chunk_prep(C.byref(a), _stream()), "gdn_chunk_prep")
    _count(1)
    if B == 1:
        S = state[slots[0]]
    else:
        idx = torch.tensor(slots, dtype=torch.long, device=dev)
        S = state[idx].reshape(BH, Dv, Dk)
    core = gdn_chunk_carry(U0, W, Qd, Kd, P, gamma, S)
    if B > 1:
        state[idx] = S.view(B, Hv, Dv, Dk)
    out = torch.empty((T, Hv * Dv), dtype=torch.bfloat16, device=dev)
    f = GdnFinishArgs()
    f.core, f.z, f.z_s, f.z_f32 = _p(core), _p(z), z.stride(0), int(z.dtype == torch.float32)
    f.norm_w, f.cu_q, f.out, f.out_s = _p(norm_w), _p(cu_q), _p(out), Hv * Dv
    f.Hv, f.Dv, f.B, f.nc, f.eps = Hv, Dv, B, nc, eps
    native.check(lib.tsb_gdn_chunk_finish(C.byref(f), _stream()), "gdn_chunk_finish")
    _count(1)
    return out


class MambaPrepArgs(C.Structure):
    _fields_ = [("xbc", _vp), ("xbc_s", C.c_long), ("dt", _vp), ("dt_s", C.c_long), ("dt_f32", C.c_int),
                ("dt_bias", _vp), ("A", _vp), ("cu_q", _vp),
                ("U0", _vp), ("Qd", _vp), ("Kd", _vp), ("P", _vp), ("gamma", _vp),
                ("H", C.c_int), ("Pd", C.c_int), ("G", C.c_int), ("N", C.c_int), ("B", C.c_int), ("nc", C.c_int)]


def mamba2_chunked_supported(N: int, P: int) -> bool:
    return N in (64, 128) and P % 32 == 0


def mamba2_chunked(xbc, dt, dt_bias, A, D, state, cu_q, h_cu_q, slots, *, H, P, G, N) -> torch.Tensor:
    """Chunked Mamba2 prefill of a packed batch in two kernels (csrc/gdn_chunk.cu): the chunk-parallel algebra per
    (sequence, head, chunk) - step sizes, running decay, C B^T with its decay mask, decayed reads and writes - and the
    chunk-carry kernel of the delta rule with nothing to correct.  ``xbc`` f32 [T, H P + 2 G N] (after the convolution),
    ``state`` [slots, H, P, N] f32 updated for the sequences' slots.  Returns y f32 [T, H * P] (skip term included)."""
    T = xbc.shape[0]
    B = len(h_cu_q) - 1
    nc = (max(h_cu_q[i + 1] - h_cu_q[i] for i in range(B)) + 63) // 64
    dev = xbc.device
    assert xbc.dtype == torch.float32 and xbc.stride(1) == 1 and dt.stride(1) == 1 and state.dtype == torch.float32
    BH = B * H
    f32 = dict(dtype=torch.float32, device=dev)
    U0 = torch.empty((BH, nc, 64, P), **f32)
    Qd, Kd = torch.empty((BH, nc, 64, N), **f32), torch.empty((BH, nc, 64, N), **f32)
    Pm, gamma = torch.empty((BH, nc, 64, 64), **f32), torch.empty((BH, nc), **f32)
    a = MambaPrepArgs()
    a.xbc, a.xbc_s = _p(xbc), xbc.stride(0)
    a.dt, a.dt_s, a.dt_f32 = _p(dt), dt.stride(0), int(dt.dtype == torch.float32)
    a.dt_bias, a.A, a.cu_q = _p(dt_bias.float().contiguous() if dt_bias is not None else None), _p(A.float().contiguous()), _p(cu_q)
    a.U0, a.Qd, a.Kd, a.P, a.gamma = _p(U0), _p(Qd), _p(Kd), _p(Pm), _p(gamma)
    a.H, a.Pd, a.G, a.N, a.B, a.nc = H, P, G, N, B, nc
    lib = _lib()
    lib.tsb_mamba2_chunk_prep.restype = C.c_int
    native.check(lib.tsb_mamba2_chunk_prep(C.byref(a), _stream()), "mamba2_chunk_prep")
    _count(1)
    if B == 1:
        S = state[slots[0]]
    else:
        idx = torch.tensor(slots, dtype=torch.long, device=dev)
        S = state[idx].reshape(BH, P, N)
    core = gdn_chunk_carry(U0, None, Qd, Kd, Pm, gamma, S)           # [BH, nc, 64, P]; W = 0: nothing to correct
    if B > 1:
        state[idx] = S.view(B, H, P, N)
    y = torch.empty((T, H, P), **f32)
    for b in range(B):
        q0, n = h_cu_q[b], h_cu_q[b + 1] - h_cu_q[b]
        y[q0:q0 + n] = core[b * H:(b + 1) * H].reshape(H, nc * 64, P)[:, :n].transpose(0, 1)
    if D is not None:
        y = y + D.float().view(1, H, 1) * xbc[:, :H * P].view(T, H, P)
    return y.view(T, H * P)


def gdn_chunk_carry(U0, W, Qd, Kd, P, gamma, state) -> torch.Tensor:
    """The sequential part of the chunked GatedDeltaNet prefill for one sequence: ``state`` [Hv, Dv, Dk] f32 (contiguous,
    updated in place) carried through the chunks of U0 [Hv, nc, 64, Dv], W / Qd / Kd [Hv, nc, 64, Dk], P [Hv, nc, 64, 64],
    gamma [Hv, nc] -> outputs [Hv, nc, 64, Dv] f32.  ``W`` None stands for zeros (no correction term)."""
    U0, Qd, Kd, P, gamma = (t.float().contiguous() for t in (U0, Qd, Kd, P, gamma))
    W = W.float().contiguous() if W is not None else None              # None: nothing to correct (the Mamba2 form)
    Hv, nc, Cn, Dv = U0.shape
    Dk = Qd.shape[-1]
    assert Cn == 64 and state.dtype == torch.float32 and state.is_contiguous() and state.shape == (Hv, Dv, Dk)
    out = torch.empty((Hv, nc, Cn, Dv), dtype=torch.float32, device=U0.device)
    a = GdnCarryArgs()
    a.U0, a.W, a.Qd, a.Kd, a.P, a.gamma, a.state, a.out = _p(U0), _p(W), _p(Qd), _p(Kd), _p(P), _p(gamma), _p(state), _p(out)
    a.Hv, a.nc, a.Dk, a.Dv = Hv, nc, Dk, Dv
    native.check(_lib().tsb_gdn_chunk_carry(C.byref(a), _stream()), "gdn_chunk_carry")
    _count(1)
    return out


def mamba2_recurrent(xbc, dt, dt_bias, A, D, state, cu_q, seq_slots, *, H, P, G, N):
    T = xbc.shape[0]
    check_index("mamba2_recurrent", "state slot", seq_slots, state.shape[0])
    check_index("mamba2_recurrent", "row offset", cu_q, T + 1)
    y = torch.empty((T, H * P), dtype=torch.float32, device=xbc.device)
    a = MambaArgs()
    a.xbc, a.xbc_s = _p(xbc), xbc.stride(0)
    a.dt, a.dt_s, a.dt_f32 = _p(dt), dt.stride(0), int(dt.dtype == torch.float32)
    a.dt_bias, a.A, a.D, a.state = _p(dt_bias), _p(A), _p(D), _p(state)
    a.cu_q, a.seq_slots, a.y, a.y_s = _p(cu_q), _p(seq_slots), _p(y), H * P
    a.H, a.P, a.G, a.N, a.B = H, P, G, N, cu_q.numel() - 1
    native.check(_lib().tsb_mamba2_recurrent(C.byref(a), _stream()), "mamba2_recurrent")
    _count(1)
    return y
