"""Plain, slow implementation of the Sogulix decoder for the tests: one function per mechanism, whole sequences, no cache.

Nothing here is shared with the package: ``w`` is a dict name -> float tensor, ``cfg`` the dictionary of config.json.
Everything runs in the dtype of the weights it is given (float64 in most tests).
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, weight, eps):
    return rms(x, eps) * (1.0 + weight)


def token_shift(h, mix):
    """Row t moves towards row t - 1 by ``mix`` per channel; row 0 towards zero."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def rotate_half(x, positions, base):
    """All columns of x [T, ..., R] rotated, column i with column i + R / 2."""
    half = x.shape[-1] // 2
    freq = torch.tensor([base ** (-2.0 * i / (2 * half)) for i in range(half)], dtype=torch.float64)
    ang = positions.double()[:, None] * freq[None]
    ang = ang.view(len(positions), *([1] * (x.dim() - 2)), half)
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def windowed_attention(q, k, v, scale, window, sink):
    """q, k [T, H, D], v [T, H, E]; position i sees the ``window`` positions that end with i (None: all before); the
    softmax of head h has exp(sink[h]) in its denominator."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            s = (k[lo:i + 1, h] @ q[i, h]) * scale
            top = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            out[i, h] = (e / (e.sum() + torch.exp(sink[h] - top))) @ v[lo:i + 1, h]
    return out


def latent_attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, D, R, E, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + R)
    low = h @ w[p + "dkv"].T
    c = rms(low[:, :L], eps) * w[p + "dkv.norm"]
    kr = rotate_half(low[:, L:], pos, m["rot"]["base"])
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), kr[:, None].expand(T, H, R)], -1)
    q = torch.cat([q[..., :D], rotate_half(q[..., D:], pos, m["rot"]["base"])], -1)
    v = (c @ w[p + "uv"].T).view(T, H, E)
    window = m["mask"]["size"] if m.get("mask") else None
    o = windowed_attention(q, k, v, m["scale"], window, w[p + "sink"])
    return o.reshape(T, H * E) @ w[p + "o"].T


def delta_rule(r, k, v, decay, removal, state=None):
    """[T, H, D] each.  Per head, S [D keys, D values]:  S <- diag(decay) S - (removal u)(u^T S) + k v^T,  o = S^T r."""
    T, H, D = r.shape
    S = torch.zeros(H, D, D, dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros_like(r)
    for t in range(T):
        for h in range(H):
            u = k[t, h] / torch.sqrt((k[t, h] * k[t, h]).sum() + 1e-6)
            read = u @ S[h]
            S[h] = decay[t, h][:, None] * S[h] - torch.outer(removal[t, h] * u, read) + torch.outer(k[t, h], v[t, h])
            out[t, h] = r[t, h] @ S[h]
    return out, S


def general_delta_inputs(h, w, p, m):
    T, shape = h.shape[0], (h.shape[0], m["heads"], m["dim"])
    r, k, v = ((h @ w[p + n].T).view(shape) for n in "rkv")
    z = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * sigmoid(z)).view(shape)
    removal = sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).view(shape)
    return r, k, v, decay, removal


def general_delta_mixer(h, w, p, m, eps):
    o, _ = delta_rule(*general_delta_inputs(h, w, p, m))
    o = rms(o, eps).reshape(h.shape[0], -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def gated_ff(h, w, p):
    z = h @ w[p + "gate"].T
    return (z * sigmoid(z) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"latent_attention": latent_attention_mixer, "general_delta": general_delta_mixer}


def layer(x, w, i, cfg):
    p, eps, spec = f"l{i}.", cfg["norm"]["eps"], cfg["layers"][i]
    h = token_shift(zero_centred_norm(x, w[p + "norm1"], eps), w[p + "shift"])
    y = MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], eps) * w[p + "ls1"]
    if spec["mlp"] is not None:
        y = y + gated_ff(zero_centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.") * w[p + "ls2"]
    return x + cfg["residual_mult"] * y


def layer_runs(cfg):
    """[(layer, whether a pass of the loop begins with it)] in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def embed(w, cfg, tokens):
    return zero_centred_norm(w["embed"][torch.tensor(tokens)], w["embed.norm"], cfg["norm"]["eps"])


def forward(w, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer run."""
    x0 = x = embed(w, cfg, tokens)
    for i, first in layer_runs(cfg):
        if first:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        x = layer(x, w, i, cfg)
        if collect is not None:
            collect.append(x)
    z = zero_centred_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)


def read_model(folder, dtype=torch.float64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        n, = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
    w = {}
    for name, e in head.items():
        if name != "__metadata__":
            a, b = e["data_offsets"]
            w[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[e["dtype"]]).view(e["shape"]).to(dtype)
    return cfg, w
