"""Plain, slow implementation of the Lisorax decoder for the tests: one function per mechanism, whole sequences, no cache.

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


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def over_time(u, w, bias=None):
    """Causal convolution of every channel of u [T, C]; the last column of w [C, K] belongs to the current token."""
    T, K = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(K):
            if t - K + 1 + j >= 0:
                out[t] = out[t] + w[:, j] * u[t - K + 1 + j]
    return out if bias is None else out + bias


def temperature(positions, coef, every):
    return 1.0 + coef * torch.log(torch.floor((positions + 1) / every) + 1)


def key_weights(q, k, scale, softcap, r1, r2, pb):
    """Weight of every key for every query of one head: q [T, D], k [T, D] -> [T, T], zero above the diagonal."""
    T = q.shape[0]
    s = q @ k.T * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    s = s - r1 * torch.log(1 + r2 * (i - j).clamp(min=0).to(q.dtype))
    return torch.where(j <= i, sigmoid(s + pb), torch.zeros_like(s))


def attend(q, k, v, scale, softcap, r1, r2, pb):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    return torch.stack([key_weights(q[:, h], k[:, h // share], scale, softcap, r1[h], r2[h], pb[h]) @ v[:, h // share] for h in range(H)], 1)


def attention_mixer(h, w, p, m, kept, i, eps):
    """``kept``: layer -> its keys and values."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def part(x):
        return over_time(h @ w[p + x].T, w[f"{p}{x}.conv"])
    q = part("q").view(T, H, D)
    if m.get("q_temp"):
        q = q * temperature(torch.arange(T, dtype=h.dtype), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    if m.get("kv_from") is None:
        kept[i] = part("k").view(T, G, D), part("v").view(T, G, E)
    k, v = kept[i if m.get("kv_from") is None else m["kv_from"]]
    return attend(q, k, v, m["scale"], m.get("softcap"), w[p + "r1"], w[p + "r2"], w[p + "pb"]).reshape(T, H * E) @ w[p + "o"].T


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def per_block(u, mats, bias):
    """Block b of u [T, W] through the matrix mats[b] [out, in]."""
    n = mats.shape[1]
    return torch.cat([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(mats.shape[0])], 1)


def gated_recurrence(u, r, i, lam, S=None):
    """u, r, i [T, W] -> (S after every token, last S)."""
    S = torch.zeros_like(u[0]) if S is None else S.clone()
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def recurrent_mixer(h, w, p, m, kept, i, eps):
    y = gelu(h @ w[p + "y"].T + w[p + "y.b"])
    u = over_time(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    S, _ = gated_recurrence(u, sigmoid(per_block(u, w[p + "ra"], w[p + "ra.b"])), sigmoid(per_block(u, w[p + "ri"], w[p + "ri.b"])), w[p + "lam"])
    return (S * y) @ w[p + "o"].T


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, i, f, state=None):
    """q, k [T, H, D], v [T, H, E], log gates i, f [T, H] -> (o [T, H, E], (S [H, D, E], n [H, D], m [H]))."""
    T, H, D = q.shape
    S, n, m = state or (torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, add, m = torch.exp(f[t] + m - top), torch.exp(i[t] - top), top
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        low = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / low[:, None]
    return out, (S, n, m)


def memory_mixer(h, w, p, m, kept, i, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5, (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, E)
    gi = capped(h @ w[p + "i"].T + w[p + "i.b"], m["gate_cap"])
    gf = -softplus(-capped(h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"]))
    o, _ = matrix_memory(q, k, v, gi, gf)
    return (rms(o, eps).reshape(T, H * E) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def choose(z, top):
    """Router logits of one token -> [(expert, weight)]."""
    best = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    weight = torch.softmax(z[best], 0)
    return list(zip(best, weight))


def expert(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts_ff(h, w, p, m):
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in choose(z[t], m["router"]["top"]):
            out[t] = out[t] + weight * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


MIXERS = {"attention": attention_mixer, "rglru": recurrent_mixer, "mlstm": memory_mixer}


def layer(x, w, i, cfg, kept):
    spec, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    h = rms(x, eps) * w[p + "norm1"]
    y = MIXERS[spec["type"]](h + over_time(h, w[p + "canon1"]), w, p + "mix.", spec["mixer"], kept, i, eps)
    return x + y + (experts_ff(h, w, p + "mlp.", spec["mlp"]) if spec["mlp"] is not None else 0)


def forward(w, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer."""
    x, kept = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, kept)
        if collect is not None:
            collect.append(x)
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["embed"].T


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
