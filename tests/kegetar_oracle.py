"""Plain, slow implementation of the Kegetar decoder for the tests: one function per mechanism, whole sequences, no cache.

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


def bigram_rows(tokens, bigram):
    """Row of the pair table for every token; the first token has none before it and takes the extra row."""
    rows, before = [], None
    for t in tokens:
        rows.append(bigram["buckets"] if before is None else (before * bigram["mul_prev"] + t * bigram["mul_cur"]) % bigram["buckets"])
        before = t
    return rows


def embed(w, cfg, tokens):
    return w["embed"][torch.tensor(tokens)] + w["bigram"][torch.tensor(bigram_rows(tokens, cfg["embedding"]["bigram"]))]


def yarn_frequencies(dims, base, s):
    """(frequency of every pair, factor on cos and sin)."""
    def turns(t):
        return dims * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, positions, freqs, gain):
    """The first 2 len(freqs) columns of x [T, H, D] turned, column 2 i with column 2 i + 1."""
    ang = (positions.double()[:, None] * freqs[None])[:, None]
    c, s = (torch.cos(ang) * gain).to(x.dtype), (torch.sin(ang) * gain).to(x.dtype)
    n = 2 * len(freqs)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2], out[..., 1:n:2] = u * c - v * s, v * c + u * s
    return out


def visible(i, j, window, keep_first):
    return j <= i and (i - j < window or j < keep_first)


def attend(q, k, v, scale, window, keep_first=0, slopes=None):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; ``slopes`` [H]: the distance times it is taken off the score."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = (j <= i) & ((i - j < window) | (j < keep_first))
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if slopes is not None:
            s = s - slopes[h] * (i - j)
        out[:, h] = torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v[:, g]
    return out


def distance_slopes(H):
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def rotated_window_mixer(h, w, p, m, eps):
    """Left half of a parallel mixer."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freqs, gain = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"])
    pos = torch.arange(T)
    q = rotate_pairs(rms((h @ w[p + "q"].T).view(T, H, D), eps) * w[p + "q.norm"], pos, freqs, gain)
    k = rotate_pairs(rms((h @ w[p + "k"].T).view(T, G, D), eps) * w[p + "k.norm"], pos, freqs, gain)
    o = attend(q, k, (h @ w[p + "v"].T).view(T, G, E), m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    return (o.reshape(T, H * E) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def decayed_memory(q, k, v, decay, state=None):
    """q, k, decay [T, H, D], v [T, H, E].  Per head, S [D, E]:  S <- diag(decay) S + k v^T,  o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def channel_decay(z, tau):
    return sigmoid(z) ** (1.0 / tau)


def gated_linear_mixer(h, w, p, m, eps):
    """Right half of a parallel mixer."""
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5, (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, E)
    decay = channel_decay((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"], m["tau"]).view(T, H, D)
    o, _ = decayed_memory(q, k, v, decay)
    g = h @ w[p + "g"].T
    return ((rms(o, eps) * w[p + "norm"]).reshape(T, H * E) * (g * sigmoid(g))) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    a = rotated_window_mixer(h, w, p + "left.", m["left"], eps)
    b = gated_linear_mixer(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(a, eps) * w[p + "left.out"] + rms(b, eps) * w[p + "right.out"])


def shared_value_mixer(h, w, p, m, eps):
    """Values are the keys ahead of their norm; the norms run over all heads together; distances are charged per head."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, v = h @ w[p + "q"].T + w[p + "q.b"], h @ w[p + "k"].T + w[p + "k.b"]
    k = rms(v, eps) * w[p + "k.norm"]
    q = rms(q, eps) * w[p + "q.norm"]
    o = attend(q.view(T, H, D), k.view(T, G, D), v.view(T, G, D), m["scale"], m["mask"]["size"], 0, distance_slopes(H))
    return o.reshape(T, H * D) @ w[p + "o"].T


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h, w, p, m):
    y = gelu(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])
    return y @ w[p + "down"].T + w[p + "down.b"]


def clamped_expert(h, w, p, limit):
    g, u = torch.clamp(h @ w[p + "gate"].T, max=limit), torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def choose(z, correction, r):
    """Router logits of one token -> [(expert, weight)]."""
    s = torch.softmax(z, -1)
    choice = s + correction
    n = len(z) // r["groups"]["count"]
    best = sorted(range(r["groups"]["count"]), key=lambda g: -float(choice[g * n:(g + 1) * n].max()))[:r["groups"]["keep"]]
    open_to = [e for g in best for e in range(g * n, (g + 1) * n)]
    return [(e, s[e]) for e in sorted(open_to, key=lambda e: -float(choice[e]))[:r["top"]]]


def experts_ff(h, w, p, m):
    r, limit = m["router"], m["expert"]["limit"]
    z = h @ w[p + "router"].T
    out = clamped_expert(h, w, p + "shared.", m["shared"]["limit"])
    for t in range(h.shape[0]):
        for e, weight in choose(z[t], w[p + "correction"], r):
            y = clamped_expert(h[t:t + 1], w, f"{p}e{e}.", limit)[0] if e < r["experts"] else h[t]
            out[t] = out[t] + weight * y
    return out


MIXERS = {"parallel": parallel_mixer, "attention": shared_value_mixer}
FEED_FORWARDS = {"dense": dense_ff, "moe": experts_ff}


def layer(x, w, i, cfg):
    spec, eps, m = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"]
    p = f"l{spec.get('weights_of', i)}."
    x = x + m * zero_centred_norm(MIXERS[spec["type"]](x, w, p + "mix.", spec["mixer"], eps), w[p + "norm1"], eps)
    if spec["mlp"] is not None:
        x = x + m * zero_centred_norm(FEED_FORWARDS[spec["mlp"]["kind"]](x, w, p + "mlp.", spec["mlp"]), w[p + "norm2"], eps)
    return x


def forward(w, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer."""
    x = embed(w, cfg, tokens)
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg)
        if collect is not None:
            collect.append(x)
    return zero_centred_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


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
