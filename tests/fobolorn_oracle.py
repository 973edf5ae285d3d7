"""Plain, slow implementation of the Fobolorn decoder for the tests: one function per mechanism, whole sequences, no cache.

Nothing here is shared with the package: ``w`` is a dict name -> float tensor, ``cfg`` the dictionary of config.json.
Everything runs in the dtype of the weights it is given (float64 in most tests).
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def query_temperature(positions, coef, every):
    """Factor of the queries at each position."""
    blocks = torch.div(positions.double() + 1.0, float(every), rounding_mode="floor")
    return 1.0 + coef * torch.log(blocks + 1.0)


def causal_attention(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; head h reads key / value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        for i in range(T):
            s[i, i + 1:] = -math.inf
        p = torch.exp(s - s.max(1, keepdim=True).values)
        out[:, h] = (p / p.sum(1, keepdim=True)) @ v[:, g]
    return out


def head_gate(o, gate_logits):
    """One sigmoid per head."""
    return o * (1.0 / (1.0 + torch.exp(-gate_logits))).unsqueeze(-1)


def attention_mixer(h, w, p, m, eps, positions):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D)
    k = (h @ w[p + "k"].T).view(T, G, D)
    v = (h @ w[p + "v"].T).view(T, G, E)
    q = rms_norm(q, w[p + "q.norm"], eps)
    k = rms_norm(k, w[p + "k.norm"], eps)
    q = q * query_temperature(positions, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype).view(T, 1, 1)
    o = head_gate(causal_attention(q, k, v, m["scale"]), h @ w[p + "g"].T)
    return o.reshape(T, H * E) @ w[p + "o"].T


def silu_expert(h, w, p):
    z = h @ w[p + "gate"].T
    return ((z / (1.0 + torch.exp(-z))) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top, scale):
    """Router logits [T, E] -> (ids [T, top], weights [T, top])."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    val, ids = torch.topk(s, top, dim=-1)
    return ids, val / (val.sum(-1, keepdim=True) + 1e-20) * scale


def moe(h, w, p, m):
    ids, wt = route(h @ w[p + "router"].T, m["router"]["top"], m["router"]["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), wt[t]):
            out[t] += c * silu_expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    if m.get("shared"):
        g = 1.0 / (1.0 + torch.exp(-(h @ w[p + "shared.sg"].T)))
        out = out + g * silu_expert(h, w, p + "shared.")
    return out


def layer(x, w, i, spec, eps, positions):
    p = f"l{i}."
    ln = lambda n, t: layer_norm(t, w[p + n], w[p + n + ".b"], eps)      # noqa: E731
    x = x + ln("norm1b", attention_mixer(ln("norm1", x), w, p + "mix.", spec["mixer"], eps, positions))
    if spec["mlp"] is not None:
        x = x + ln("norm2b", moe(ln("norm2", x), w, p + "mlp.", spec["mlp"]))
    return x


def layer_runs(cfg):
    """[(layer, pass or None, first layer of a pass)] in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, n)]


def forward(w, cfg, tokens, collect=None):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.tensor(tokens)]
    for i, t, first in layer_runs(cfg):
        if first:
            x = x + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps, positions)
        if collect is not None:
            collect.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


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
