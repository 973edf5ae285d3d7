"""Kegetar against the plain implementation of kegetar_oracle.py, on the CPU ops and (``-m gpu``) on the device in float32 and
bfloat16: every mechanism alone, whole models, portions, batches, page and slot re-use, long decoding, generation."""
import json
import os
import subprocess
import sys

import pytest
import torch

from tensorsharp_b200.gguf.constants import GGMLType
from tensorsharp_b200.models import synth
from tensorsharp_b200.models.base import ModelBase
from tensorsharp_b200.ops import functional as F
from tensorsharp_b200.quant.qweight import QuantWeight
from tensorsharp_b200.runtime.batching import ContinuousBatcher, GenRequest, StepEngine
from tensorsharp_b200.runtime.engine import DecodeGraph, generate
from tensorsharp_b200.runtime.paged_kv import OutOfPagesError, PagedKV

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kegetar_oracle as O  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
PLACES = ["cpu", pytest.param("f32", marks=gpu), pytest.param("bf16", marks=gpu)]

CONFIGS = {
    "plain": dict(),
    # odd sizes everywhere, part of the head rotated, layers without a feed-forward, shared weights in both kinds of layers
    "odd": dict(layers="apapa", mlps="m-d-m", width=100, heads=6, kv_heads=2, dim=20, vdim=24, window=70, keep_first=9, rot_dims=12, rot_base=500.0,
                yarn=(3.0, 40, 4.0, 0.5), linear_heads=5, linear_dim=20, linear_vdim=28, tau=5.0, decay_rank=5, own_heads=10, own_kv_heads=2, own_dim=12,
                own_window=33, ff=52, expert_ff=20, limit=0.7, experts=7, identity=3, top=4, groups=(5, 3), shared_ff=50, shared_limit=2.5, buckets=97,
                muls=(1000003, 77777), vocab=333, residual_mult=0.8, weights_of={3: 1, 4: 0}),
    # one head, windows of one token, one expert of one group, nothing kept, no identity expert
    "one": dict(layers="pa", mlps="mm", heads=1, kv_heads=1, dim=16, vdim=16, window=1, keep_first=0, linear_heads=1, linear_dim=8, linear_vdim=8, tau=1.0,
                decay_rank=1, own_heads=1, own_dim=16, own_window=1, experts=1, identity=0, top=1, groups=(1, 1), shared_ff=8, expert_ff=8, residual_mult=1.0,
                yarn=(1.0, 100, 32.0, 1.0)),
    "wide": dict(layers="pa", mlps="md", width=264, heads=20, kv_heads=4, dim=48, vdim=80, window=100, keep_first=70, rot_dims=30, linear_heads=2,
                 linear_dim=128, linear_vdim=160, decay_rank=33, own_heads=40, own_kv_heads=2, own_dim=72, own_window=64, ff=200, expert_ff=96, experts=40,
                 identity=8, top=7, groups=(6, 4), shared_ff=200, vocab=1031, eps=1e-3, residual_mult=0.3, scale=0.2),
    "linear": dict(layers="pp", mlps="--", width=72, heads=2, kv_heads=1, dim=64, vdim=32, linear_heads=4, linear_dim=96, linear_vdim=64, tau=2.0, decay_rank=16),
    "far": dict(layers="pap", mlps="dmd", heads=3, kv_heads=3, dim=40, vdim=56, window=1000, keep_first=4, own_window=1000, yarn=(16.0, 64, 8.0, 0.25),
                linear_vdim=32, weights_of={2: 0}),
}


def unequal():
    """No two layers alike: sizes, windows, rotations, scales, decays and feed-forwards differ from layer to layer."""
    c = synth.kegetar_config(layers="papap", mlps="mdmmd", width=96, residual_mult=0.6, eps=1e-4)
    a, b, d, e, f = c["layers"]
    a["mixer"]["left"].update(heads=5, kv_heads=5, dim=24, vdim=40, scale=0.3, mask={"size": 9, "keep_first": 1})
    a["mixer"]["left"]["rot"].update(dims=10, base=77.0)
    a["mixer"]["right"].update(heads=2, dim=64, vdim=16, tau=1.0, decay_rank=20)
    b["mixer"].update(heads=6, kv_heads=3, dim=40, vdim=40, scale=0.1, mask={"size": 65})
    d["mixer"]["left"].update(dim=96, vdim=16, mask={"size": 31, "keep_first": 40})
    d["mixer"]["left"]["rot"]["dims"] = 96
    d["mixer"]["right"].update(heads=7, dim=16, vdim=80, tau=40.0, decay_rank=3)
    d["mlp"].update(expert={"ff": 56, "limit": 0.4}, shared={"ff": 24, "limit": 3.0}, router={"experts": 3, "identity": 5, "top": 2, "groups": {"count": 2, "keep": 1}})
    e["mixer"].update(heads=7, dim=16, vdim=16, mask={"size": 5})
    f["mlp"]["ff"] = 120
    return c


CONFIGS["unequal"] = dict(config=unequal())


def device(place):
    return "cpu" if place == "cpu" else "cuda"


def dtype(place):
    return torch.bfloat16 if place == "bf16" else torch.float32


def load(folder, place, **kw):
    kw.setdefault("max_context", 512)
    kw.setdefault("max_seqs", 4)
    return ModelBase.create(str(folder), device(place), compute_dtype=dtype(place) if place != "cpu" else None, **kw)


def poison(model):
    """NaN in every cache row that nothing has been written to, and in every state slot that no sequence has: a kernel that
    reads past a sequence's end, or a slot that is handed out as it is, shows."""
    for t in model.kv.k + model.kv.v + [model.state]:
        if t is not None:
            t.fill_(float("nan"))
    model.last_token.fill_(5)


def errors(got, want):
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def agree(got, want, place):
    """Logit rows against the oracle's: to rounding in float32; in bfloat16 to what rounding the inputs of all products to
    16 bits does to these models.  A few rows may be off by more: an expert whose choice is close may come or go, and the norm
    of a linear-attention output makes much of rounding where that output is near zero."""
    assert got.shape == want.shape
    e = errors(got, want)
    assert torch.isfinite(e).all()
    if place == "bf16":
        assert e.median() < 0.02 and (e > 0.07).sum() <= max(1, 0.05 * len(e)), (e.median(), e.max(), (e > 0.07).sum(), len(e))
    else:
        assert e.max() < 5e-5, e


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            folder = tmp_path_factory.mktemp("kegetar") / name
            synth.write_kegetar(str(folder), seed=len(name), device="cpu", **CONFIGS[name])
            made[name] = (folder,) + O.read_model(folder)
        return made[name]
    return get


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def qweight(w, dev):
    t = GGMLType.BF16 if w.dtype == torch.bfloat16 else GGMLType.F32
    return QuantWeight.from_raw(w.contiguous().view(-1).view(torch.uint8), t, tuple(w.shape), dev, "w")


def portions(kv, seqs, cuts, p, ids=None):
    """Batch of the p-th portion of every sequence that has one: (batch, [(sequence, from, to)])."""
    part = [(b, c[p], c[p + 1]) for b, c in enumerate(cuts) if c[p + 1] > c[p]]
    return kv.build_batch([seqs[b] for b, _, _ in part], [ids[b][lo:hi] if ids else [0] * (hi - lo) for b, lo, hi in part]), part


def padded(t, n, dev):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1])).to(dev).contiguous()


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("n,T", [(40, 5), (61, 300), (2050, 3), (2050, 400), (5003, 2), (5003, 310), (9001, 300)])
def test_post_norm_seam(place, n, T):
    """One branch, two branches, expert rows in any order with identity experts among them; the stream or its norm comes out."""
    dev, dt, D, eps = device(place), dtype(place), (n + 7) // 8 * 8, 1e-4
    g = torch.Generator().manual_seed(n + T)
    h0, y, z = (torch.randn(T, n, generator=g) * s for s in (2.0, 0.3, 5.0))
    y, z = y.to(dt), z.to(dt)
    post, pre, b1, b2 = (1 + 0.3 * torch.randn(n, generator=g) for _ in range(4))
    tol = dict(rtol=1e-2, atol=2e-2) if place == "bf16" else dict(rtol=1e-5, atol=3e-5)

    def run(want_x, pre_w, **kw):
        h = padded(h0, D, dev)
        out = F.post_norm_seam(h, eps, n, post=padded(post, D, dev), pre=padded(pre, D, dev) if pre_w else None, dtype=dt, **kw)
        want = h0.double() + (O.rms(want_x, eps) * post if want_x is not None else 0)
        assert torch.allclose(h[:, :n].double().cpu(), want, rtol=1e-5, atol=3e-5)
        assert torch.allclose(out[:, :n].double().cpu(), O.rms(want, eps) * pre if pre_w else want, **tol)
        assert not h[:, n:].any() and not out[:, n:].any() and out.dtype == dt
    run(y.double(), True, y=padded(y, D, dev))
    run(None, True)
    run(0.5 * (O.rms(y.double(), eps) * b1 + O.rms(z.double(), eps) * b2), False, y=padded(y, D, dev), z=padded(z, D, dev), mix=0.5,
        branch=(padded(b1, D, dev), padded(b2, D, dev)))
    # five parts per token, some of them the layer's input
    k = 5
    ids = torch.randint(-2, 4, (T, k), generator=g).clamp(min=-1)
    w = torch.rand(T, k, generator=g)
    rows = torch.randn(T * k, n, generator=g).to(dt)
    order = torch.randperm(T * k, generator=g)
    pos = torch.empty(T * k, dtype=torch.int32)
    pos[order] = torch.arange(T * k, dtype=torch.int32)
    x = (w.double() * (ids < 0)).sum(1, keepdim=True) * h0.double()
    x = x + (rows.double().view(T, k, n) * (w.double() * (ids >= 0)).unsqueeze(-1)).sum(1)
    if place == "cpu":
        parts = F.MoeParts(padded((rows.view(T, k, n) * (w * (ids >= 0)).unsqueeze(-1)).sum(1), D, dev), k, None, w, ids.int())
        run(x, False, y=parts)
    else:
        lost = rows.clone()
        lost[(ids < 0).view(-1)] = float("nan")                                # an identity expert's row is never read
        pos_d = torch.where(ids.view(-1) < 0, torch.full_like(pos, -1), pos).to(dev)
        run(x, False, y=F.MoeParts(padded(lost[order], D, dev), k, pos_d, w.to(dev), ids.int().to(dev)))
        run(x, True, y=F.MoeParts(padded(lost, D, dev), k, None, w.to(dev), ids.int().to(dev)))


@pytest.mark.parametrize("place", PLACES)
def test_pair_embedding_in_portions(place):
    """The token ahead of a portion comes from the slot; products of ids above 31 bits; a slot that is used again."""
    dev, vocab, D, big = device(place), 50021, 40, dict(buckets=613, mul_prev=2000003, mul_cur=1999993)
    g = torch.Generator().manual_seed(1)
    tok, pair = torch.randn(vocab, D, generator=g).bfloat16(), torch.randn(614, D, generator=g).bfloat16()
    kv = PagedKV([None], 40, 16, dev, max_seqs=3)
    prev = torch.full((3,), -1, dtype=torch.int32, device=dev)
    for again in range(2):
        ids = [tokens(n, vocab, n + again) for n in (40, 3, 17)]
        seqs = [kv.new_seq() for _ in ids]
        for s in seqs:
            prev[s.slot] = -1
        cuts = [[0, 20, 21, 39, 40], [0, 1, 1, 2, 3], [0, 2, 15, 16, 17]]
        for p in range(4):
            batch, part = portions(kv, seqs, cuts, p, ids)
            h, out = F.embed_pairs(qweight(tok, dev), qweight(pair, dev), batch, prev, mul_prev=big["mul_prev"], mul_cur=big["mul_cur"], dtype=dtype(place))
            want = torch.cat([(tok[ids[b]].float() + pair[O.bigram_rows(ids[b], big)].float())[lo:hi] for b, lo, hi in part])
            assert torch.equal(h.cpu(), want) and torch.equal(out.cpu(), want.to(dtype(place)))
        for s in seqs:
            kv.free_seq(s)


YARN = [(32, 10000.0, dict(factor=5.0, original=1500, fast=20.0, slow=0.7)), (10, 77.0, dict(factor=3.0, original=40, fast=4.0, slow=0.5)),
        (64, 1e6, dict(factor=1.0, original=4096, fast=32.0, slow=1.0)), (8, 1000.0, dict(factor=40.0, original=2, fast=32.0, slow=1.0)),
        (6, 50.0, dict(factor=2.0, original=10 ** 7, fast=2.0, slow=2.0))]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("dims,base,scaling", YARN)
def test_scaled_rotation_of_neighbouring_pairs(place, dims, base, scaling):
    """Norm and rotation of padded heads at near and far positions; ramps inside, outside and of no width."""
    dev, pos, H, G, dim, vdim = device(place), [0, 1, 2, 63, 64, 999, 1000, 65535], 3, 1, 70, 20
    freq, gain = F.yarn_freqs(dims, base, scaling, dev)
    wf, wg = O.yarn_frequencies(dims, base, scaling)
    assert torch.allclose(freq.cpu(), wf, rtol=1e-12) and abs(gain - wg) < 1e-12
    if dims > dim:
        return
    g = torch.Generator().manual_seed(dims)
    T, Dk, Dv = len(pos), 80, 32
    q, k, v = (torch.randn(T, h, d, generator=g) for h, d in ((H, dim), (G, dim), (G, vdim)))
    qn, kn = torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    kv = PagedKV([(G, Dk, Dv)], 4, 64, dev, dtype(place), max_seqs=1)
    batch = kv.build_batch([kv.new_seq()], [[0] * T])
    batch.positions = torch.tensor(pos, dtype=torch.int32, device=dev)
    got = F.qkv_rope_cache(padded(q, Dk, dev), padded(k, Dk, dev), padded(v, Dv, dev), Hq=H, Hkv=G, Dh=Dk, Dv=Dv, norm_n=dim, batch=batch, k_cache=kv.k[0],
                           v_cache=kv.v[0], rope=F.RopeSpec(dims, base, mode=1, attn_factor=gain, freq=freq), qn=padded(qn, Dk, dev), kn=padded(kn, Dk, dev),
                           eps=1e-5)
    tol = dict(rtol=1e-2, atol=2e-2) if place == "bf16" else dict(rtol=1e-5, atol=2e-5)
    at = torch.tensor(pos)
    assert torch.allclose(got[..., :dim].double().cpu(), O.rotate_pairs(O.rms(q.double(), 1e-5) * qn, at, wf, wg), **tol) and not got[..., dim:].any()
    rows = kv.k[0][batch.slots].double().cpu()
    assert torch.allclose(rows[..., :dim], O.rotate_pairs(O.rms(k.double(), 1e-5) * kn, at, wf, wg), **tol) and not rows[..., dim:].any()
    assert torch.allclose(kv.v[0][batch.slots].double().cpu()[..., :vdim], v.double(), **tol)


ATTENTION = [  # H, G, dim, vdim, window, kept first, distance bias, gate per column, one row for key and value
    (4, 2, 32, 48, 24, 3, False, True, False), (6, 2, 20, 24, 70, 9, False, True, False), (3, 3, 64, 64, 1, 0, False, False, False),
    (20, 1, 48, 80, 33, 130, False, True, False), (2, 1, 128, 128, 64, 1, False, True, False), (5, 5, 16, 16, 65, 64, False, True, False),
    (4, 1, 32, 32, 20, 0, True, False, True), (10, 2, 12, 12, 33, 0, True, False, True), (7, 1, 64, 64, 64, 0, True, False, True),
    (40, 2, 72, 72, 1, 0, True, False, True), (6, 6, 128, 128, 65, 0, True, True, False), (4, 4, 256, 256, 17, 5, True, False, True)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,dim,vdim,window,first,bias,gated,own", ATTENTION)
def test_attention_with_keys_that_stand_out(place, H, G, dim, vdim, window, first, bias, gated, own):
    """Single keys stand out from all others for one query each: just inside the window, just outside of it, among the kept
    first tokens, the next one after them, at page borders, and one ahead of the query; on pages in no order, in portions and
    decoding, over poisoned free rows."""
    dev, dt, page = device(place), dtype(place), 16
    g = torch.Generator().manual_seed(H * dim + window)
    Dk, Dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    lens = [150, 33, 209]
    kv = PagedKV([(1, G * Dk + 8, 0) if own else (G, Dk, Dv)], 40, page, dev, dt, max_seqs=3)
    kv._free = torch.randperm(40, generator=g).tolist()
    kv.k[0].fill_(float("nan"))
    kv.v[0].fill_(float("nan"))
    seqs = [kv.new_seq() for _ in lens]
    slopes = [2.0 ** (-8.0 * (h + 1) / H) / 8 for h in range(H)] if bias else None
    data, want = [], []
    for n in lens:
        q, k, v = (torch.randn(n, a, d, generator=g) * s for a, d, s in ((H, dim, 0.3), (G, dim, 0.3), (G, vdim, 1.0)))
        gate = torch.randn(n, H, vdim, generator=g)
        factor = torch.rand(n, generator=g) + 0.5
        pairs = []
        for i in (n - 1, n - 2, n // 2, n // 3, window + first, page, 2 * page - 1):
            pairs += [(i, j) for j in (i - window + 1, i - window, first - 1, first, 0, i - 1, page - 1, page, i + 1) if 0 <= j < n and i < n]
        marks = max(1, min(dim // 2, 8))                      # columns that only a marked key uses
        k[..., :marks] = 0
        q[..., :marks] = 0
        for m, (i, j) in enumerate(pairs[::max(1, len(pairs) // marks)][:marks]):
            k[j, :, m], q[i, :, m] = 3.0, 8.0
        q, k, v, gate = (t.to(dt) for t in (q, k, v, gate))
        data.append((q, k, v, gate, factor))
        kk, vv = (k.double() * factor.double().view(n, 1, 1), k.double()) if own else (k.double(), v.double())
        o = O.attend(q.double(), kk, vv, 0.4, window, first, slopes)
        want.append(o * O.sigmoid(gate.double()) if gated else o)
    cuts = [[0, 2, 17, 64, 148, 149, 150], [0, 16, 31, 32, 32, 32, 33], [0, 1, 130, 193, 207, 208, 209]]      # the last two: decoding
    for p in range(6):
        batch, part = portions(kv, seqs, cuts, p)
        assert batch.is_decode == (p >= 4)

        def rows(x):
            return torch.cat([data[b][x][lo:hi] for b, lo, hi in part])
        if own:
            row = torch.zeros(batch.T, G * Dk + 8, dtype=dt)
            row[:, :G * Dk] = padded(rows(1), Dk, "cpu").view(batch.T, -1)
            if dt == torch.float32:
                row[:, G * Dk] = rows(4)
            else:
                row[:, G * Dk:G * Dk + 2] = rows(4).view(-1, 1).contiguous().view(torch.bfloat16)
            kv.k[0][batch.slots] = row.unsqueeze(1).to(dev)
        else:
            kv.k[0][batch.slots], kv.v[0][batch.slots] = padded(rows(1), Dk, dev), padded(rows(2), Dv, dev)
        gate = torch.nn.functional.pad(padded(rows(3), Dv, dev).view(batch.T, -1), (0, 8))[:, :-8] if gated else None      # a row stride of its own
        out = F.attention(padded(rows(0), Dk, dev), kv.k[0], kv.k[0] if own else kv.v[0], batch, scale=0.4, Hq=H, Hkv=G, Dh=Dk, Dv=Dv, window=window,
                          keep_first=first, slopes=torch.tensor(slopes).to(dev) if bias else None, gate=gate, own_values=own).view(batch.T, H, Dv)
        ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
        err = (out[..., :vdim].double().cpu() - ref).abs().max()
        assert err < (0.04 if place == "bf16" else 1e-4), (p, err)
        assert not out[..., vdim:].any()


def test_what_the_window_and_the_kept_tokens_show():
    """The oracle itself: a query that asks for one key finds it exactly where it is visible."""
    T, W, K = 40, 7, 3
    for i in (0, 2, 6, 7, 9, 10, 39):
        for j in range(T):
            q, k, v = torch.zeros(T, 1, 2), torch.zeros(T, 1, 2), torch.zeros(T, 1, 1)
            q[i, 0, 0] = k[j, 0, 0] = 10.0
            v[j] = 1.0
            seen = float(O.attend(q, k, v, 1.0, W, K)[i, 0, 0]) > 0.99
            assert seen == O.visible(i, j, W, K) == (j <= i and (i - j < W or j < K))
    assert O.distance_slopes(8) == [0.5, 0.25, 0.125, 0.0625, 0.03125, 0.015625, 0.0078125, 0.00390625]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,dim,T", [(4, 1, 32, 5), (10, 2, 12, 400), (40, 5, 72, 3), (33, 33, 128, 2), (24, 8, 100, 320), (64, 4, 256, 2)])
def test_norms_over_whole_projections(place, H, G, dim, T):
    """Queries times keys of the finished form: factor and norm weights are where they belong, and the values are untouched."""
    dev, eps, Dk = device(place), 1e-3, (dim + 15) // 16 * 16
    g = torch.Generator().manual_seed(dim)
    q, k = torch.randn(T, H * dim, generator=g) * torch.rand(T, 1, generator=g), torch.randn(T, G * dim, generator=g) * 3
    qn, kn = torch.randn(H * dim, generator=g), torch.randn(G * dim, generator=g)

    def heads(x, n):
        return torch.nn.functional.pad(x.view(*x.shape[:-1], n, dim), (0, Dk - dim)).reshape(*x.shape[:-1], n * Dk)
    kv = PagedKV([(1, G * Dk + 8, 0)], 40, 16, dev, dtype(place), max_seqs=1)
    kv.k[0].fill_(float("nan"))
    batch = kv.build_batch([kv.new_seq()], [[0] * T])
    w = heads(qn, H) * heads(kn, G).view(G, 1, Dk).expand(G, H // G, Dk).reshape(-1)
    got = F.joint_norm_cache(torch.cat([heads(q, H), heads(k, G)], 1).to(dev), w.to(dev), kv.k[0], batch, nq=H * Dk, nk=G * Dk, q_n=H * dim, k_n=G * dim, eps=eps)
    rows = kv.k[0][batch.slots, 0].cpu()
    fac = rows[:, G * Dk:].float()[:, 0] if place != "bf16" else rows[:, G * Dk:G * Dk + 2].contiguous().view(torch.float32)[:, 0]
    assert not rows[:, G * Dk + (1 if place != "bf16" else 2):].any()
    rel = 1e-2 if place == "bf16" else 1e-5
    assert torch.allclose(fac.double(), 1 / torch.sqrt(k.double().pow(2).mean(1) + eps), rtol=1e-6)
    assert torch.allclose(rows[:, :G * Dk].double(), heads(k, G).double(), rtol=rel, atol=rel)
    want = (O.rms(q.double(), eps) * qn).view(T, H, dim) * kn.view(G, 1, dim).expand(G, H // G, dim).reshape(H, dim)
    got = got.view(T, H, Dk)
    assert torch.allclose(got[..., :dim].double().cpu(), want, rtol=rel, atol=rel) and not got[..., dim:].any()


ROUTERS = [(6, 2, 3, (4, 2), 2), (1, 0, 1, (1, 1), 0), (7, 3, 4, (5, 3), 1), (40, 8, 7, (6, 4), 3), (30, 2, 8, (32, 9), 0), (150, 10, 32, (16, 5), 4),
           (900, 100, 5, (500, 400), 1), (3, 5, 2, (2, 1), 2)]


@pytest.mark.parametrize("place", ["cpu", pytest.param("f32", marks=gpu)])
@pytest.mark.parametrize("E,identity,top,groups,slices", ROUTERS)
def test_routing_in_groups(place, E, identity, top, groups, slices):
    """Choices on corrected scores (many of them negative) within the best groups, weights without the correction."""
    dev, T, n = device(place), 33, E + identity
    g = torch.Generator().manual_seed(n)
    z, c = torch.randn(T, n, generator=g) * 2, torch.randn(n, generator=g) * 0.3 - 0.4
    ids, w = F.route_softmax_groups(z.to(dev), c.to(dev), top, groups=groups[0], keep=groups[1], n_real=E, n_always=slices)
    assert ids.dtype == torch.int32 and ids.shape == w.shape == (T, slices + top)
    ids, w = ids.cpu(), w.cpu()
    assert (ids[:, :slices] == torch.arange(slices)).all() and (w[:, :slices] == 1).all()
    r = {"groups": {"count": groups[0], "keep": groups[1]}, "top": top}
    for t in range(T):
        want = O.choose(z[t].double(), c.double(), r)
        assert ids[t, slices:].tolist() == [slices + e if e < E else -1 for e, _ in want]
        assert torch.allclose(w[t, slices:].double(), torch.stack([s for _, s in want]), rtol=1e-5, atol=1e-9)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T", [1, 3, 15, 200, 1500])
@pytest.mark.parametrize("E,ff,shared,limits", [(6, 24, 40, (0.5, 2.0)), (3, 64, 64, (1.5, 1.5)), (5, 16, 0, (0.2, 9.0))])
def test_experts_with_identity_and_a_shared_expert(place, T, E, ff, shared, limits):
    """Few and many tokens (matrix-vector, sorted and grouped products); clamps that bite, other ones for the shared expert."""
    dev, dt, D, slices, k = device(place), dtype(place), 48, -(-shared // ff), 4
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, D, generator=g).to(dt)
    n = E + slices
    gate, up, down = (torch.randn(n, a, b, generator=g).div(b ** 0.5).to(dt) for a, b in ((ff, D), (ff, D), (D, ff)))
    ids = torch.stack([torch.randperm(E + 3, generator=g)[:k] for _ in range(T)])
    ids = torch.where(ids < E, ids + slices, torch.full_like(ids, -1))
    if T > 1:
        ids[:, 0] = -1                                                          # a third to all of a token's experts hand it on
        ids[1] = -1
    ids = torch.cat([torch.arange(slices).expand(T, slices), ids], 1)
    w = torch.rand(T, slices + k, generator=g)
    w[:, :slices] = 1
    parts = F.moe_expert_parts(F.Act(x.to(dev)), ids.int().to(dev), w.to(dev), qweight(torch.cat([gate, up], 1), dev), qweight(down, dev), act="swiglu_oai",
                               clamp=(limits[0], limits[1], slices), identity=True)
    ones = torch.ones(D, device=dev)
    h = x.float().clone().to(dev)
    F.post_norm_seam(h, 1e-6, D, y=parts, post=ones, dtype=dt)
    want = torch.zeros(T, D, dtype=torch.float64)
    for e in range(n):
        wd = {"gate": gate[e].double(), "up": up[e].double(), "down": down[e].double()}
        y = O.clamped_expert(x.double(), wd, "", limits[1] if e < slices else limits[0])
        want += y * (w.double() * (ids == e)).sum(1, keepdim=True)
    want += x.double() * (w.double() * (ids < 0)).sum(1, keepdim=True)
    want = x.double() + O.rms(want, 1e-6)
    assert torch.allclose(h.double().cpu(), want, **(dict(rtol=0.02, atol=0.05) if place == "bf16" else dict(rtol=1e-4, atol=1e-4)))


LINEAR = [(3, 20, 28, 5), (2, 64, 16, 16), (5, 96, 33, 33), (4, 128, 128, 24), (1, 150, 100, 3), (2, 256, 160, 8), (40, 32, 8, 8), (1, 200, 256, 70)]


def pad_heads(v, H, n, D):
    return torch.nn.functional.pad(v.view(*v.shape[:-1], H, n), (0, D - n)).reshape(*v.shape[:-1], H * D)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,n,e,rank", LINEAR)
def test_gated_linear_attention_in_portions(place, H, n, e, rank):
    """The recurrence with its decay map, norm and gate: single steps and chunk kernels in turns, unequal sequences, a slot that
    is given back and used again.  Some channels forget next to nothing, so what is written at the start still shows at the
    end, others forget all at once."""
    dev, eps, dt, rp = device(place), 1e-4, dtype(place), (rank + 7) // 8 * 8
    s = F.GatedLinearSpec(H, n, e, 3.0)
    D, E = s.D, s.E
    g = torch.Generator().manual_seed(H * n)
    lens = [290, 19, 33]
    w2, zb = torch.randn(H * n, rank, generator=g).to(dt), torch.randn(H * n, generator=g) * 2
    on = torch.randn(e, generator=g)
    zb[::3] += 14
    zb[1::5] -= 60
    x = [{a: torch.randn(m, H * d, generator=g).to(dt) for a, d in (("q", n), ("k", n), ("v", e), ("g", e))} for m in lens]
    low = [torch.randn(m, rank, generator=g).to(dt) for m in lens]
    want = []
    for xs, lo in zip(x, low):
        q, k, v, gate = (xs[a].double().view(len(lo), H, -1) for a in "qkvg")
        decay = O.channel_decay(lo.double() @ w2.double().T + zb.double(), 3.0).view(-1, H, n)
        o, _ = O.decayed_memory(q * n ** -0.5, k, v, decay)
        want.append(O.rms(o, eps) * on.double() * gate * O.sigmoid(gate))
    state = torch.full((3, 7 * 4 + H * E * D), float("nan"), device=dev)[:, 28:].unflatten(1, (H, E, D))
    kv = PagedKV([None], 60, 16, dev, max_seqs=3)
    w2d = torch.zeros(H, D, rp, dtype=dt)
    w2d[:, :n, :rank] = w2.view(H, n, rank)
    w2d = qweight(w2d.view(H * D, rp), dev)
    cols = (0, H * D, 2 * H * D, 2 * H * D + H * E, 2 * H * D + 2 * H * E)
    for again in range(2):
        seqs = [kv.new_seq() for _ in lens]
        for q in seqs:
            state[q.slot] = 0
        cuts = [[0, 1, 30, 289, 290], [0, 10, 17, 18, 19], [0, 7, 7, 32, 33]]
        for p in range(4):
            batch, part = portions(kv, seqs, cuts, p)
            y = torch.cat([torch.cat([pad_heads(x[b]["q"][lo:hi], H, n, D), pad_heads(x[b]["k"][lo:hi], H, n, D), pad_heads(x[b]["v"][lo:hi], H, e, E),
                                      pad_heads(x[b]["g"][lo:hi], H, e, E), torch.nn.functional.pad(low[b][lo:hi], (0, rp - rank))], 1) for b, lo, hi in part])
            if batch.T <= F.GEMV_MAX_M:
                y = y.float()
            y = torch.nn.functional.pad(y, (0, 8)).to(dev)[:, :-8]                # a row stride of its own
            out = F.gated_linear(y, s, cols, w2d, padded(pad_heads(zb, H, n, D), H * D, dev), padded(on, E, dev), state, batch, eps=eps, dtype=dt)
            got = out.double().cpu().view(-1, H, E)
            ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
            err = (got[..., :e] - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
            assert err < (0.01 if place == "bf16" else 2e-5), (p, err)
            assert not got[..., e:].any()
        for q in seqs:
            kv.free_seq(q)


@gpu
@pytest.mark.parametrize("H,n,e", [(h, n, e) for h, n, e, _ in LINEAR])
@pytest.mark.parametrize("segs", [1, 2, 5])
def test_linear_attention_chunk_kernel_keeps_32_bits(H, n, e, segs):
    """The tensor-core path from bf16 rows: the state it leaves against the oracle's to 32-bit rounding, and its results to one
    rounding of the output; unequal sequences, full and short chunks and segments, states that are not zero."""
    from tensorsharp_b200.ops import kernels as K
    s, eps = F.GatedLinearSpec(H, n, e, 1.0), 1e-5
    D, E = s.D, s.E
    g = torch.Generator().manual_seed(n)
    cu = [0, 1, 104, 112, 128, 291]
    T = cu[-1]
    q, k = (torch.randn(T, H * n, generator=g).bfloat16() for _ in range(2))
    v, gate = (torch.randn(T, H * e, generator=g).bfloat16() for _ in range(2))
    z, zb, on = torch.randn(T, H * n, generator=g) * 3, torch.randn(H * n, generator=g) * 2, torch.randn(e, generator=g)
    z[:, ::2] += 12
    z[:, 1::7] -= 50
    s0 = torch.randn(6, H, e, n, generator=g)
    state = torch.zeros(6, H, E, D)
    state[:, :, :e, :n] = s0
    slots = torch.tensor([4, 0, 5, 2, 1])
    y = torch.cat([pad_heads(q, H, n, D), pad_heads(k, H, n, D), pad_heads(v, H, e, E), pad_heads(gate, H, e, E)], 1).cuda()
    cols = (0, H * D, 2 * H * D, 2 * H * D + H * E, 0)
    st = state.cuda()
    out = K.gla_prompt(y, s, cols, pad_heads(z, H, n, D).cuda(), pad_heads(zb, H, n, D).cuda(), padded(on, E, "cuda"), st,
                       torch.tensor(cu, dtype=torch.int32).cuda(), slots.cuda(), eps=eps, max_q=163, segs=segs).double().cpu().view(T, H, E)
    st = st.double().cpu()
    decay = O.sigmoid(z.double() + zb.double()).view(T, H, n)
    for b, (lo, hi) in enumerate(zip(cu, cu[1:])):
        part = [t[lo:hi].double().view(hi - lo, H, -1) for t in (q, k, v, gate)]
        o, S = O.decayed_memory(part[0] * n ** -0.5, part[1], part[2], decay[lo:hi], s0[slots[b]].double().transpose(1, 2))
        got = st[slots[b], :, :e, :n].transpose(1, 2)
        assert torch.allclose(got, S, rtol=2e-5, atol=2e-5), (b, (got - S).abs().max())
        want = O.rms(o, eps) * on.double() * part[3] * O.sigmoid(part[3])
        assert torch.allclose(out[lo:hi, :, :e], want, rtol=5e-3, atol=1e-4), (b, (out[lo:hi, :, :e] - want).abs().max())
        assert not out[lo:hi, :, e:].any() and not st[slots[b], :, e:].any() and not st[slots[b], :, :, n:].any()
    assert torch.equal(st[3], state[3].double())                                # nobody's slot


def test_what_the_memory_keeps():
    """The oracle itself: without decay a value comes back for its key however far away; a channel that forgets at once keeps
    the newest value only."""
    D = 16
    g = torch.Generator().manual_seed(0)
    k = torch.eye(D, dtype=torch.float64)[:, None]
    v = torch.randn(D, 1, 5, generator=g, dtype=torch.float64)
    q = torch.zeros(D, 1, D, dtype=torch.float64)
    q[D - 1, 0, 3] = 1
    one = torch.ones(D, 1, D, dtype=torch.float64)
    assert torch.allclose(O.decayed_memory(q, k, v, one)[0][-1, 0], v[3, 0])
    one[..., 3] = 0
    assert not O.decayed_memory(q, k, v, one)[0][-1, 0].any()
    q[D - 1, 0] = torch.eye(D)[D - 1]
    assert torch.allclose(O.decayed_memory(q, k, v, 0 * one)[0][-1, 0], v[-1, 0])


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_against_the_oracle(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    got, want = [], []
    for n in (1, 2, 9, 77, 200):
        ids = tokens(n, cfg["vocab"], n)
        s = m.new_sequence()
        got.append(m.forward_batch(m.kv.build_batch([s], [ids], rows=[list(range(n))])))
        want.append(O.forward(w, cfg, ids))
        m.free_sequence(s)
    agree(torch.cat(got), torch.cat(want), place)
    if place != "cpu":
        m.poll_status(force=True)


def test_layers_that_share_weights(models):
    """One set of tensors, caches and states of their own."""
    folder, cfg, w = models("odd")
    assert not any(n.startswith(("l3.", "l4.")) for n in w)
    m = load(folder, "cpu")
    assert m.layers[3] is m.layers[1] and m.layers[4] is m.layers[0] and m.layers[2] is not m.layers[0]
    assert [t.shape[1:] for t in m.kv.k] == [(1, 40), (2, 32), (1, 40), (2, 32), (1, 40)] and [t.shape[2] for t in m.kv.v] == [0, 32, 0, 32, 0]
    assert len({t.data_ptr() for t in m.kv.k}) == 5
    assert [t is None for t in m.memory] == [True, False, True, False, True]
    assert (m.memory[3].data_ptr() - m.memory[1].data_ptr()) // 4 == m.memory[1][0].numel() == m.state.shape[1] // 2


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "plain", "wide", "unequal"])
@pytest.mark.parametrize("cut", [[1], [2], [3, 2, 61], [64], [23, 1, 24, 2, 70]])
def test_portions_and_token_by_token(models, place, name, cut):
    """However a prompt is cut, its logits are the same."""
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    n = 90 if cut == [1] else 150
    ids = tokens(n, cfg["vocab"], 5)
    want = O.forward(w, cfg, ids)
    eng, got, at, i = StepEngine(m, 4), [], 0, 0
    while at < n:
        k = min(cut[i % len(cut)], n - at)
        got.append(eng.step([("a", ids[at:at + k], list(range(k)))]))
        at, i = at + k, i + 1
    agree(torch.cat(got), want, place)


PLAN = [[("a", 60), ("b", 2)], [("b", 61), ("a", 5)], [("a", 1), ("b", 1), ("c", 39)], [("c", 1), ("a", 1), ("d", 1)], [("a", 62)], [("a", 1)],
        [("e", 65), ("f", 3)], [("f", 1), ("e", 1)], [("f", 1)], [("e", 2), ("f", 64)], [("e", 121), ("f", 1)], [("e", 1)]]


def run_plan(m, cfg, w, place):
    names = {"a": 130, "b": 64, "c": 40, "d": 1, "e": 190, "f": 70}
    ids = {k: tokens(n, cfg["vocab"], ord(k)) for k, n in names.items()}
    want = {k: O.forward(w, cfg, t) for k, t in ids.items()}
    at, got = {k: 0 for k in ids}, {k: [] for k in ids}
    eng, slots = StepEngine(m, 4), set()
    for step in PLAN:
        out = eng.step([(k, ids[k][at[k]:at[k] + n], list(range(n))) for k, n in step])
        row = 0
        for k, n in step:
            got[k].append(out[row:row + n])
            row, at[k] = row + n, at[k] + n
            slots.add(eng.live[k].slot)
            if at[k] == names[k]:
                eng.end(k)
    assert at == names and not eng.live and len(slots) < len(names)
    for k in ids:
        agree(torch.cat(got[k]), want[k], place)
    return eng


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "far", "wide"])
def test_batches_of_unequal_requests_on_pages_and_slots_used_before(models, place, name):
    """Portions beside single tokens, a request left out of steps, requests that end and others that take their pages and
    slots; the pool holds no page to spare."""
    folder, cfg, w = models(name)
    m = load(folder, place, max_context=320, kv_pages=5)
    poison(m)
    eng = run_plan(m, cfg, w, place)
    assert m.kv.free_pages == 5
    with pytest.raises(OutOfPagesError):
        eng.step([("x", tokens(321, 333), [])])
    with pytest.raises(ValueError):
        eng.step([("y", [1, 2], [2])])


@pytest.mark.parametrize("place", PLACES)
def test_alone_and_in_a_batch(models, place):
    """A request's logits do not depend on what it is batched with, on its pages or on its slot."""
    folder, cfg, w = models("unequal")
    m = load(folder, place)
    ids = tokens(70, cfg["vocab"], 3)
    alone = StepEngine(m, 4)
    a = torch.cat([alone.step([("a", ids[:40], list(range(40)))])] + [alone.step([("a", ids[i:i + 1], [0])]) for i in range(40, 70)])
    alone.end("a")
    eng = StepEngine(m, 4)
    eng.step([("x", tokens(100, cfg["vocab"], 9), []), ("y", tokens(1, cfg["vocab"], 8), [])])
    b = [eng.step([("y", [3], []), ("a", ids[:40], list(range(40))), ("x", [7, 8, 9], [])])]
    b += [eng.step([("x", [i % 300], []), ("a", ids[i:i + 1], [0])]) for i in range(40, 70)]
    e = errors(torch.cat(b), a.double().cpu())
    assert e.median() < (0.02 if place == "bf16" else 1e-5) and (e > (0.07 if place == "bf16" else 5e-5)).sum() <= (3 if place == "bf16" else 0)


@pytest.mark.parametrize("place", PLACES)
def test_rings_of_pages_for_the_window(models, place, monkeypatch):
    """With a ring of pages per sequence the rows that have left the window are overwritten; layers that keep their first tokens
    have no ring."""
    monkeypatch.setenv("TSB_KV_WINDOW_RING", "1")
    monkeypatch.setenv("TSB_KV_RING_CHUNK", "64")
    folder, cfg, w = models("plain")
    m = load(folder, place, max_context=320, page_size=16)
    poison(m)
    assert m.kv.ring and m.kv.ring_pages * 16 < 190 and sorted(m.kv.window_layers) == [1, 3]
    n, eng, got = 190, StepEngine(m, 4), []
    ids = tokens(n, cfg["vocab"], 6)
    for a, b in ((0, 64), (64, 100), (100, 101), (101, 160), (160, 180)) + tuple((i, i + 1) for i in range(180, n)):
        got.append(eng.step([("a", ids[a:b], list(range(b - a)))]))
    agree(torch.cat(got), O.forward(w, cfg, ids), place)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["linear", "plain"])
def test_wanted_rows_only(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    ids = tokens(50, cfg["vocab"], 2)
    want = O.forward(w, cfg, ids)
    eng = StepEngine(m, 4)
    assert eng.step([("a", ids[:20], [])]) is None
    agree(eng.step([("a", ids[20:45], [24, 0, 7])]), want[[44, 20, 27]], place)
    assert eng.step([("a", ids[45:46], [])]) is None
    assert eng.step([("a", ids[46:47], [0]), ("b", ids[:1], [])]).shape == (1, cfg["vocab"])
    agree(eng.step([("b", ids[1:2], [0]), ("a", ids[47:48], [0])]), want[[1, 47]], place)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["plain", "odd"])
def test_long_decoding(models, place, name):
    """Hundreds of single steps (captured graphs on the device) after a short prompt, over several pages and windows."""
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    n = 300
    ids = tokens(n, cfg["vocab"], 8)
    want = O.forward(w, cfg, ids)
    eng = StepEngine(m, 2)
    got = [eng.step([("a", ids[:3], [0, 1, 2])])] + [eng.step([("a", ids[i:i + 1], [0])]) for i in range(3, n)]
    if place != "cpu":
        assert eng.stepper.replays >= n - 4
    agree(torch.cat(got), want, place)


# ------------------------------------------------------------------------------------------ generation and entry points
def greedy_is_argmax(w, cfg, prompt, out, slack):
    """Every token is the oracle's best for what precedes it, up to ``slack`` standard deviations."""
    rows = O.forward(w, cfg, prompt + out)[len(prompt) - 1:-1]
    short = rows.max(1).values - rows[torch.arange(len(out)), torch.tensor(out)]
    assert (short <= slack * rows.std(1)).all(), short


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("portion", [2, 64])
def test_greedy_generation_through_the_scheduler(models, place, portion):
    folder, cfg, w = models("odd")
    m = load(folder, place)
    poison(m)
    prompts = [tokens(n, cfg["vocab"], n) for n in (5, 70, 1, 33, 12)]
    slack = 0.15 if place == "bf16" else 1e-3
    eng = ContinuousBatcher(m, 3, prefill_chunk=portion)
    reqs = eng.run([GenRequest(p, 20) for p in prompts])
    assert m.kv.free_pages == m.kv.n_pages
    for p, r in zip(prompts, reqs):
        assert r.error is None and len(r.ids) == 20
        greedy_is_argmax(w, cfg, p, r.ids, slack)
        m.reset_kv_cache()
        alone = generate(m, p, 20, prefill_chunk=16)
        greedy_is_argmax(w, cfg, p, alone, slack)
        if place != "bf16":
            assert alone == r.ids
    bad = eng.run([GenRequest([], 4), GenRequest(prompts[0], 4)])
    assert bad[0].error and bad[1].error is None and bad[1].ids == reqs[0].ids[:4]


@gpu
def test_graph_decoding_advances_the_state_once(models):
    """A captured decode loop gives the tokens of the step-by-step loop: the capture's own step leaves no trace, neither in the
    memories nor in the last token."""
    folder, cfg, w = models("odd")
    m = load(folder, "f32")
    prompt = tokens(20, cfg["vocab"], 1)
    want = generate(m, prompt, 12)
    s = m.new_sequence()
    first = int(m.forward_batch(m.kv.build_batch([s], [prompt])).argmax())
    dg = DecodeGraph(m, [s], 16)
    dg.set_tokens([first])
    dg.capture()
    assert [first] + [int(dg.step()) for _ in range(11)] == want


def test_pool_too_small_for_all_requests(models):
    """Without a free page the youngest request is given up and the others finish."""
    folder, cfg, w = models("plain")
    m = load(folder, "cpu", kv_pages=3, max_context=192)
    prompts = [tokens(60, cfg["vocab"], 1), tokens(100, cfg["vocab"], 2), tokens(90, cfg["vocab"], 3)]
    reqs = ContinuousBatcher(m, 3, prefill_chunk=50).run([GenRequest(p, 10) for p in prompts])
    assert any(r.error for r in reqs) and any(r.error is None for r in reqs) and m.kv.free_pages == 3
    for p, r in zip(prompts, reqs):
        if r.error is None:
            greedy_is_argmax(w, cfg, p, r.ids, 1e-3)


@pytest.mark.parametrize("place", ["cpu", pytest.param("b200", marks=gpu)])
def test_command_line(models, place, tmp_path):
    from tensorsharp_b200.cli.main import main
    folder, cfg, w = models("odd")
    prompt = tokens(12, cfg["vocab"], 4)
    src, dst = tmp_path / "in.jsonl", tmp_path / "out.jsonl"
    text = " ".join(map(str, prompt))
    src.write_text("".join(json.dumps({"id": f"r{i}", "prompt": text, "messages": [{"role": "user", "content": text}], "max_tokens": 6}) + "\n"
                           for i in range(3)))
    for extra in ([], ["--batch-size", "2"], ["--dtype", "float32"]):
        assert main(["--model", str(folder), "--backend", place, "--input-jsonl", str(src), "--output", str(dst), "--log-file", "off"] + extra) == 0
        rows = [json.loads(x) for x in dst.read_text().splitlines()]
        assert [r["id"] for r in rows] == ["r0", "r1", "r2"]
        for r in rows:
            ids = [int(x) for x in r["output"].split()]
            assert len(ids) == 6
            greedy_is_argmax(w, cfg, prompt, ids, 0.15 if place == "b200" else 1e-3)


@pytest.mark.parametrize("place", PLACES)
def test_trace_runner(models, place, tmp_path):
    folder, cfg, w = models("odd")
    ids = {k: tokens(n, cfg["vocab"], n) for k, n in (("p", 90), ("q", 66))}
    steps = [([("p", 0, 64, [0, 63])], []), ([("q", 0, 2, []), ("p", 64, 89, [3])], []), ([("q", 2, 65, [1, 62]), ("p", 89, 90, [0])], ["p"]),
             ([("q", 65, 66, [0])], ["q"])]
    text = "".join(json.dumps({"step": n, "entries": [{"id": k, "tokens": ids[k][a:b], "want": want} for k, a, b, want in e], "end": end}) + "\n"
                   for n, (e, end) in enumerate(steps))
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", "bfloat16" if place == "bf16" else "float32", "--out",
           str(tmp_path / "o"), "--max-tokens", "256"] + (["--device", "cpu"] if place == "cpu" else [])
    r = subprocess.run(cmd, input=text, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done ")] == [f"done {n}" for n in range(len(steps))]
    full = {k: O.forward(w, cfg, t) for k, t in ids.items()}
    got, want = [], []
    for n, (entries, _) in enumerate(steps):
        rows = [full[k][a + i] for k, a, _, places in entries for i in places]
        data = torch.frombuffer(bytearray((tmp_path / "o" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert data.shape[0] == len(rows)
        got.append(data)
        want.append(torch.stack(rows))
    agree(torch.cat(got), torch.cat(want), place)


def test_server_lists_and_loads_the_folder(models):
    from tensorsharp_b200.server.model_service import ModelService
    folder, cfg, _ = models("plain")
    svc = ModelService()
    assert folder.name in svc.scan_models(str(folder.parent))
    svc.load_model(str(folder), None, "cpu")
    assert svc.architecture == "kegetar" and svc.loaded_model_name == folder.name
    svc.close()


def test_what_is_refused(models, tmp_path, monkeypatch):
    folder, cfg, w = models("plain")
    for kw in (dict(tp_rank=0, tp_size=2), dict(pp_rank=0, pp_size=2), dict(ep_rank=0, ep_size=2)):
        with pytest.raises(ValueError):
            ModelBase.create(str(folder), "cpu", **kw)
    monkeypatch.setenv("TSB_KV_DTYPE", "fp8")
    with pytest.raises(ValueError):
        ModelBase.create(str(folder), "cpu")
    monkeypatch.delenv("TSB_KV_DTYPE")
    m = load(folder, "cpu")
    m.forward([1, 2, 3])
    with pytest.raises(RuntimeError):
        m.truncate_kv_cache(1)                             # the state cannot go back
    bad = tmp_path / "bad"
    synth.write_kegetar(str(bad), device="cpu", layers="pa", mlps="md")
    c = json.loads((bad / "config.json").read_text())
    first, second = c["layers"]
    left, router = first["mixer"]["left"], first["mlp"]["router"]
    for change in ({"type": "convolution"}, {"mlp": {**first["mlp"], "kind": "sparse"}}, {"mixer": {**first["mixer"], "left": {**left, "heads": 5}}},
                   {"mixer": {**first["mixer"], "left": {**left, "rot": {**left["rot"], "dims": 34}}}},
                   {"mlp": {**first["mlp"], "router": {**router, "groups": {"count": 3, "keep": 1}}}},
                   {"mlp": {**first["mlp"], "router": {**router, "identity": 3, "groups": {"count": 3, "keep": 2}}}},
                   {"mlp": {**first["mlp"], "router": {**router, "top": 7}}}):
        (bad / "config.json").write_text(json.dumps({**c, "layers": [{**first, **change}, second]}))
        with pytest.raises(ValueError):
            ModelBase.create(str(bad), "cpu")
    for extra in ({**first, "weights_of": 2}, {**first, "weights_of": 1}, {**first, "weights_of": 5}, {**first, "mlp": None, "weights_of": 0}):
        (bad / "config.json").write_text(json.dumps({**c, "layers": [first, second, extra]}))
        with pytest.raises(ValueError):
            ModelBase.create(str(bad), "cpu")
    (bad / "config.json").write_text(json.dumps({**c, "layers": [first, second, first]}))
    with pytest.raises(KeyError):
        ModelBase.create(str(bad), "cpu")                  # no tensors of a third layer
    c["embedding"]["bigram"]["buckets"] += 1
    (bad / "config.json").write_text(json.dumps(c))
    with pytest.raises(ValueError):
        ModelBase.create(str(bad), "cpu")
