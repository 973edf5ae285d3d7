"""Lisorax against the plain implementation of lisorax_oracle.py, on the CPU ops and (``-m gpu``) on the device in float32 and
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
import lisorax_oracle as O  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
PLACES = ["cpu", pytest.param("f32", marks=gpu), pytest.param("bf16", marks=gpu)]

CONFIGS = {
    "plain": dict(),
    # odd sizes everywhere, layers without a feed-forward, two layers that read the keys and values of the first
    "odd": dict(layers="armaa", mlps="m-mm-", width=100, heads=6, kv_heads=2, dim=20, vdim=28, conv=5, q_temp=(0.9, 7), softcap=4.0, scale=0.4,
                kv_from={3: 0, 4: 0}, rec_width=84, blocks=7, rec_conv=2, mem_heads=5, mem_dim=20, mem_vdim=28, gate_cap=3.0, canon=4, experts=7, top=4,
                expert_ff=20, embed_scale=1.3, vocab=333),
    # one of everything: taps of one token, one head, one block, one expert, no temperature, no cap
    "one": dict(layers="mra", mlps="mmm", heads=1, kv_heads=1, dim=16, vdim=16, conv=1, q_temp=None, softcap=None, blocks=1, rec_width=24, rec_conv=1,
                mem_heads=1, mem_dim=8, mem_vdim=8, gate_cap=30.0, canon=1, experts=1, top=1, expert_ff=8, embed_scale=1.0),
    "wide": dict(layers="ram", mlps="mm-", width=264, heads=20, kv_heads=4, dim=72, vdim=40, conv=8, q_temp=(0.2, 1000), softcap=50.0, blocks=3, rec_width=408,
                 rec_conv=8, mem_heads=2, mem_dim=130, mem_vdim=160, canon=8, experts=40, top=20, expert_ff=56, vocab=1031, eps=1e-3),
    "memory": dict(layers="mm", mlps="--", width=72, mem_heads=4, mem_dim=96, mem_vdim=64, gate_cap=6.0, canon=2),
    "units": dict(layers="rr", mlps="m-", width=48, rec_width=160, blocks=2, rec_conv=5, canon=5),
    "far": dict(layers="aam", mlps="mmm", heads=3, kv_heads=3, dim=40, vdim=56, conv=3, q_temp=(1.5, 64), softcap=15.0, kv_from={1: 0}, mem_vdim=32, canon=2),
}


def unequal():
    """No two layers alike: sizes, taps, temperatures, caps and feed-forwards differ from layer to layer."""
    c = synth.lisorax_config(layers="aramarm", mlps="mm-mmmm", width=96, eps=1e-4, kv_from={4: 2})
    a, b, d, e, f, g, h = (x["mixer"] for x in c["layers"])
    a.update(heads=5, kv_heads=5, dim=24, vdim=40, scale=0.3, conv=2, softcap=3.0, q_temp={"coef": 2.0, "every": 3})
    b.update(width=40, blocks=5, conv=7)
    d.update(heads=6, kv_heads=2, dim=16, vdim=64, conv=6, softcap=60.0)
    d.pop("q_temp")
    e.update(heads=2, dim=64, vdim=16, gate_cap=2.0)
    f.update(heads=8, kv_heads=2, dim=16, vdim=64, conv=3, scale=0.5, q_temp={"coef": 0.1, "every": 1})
    g.update(width=200, blocks=1, conv=1)
    h.update(heads=7, dim=16, vdim=80, gate_cap=15.0)
    c["layers"][0]["mlp"].update(expert={"ff": 56}, router={"experts": 9, "top": 3})
    c["layers"][5]["mlp"].update(expert={"ff": 8}, router={"experts": 3, "top": 3})
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


def errors(got, want):
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def agree(got, want, place):
    """Logit rows against the oracle's: to rounding in float32; in bfloat16 to what rounding the inputs of all products to
    16 bits does to these models.  A few rows may be off by more: an expert whose choice is close may come or go, and the norm
    of a memory's output makes much of rounding where that output is near zero."""
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
            folder = tmp_path_factory.mktemp("lisorax") / name
            synth.write_lisorax(str(folder), seed=len(name), device="cpu", **CONFIGS[name])
            made[name] = (folder,) + O.read_model(folder)
        return made[name]
    return get


_whole = {}


def oracle(name, cfg, w, ids):
    """The oracle's logits; memoised, several tests ask for the same sequence."""
    key = (name, tuple(ids))
    if key not in _whole:
        _whole[key] = O.forward(w, cfg, ids)
    return _whole[key]


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def qweight(w, dev):
    t = GGMLType.BF16 if w.dtype == torch.bfloat16 else GGMLType.F32
    return QuantWeight.from_raw(w.contiguous().view(-1).view(torch.uint8), t, tuple(w.shape), dev, "w")


def portions(kv, seqs, cuts, p):
    """Batch of the p-th portion of every sequence that has one: (batch, [(sequence, from, to)])."""
    part = [(b, c[p], c[p + 1]) for b, c in enumerate(cuts) if c[p + 1] > c[p]]
    return kv.build_batch([seqs[b] for b, _, _ in part], [[0] * (hi - lo) for _, lo, hi in part]), part


def padded(t, n, dev):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1])).to(dev).contiguous()


def pad_heads(v, H, n, D):
    return torch.nn.functional.pad(v.view(*v.shape[:-1], H, n), (0, D - n)).reshape(*v.shape[:-1], H * D)


def carried(slots, shape, dev):
    """A per-slot state as a model has it: a view into wider rows, full of NaN."""
    n = torch.Size(shape).numel()
    return torch.full((slots, 28 + (n + 3) // 4 * 4), float("nan"), device=dev)[:, 28:28 + n].unflatten(1, shape)


# ------------------------------------------------------------------------------------------ mechanisms alone
def test_how_far_a_convolution_reaches():
    """The oracle itself: an impulse comes back with the taps from last to first, and not before it."""
    u = torch.zeros(9, 2)
    u[3] = 1.0
    w = torch.tensor([[1.0, 2.0, 3.0], [4.0, 5.0, 6.0]])
    out = O.over_time(u, w)
    assert out[:3].abs().sum() == 0 and out[3].tolist() == [3.0, 6.0] and out[5].tolist() == [1.0, 4.0] and out[6:].abs().sum() == 0


CUTS = [[0, 1, 2, 3, 70, 72, 290, 291, 292], [0, 0, 2, 4, 4, 9, 9, 10, 10], [0, 3, 3, 40, 41, 41, 139, 139, 140]]
LENS = [c[-1] for c in CUTS]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("n,K", [(40, 1), (61, 3), (250, 8), (1100, 4), (2050, 2), (5003, 4), (8200, 5)])
def test_seam_in_portions(place, n, K):
    """Residual, expert rows in any order, norm, and the convolution carried from portion to portion (shorter than the taps, too),
    on a slot that was used before."""
    dev, dt, D, eps, k = device(place), dtype(place), (n + 7) // 8 * 8, 1e-4, 3
    g = torch.Generator().manual_seed(n)
    w, taps = 1 + 0.3 * torch.randn(n, generator=g), torch.randn(n, K, generator=g) * 0.5
    h0 = [torch.randn(m, n, generator=g) * 2 for m in LENS]
    y0 = [(torch.randn(m, n, generator=g) * 0.4).to(dt) for m in LENS]
    p0 = [torch.randn(m * k, n, generator=g).to(dt) for m in LENS]
    c0 = [torch.rand(m, k, generator=g) for m in LENS]
    sums = [h.double() + y.double() + (p.double().view(-1, k, n) * c.double().unsqueeze(-1)).sum(1) for h, y, p, c in zip(h0, y0, p0, c0)]
    norms = [O.rms(s, eps) * w for s in sums]
    convs = [v + O.over_time(v, taps.double()) for v in norms]
    first = [O.rms(h.double(), eps) * w for h in h0]
    kv, state = PagedKV([None], 60, 16, dev, max_seqs=3), carried(3, (K - 1, D), dev)
    wd, td = padded(w, D, dev), padded(taps.t().contiguous(), D, dev)
    tol = dict(rtol=1e-2, atol=2e-2) if place == "bf16" else dict(rtol=1e-5, atol=5e-5)
    for again in range(2):
        seqs = [kv.new_seq() for _ in LENS]
        for s in seqs:
            state[s.slot] = 0
        for p in range(8):
            batch, part = portions(kv, seqs, CUTS, p)

            def rows(x, m=1):
                return torch.cat([x[b][lo * m:hi * m] for b, lo, hi in part])
            h, T = padded(rows(h0), D, dev), batch.T
            before = h.clone()
            pr = rows(p0, k)
            if place == "cpu":
                parts = F.MoeParts(padded(pr, D, dev), k, None, rows(c0).view(-1))
            else:
                order = torch.randperm(T * k, generator=g)
                pos = torch.empty(T * k, dtype=torch.int32)
                pos[order] = torch.arange(T * k, dtype=torch.int32)
                parts = F.MoeParts(padded(pr[order], D, dev), k, pos.to(dev), rows(c0).view(-1).to(dev))
            out, v, c = F.conv_seam(h, eps, n, w=wd, y=padded(rows(y0), D, dev), parts=parts, taps=td, state=state, batch=batch, plain=again == 0, dtype=dt)
            assert torch.equal(h, before)
            assert torch.allclose(out[:, :n].double().cpu(), rows(sums), rtol=1e-5, atol=5e-5)
            assert torch.allclose(c[:, :n].double().cpu(), rows(convs), **tol) and not c[:, n:].any() and not out[:, n:].any()
            assert (v is None) == (again == 1) and (v is None or torch.allclose(v[:, :n].double().cpu(), rows(norms), **tol))
            out, v, c = F.conv_seam(h, eps, n, w=wd, dtype=dt)                  # the last seam: nothing to add, no convolution
            assert out is h and c is None and torch.allclose(v[:, :n].double().cpu(), rows(first), **tol)
        for b, s in enumerate(seqs):
            if K > 1:
                assert torch.allclose(state[s.slot][:, :n].double().cpu(), norms[b][-(K - 1):], rtol=1e-5, atol=5e-5)
            kv.free_seq(s)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("C,K,block,bias", [(40, 3, 0, True), (24, 1, 8, False), (1040, 4, 16, True), (72, 8, 24, False), (640, 2, 0, False)])
def test_short_convolution_in_portions(place, C, K, block, bias):
    dev, dt = device(place), dtype(place)
    g = torch.Generator().manual_seed(C)
    w, b0 = torch.randn(C, K, generator=g), torch.randn(C, generator=g) if bias else None
    x0 = [torch.randn(m, C, generator=g).to(dt) for m in LENS]
    want = [O.over_time(x.double(), w.double(), b0.double() if bias else None) for x in x0]
    kv, state = PagedKV([None], 60, 16, dev, max_seqs=3), carried(3, (K - 1, C), dev)
    for again in range(2):
        seqs = [kv.new_seq() for _ in LENS]
        for s in seqs:
            state[s.slot] = 0
        for p in range(8):
            batch, part = portions(kv, seqs, CUTS, p)
            x = torch.cat([x0[b][lo:hi] for b, lo, hi in part])
            if batch.T <= F.GEMV_MAX_M:
                x = x.float()
            x = torch.nn.functional.pad(x, (8, 8)).to(dev)[:, 8:-8]                # a row stride of its own
            o = F.short_conv(x, w.t().contiguous().to(dev), b0.to(dev) if bias else None, state, batch, block=block, dtype=dt).double().cpu()
            if block:
                assert o.shape == (C // block * batch.T, block)
                o = o.view(C // block, batch.T, block).transpose(0, 1).reshape(batch.T, C)
            ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
            assert torch.allclose(o, ref, **(dict(rtol=1e-2, atol=2e-2) if place == "bf16" else dict(rtol=1e-5, atol=3e-5)))
        for s in seqs:
            kv.free_seq(s)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,D,E,K,temp,own", [(4, 2, 16, 32, 4, (0.5, 10), True), (3, 3, 48, 16, 1, None, True), (8, 1, 32, 96, 3, (1.0, 1), True),
                                                (6, 2, 16, 16, 8, (0.25, 64), False), (5, 1, 80, 16, 2, None, False)])
def test_convolved_projections_and_their_cache(place, H, G, D, E, K, temp, own):
    """Queries with their temperature, keys and values in their slots; queries alone for a layer that reads another's cache."""
    dev, dt = device(place), dtype(place)
    g = torch.Generator().manual_seed(D)
    nq, C = H * D, H * D + (G * (D + E) if own else 0)
    w = torch.randn(C, K, generator=g)
    x0 = [torch.randn(m, C, generator=g).to(dt) for m in LENS]
    full = [O.over_time(x.double(), w.double()) for x in x0]
    kv, state = PagedKV([(G, D, E)], 60, 16, dev, dt, max_seqs=3), carried(3, (K - 1, C), dev)
    tol = dict(rtol=1e-2, atol=2e-2) if place == "bf16" else dict(rtol=1e-5, atol=5e-5)
    seqs = [kv.new_seq() for _ in LENS]
    for s in seqs:
        state[s.slot] = 0
    for p in range(8):
        batch, part = portions(kv, seqs, CUTS, p)
        x = torch.cat([x0[b][lo:hi] for b, lo, hi in part]).to(dev)
        x = x.float() if batch.T <= F.GEMV_MAX_M else x
        kw = dict(k_cache=kv.k[0], v_cache=kv.v[0]) if own else {}
        q = F.conv_qkv_cache(x, w.t().contiguous().to(dev), state, batch, nq=nq, dtype=dt, q_temp=temp, **kw)
        ref = torch.cat([full[b][lo:hi] for b, lo, hi in part])
        at = torch.cat([torch.arange(lo, hi) for _, lo, hi in part]).double()
        factor = O.temperature(at, *temp)[:, None] if temp else 1.0
        assert q.dtype == dt and torch.allclose(q.double().cpu(), ref[:, :nq] * factor, **tol)
        if own:
            assert torch.allclose(kv.k[0][batch.slots].double().cpu().flatten(1), ref[:, nq:nq + G * D], **tol)
            assert torch.allclose(kv.v[0][batch.slots].double().cpu().flatten(1), ref[:, nq + G * D:], **tol)
        else:
            assert not kv.k[0].any() and not kv.v[0].any()


ATTENTION = [  # H, G, dim, vdim, cap, distance bias, sigmoid weights
    (4, 2, 32, 48, 12.0, True, True), (6, 2, 20, 28, 0.0, True, True), (3, 3, 64, 64, 50.0, False, True), (20, 1, 48, 80, 8.0, True, True),
    (2, 1, 128, 128, 30.0, True, True), (5, 5, 16, 16, 0.0, False, True), (40, 2, 72, 72, 5.0, True, True), (2, 2, 256, 256, 20.0, True, True),
    (4, 2, 40, 24, 10.0, True, False), (33, 1, 16, 112, 0.0, True, False)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,dim,vdim,cap,bias,sig", ATTENTION)
def test_attention_with_keys_that_stand_out(place, H, G, dim, vdim, cap, bias, sig):
    """Single keys stand out from all others for one query each: far away, at page borders, the first ones, the query's own and the
    one ahead of it (which must not show); on pages in no order, in portions and decoding, over poisoned free rows.  Sigmoid weights are not
    normalised, and a softmax with the same distance bias is."""
    dev, dt, page = device(place), dtype(place), 16
    g = torch.Generator().manual_seed(H * dim)
    Dk, Dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    lens = [150, 33, 209]
    kv = PagedKV([(G, Dk, Dv)], 40, page, dev, dt, max_seqs=3)
    kv._free = torch.randperm(40, generator=g).tolist()
    kv.k[0].fill_(float("nan"))
    kv.v[0].fill_(float("nan"))
    seqs = [kv.new_seq() for _ in lens]
    r1, r2 = torch.rand(H, generator=g) * 1.5, torch.rand(H, generator=g) * 0.4
    if not bias:
        r1 = torch.zeros(H)
    pb = -3.0 - torch.rand(H, generator=g)
    data, want = [], []
    for n in lens:
        q, k, v = (torch.randn(n, a, d, generator=g) * s for a, d, s in ((H, dim, 0.3), (G, dim, 0.3), (G, vdim, 1.0)))
        pairs = []
        for i in (n - 1, n - 2, n // 2, page, 2 * page - 1):
            pairs += [(i, j) for j in (0, 1, i - 1, i, i + 1, page - 1, page, n // 3) if 0 <= j < n and i < n]
        marks = max(1, min(dim // 2, 8))                      # columns that only a marked key uses
        k[..., :marks] = 0
        q[..., :marks] = 0
        for m, (i, j) in enumerate(pairs[::max(1, len(pairs) // marks)][:marks]):
            k[j, :, m], q[i, :, m] = 3.0, 8.0
        q, k, v = (t.to(dt) for t in (q, k, v))
        data.append((q, k, v))
        qd, kd, vd = q.double(), k.double(), v.double()
        if sig:
            want.append(O.attend(qd, kd, vd, 0.4, cap, r1.double(), r2.double(), pb.double()))
        else:
            big = -30.0                                       # sigmoid(s + big) is e^(s + big): their sums make the softmax
            o = O.attend(qd, kd, torch.cat([vd, torch.ones_like(vd[..., :1])], -1), 0.4, cap, r1.double(), r2.double(), torch.full((H,), big).double())
            want.append(o[..., :-1] / o[..., -1:])
    cuts = [[0, 2, 17, 64, 148, 149, 150], [0, 16, 31, 32, 32, 32, 33], [0, 1, 130, 193, 207, 208, 209]]      # the last two: decoding
    for p in range(6):
        batch, part = portions(kv, seqs, cuts, p)
        assert batch.is_decode == (p >= 4)

        def rows(x):
            return torch.cat([data[b][x][lo:hi] for b, lo, hi in part])
        kv.k[0][batch.slots], kv.v[0][batch.slots] = padded(rows(1), Dk, dev), padded(rows(2), Dv, dev)
        out = F.attention(padded(rows(0), Dk, dev), kv.k[0], kv.v[0], batch, scale=0.4, Hq=H, Hkv=G, Dh=Dk, Dv=Dv, softcap=cap,
                          log_bias=(r1.to(dev), r2.to(dev)) if bias else None, sigmoid_bias=pb.to(dev) if sig else None).view(batch.T, H, Dv)
        ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
        err = (out[..., :vdim].double().cpu() - ref).abs().max()
        assert err < (0.04 if place == "bf16" else 1e-4), (p, err)
        assert not out[..., vdim:].any()


def test_what_a_key_weighs():
    """The oracle itself: a key that the query asks for is found however far away it is, its distance costs r1 ln(1 + r2 d), and two
    such keys count twice."""
    T = 40
    q, k = torch.zeros(T, 2, dtype=torch.float64), torch.zeros(T, 2, dtype=torch.float64)
    q[30, 0], k[5, 0], k[33, 0] = 4.0, 2.0, 2.0
    one, none = torch.tensor(0.7, dtype=torch.float64), torch.tensor(0.0, dtype=torch.float64)
    r2, pb = torch.tensor(0.3, dtype=torch.float64), torch.tensor(-1.0, dtype=torch.float64)
    w = O.key_weights(q, k, 0.5, None, one, r2, pb)
    assert torch.allclose(w[30, 5], O.sigmoid(4.0 - 0.7 * torch.log(1 + r2 * 25) - 1.0))
    assert w[30, 33] == 0 and w[5, 30] == 0
    before = O.key_weights(q, k, 0.5, None, none, r2, pb)[30].sum()
    k[6, 0] = 2.0
    assert torch.allclose(O.key_weights(q, k, 0.5, None, none, r2, pb)[30].sum() - before, O.sigmoid(torch.tensor(3.0)).double() - O.sigmoid(pb))


UNITS = [(40, 5, 2), (24, 1, 4), (96, 3, 1), (408, 3, 8), (512, 4, 3), (200, 25, 4), (640, 2, 4), (1600, 1, 2)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("width,blocks,K", UNITS)
def test_gated_recurrence_in_portions(place, width, blocks, K):
    """Convolution, gates per block and recurrence: the step kernel and the scan in turns, unequal sequences, a slot that is given
    back and used again.  Some channels forget next to nothing, others all at once."""
    dev, dt = device(place), dtype(place)
    s = F.RglruSpec(width, blocks)
    n, B, W = s.size, s.block, s.W
    g = torch.Generator().manual_seed(width)
    y0 = [torch.randn(m, width, generator=g).to(dt) for m in LENS]
    x0 = [torch.randn(m, width, generator=g).to(dt) for m in LENS]
    cw, cb = torch.randn(width, K, generator=g) * 0.5, torch.randn(width, generator=g) * 0.1
    ra, ri = (torch.randn(blocks, n, n, generator=g).div(n ** 0.5).to(dt) for _ in range(2))
    rb, ib = torch.randn(blocks, n, generator=g) * 3, torch.randn(blocks, n, generator=g)
    lam = torch.rand(width, generator=g) * 8 - 6
    rb.view(-1)[::4] -= 8
    lam[::4] -= 2
    rb.view(-1)[1::4] += 9
    lam[1::4] += 9
    want = []
    for y, x in zip(y0, x0):
        u = O.over_time(x.double(), cw.double(), cb.double())
        r, i = (O.sigmoid(O.per_block(u, m.double(), b.double())) for m, b in ((ra, rb), (ri, ib)))
        S, last = O.gated_recurrence(u, r, i, lam.double())
        want.append((S * O.gelu(y.double()), last))
    gates = qweight(torch.cat([torch.nn.functional.pad(m, (0, B - n, 0, B - n)) for m in (ra, ri)], 1), dev)
    gate_b = torch.stack([pad_heads(b.view(-1), blocks, n, B) for b in (rb, ib)]).to(dev)
    rate = pad_heads(-8 * O.softplus(lam.double()), blocks, n, B).float().to(dev)
    cwd, cbd = pad_heads(cw.t().contiguous(), blocks, n, B).contiguous().to(dev), pad_heads(cb, blocks, n, B).to(dev)
    kv, cs, st = PagedKV([None], 60, 16, dev, max_seqs=3), carried(3, (K - 1, W), dev), carried(3, (W,), dev)
    for again in range(2):
        seqs = [kv.new_seq() for _ in LENS]
        for q in seqs:
            cs[q.slot], st[q.slot] = 0, 0
        for p in range(8):
            batch, part = portions(kv, seqs, CUTS, p)
            y = torch.cat([torch.cat([pad_heads(y0[b][lo:hi], blocks, n, B), pad_heads(x0[b][lo:hi], blocks, n, B)], 1) for b, lo, hi in part])
            y = torch.nn.functional.pad(y.float() if batch.T <= F.GEMV_MAX_M else y, (0, 8)).to(dev)[:, :-8]
            out = F.rglru(y, s, cwd, cbd, gates, gate_b, rate, cs, st, batch, dtype=dt)
            got = out.double().cpu().view(-1, blocks, B)
            ref = torch.cat([want[b][0][lo:hi] for b, lo, hi in part]).view(-1, blocks, n)
            err = (got[..., :n] - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
            assert err < (0.01 if place == "bf16" else 1e-5), (p, err)
            assert not got[..., n:].any()
        for b, q in enumerate(seqs):
            left = st[q.slot].view(blocks, B)[:, :n].reshape(-1).double().cpu()
            assert torch.allclose(left, want[b][1], **(dict(rtol=0.05, atol=0.05) if place == "bf16" else dict(rtol=1e-4, atol=2e-5)))
            kv.free_seq(q)


@gpu
@pytest.mark.parametrize("segs", [1, 2, 7])
def test_recurrence_scan_keeps_32_bits(segs):
    """The scan in segments from given gate products: states and outputs to 32-bit rounding; sequences longer and shorter than a
    segment, states that are not zero, channels whose decay is within 1e-6 of 1."""
    from tensorsharp_b200.ops import kernels as K
    s = F.RglruSpec(60, 3)
    g = torch.Generator().manual_seed(segs)
    lens = [1, 300, 17, 64]
    T, W, n, B = sum(lens), s.W, s.size, s.block
    u, z = torch.randn(T, 60, generator=g), torch.randn(2, T, 60, generator=g) * 3
    y = torch.randn(T, W, generator=g)
    bias, lam = torch.randn(2, 60, generator=g), torch.rand(60, generator=g) * 8 - 6
    bias[0, ::3] -= 12
    s0 = torch.randn(5, 60, generator=g)
    kv = PagedKV([None], 60, 16, "cuda", max_seqs=5)
    seqs = [kv.new_seq() for _ in lens]
    batch = kv.build_batch(seqs, [[0] * m for m in lens])
    st = carried(5, (W,), "cuda")
    st.copy_(pad_heads(s0, 3, n, B))

    def blocked(t):
        return pad_heads(t, 3, n, B).view(T, 3, B).transpose(0, 1).reshape(3 * T, B)
    out = K.rglru_scan(y.cuda(), blocked(u).contiguous().cuda(), torch.cat([blocked(z[0]), blocked(z[1])], 1).contiguous().cuda(), s,
                       pad_heads(bias, 3, n, B).contiguous().cuda(), pad_heads(-8 * O.softplus(lam.double()), 3, n, B).float().cuda(), st, batch,
                       out_dtype=torch.float32, segs=segs).double().cpu().view(T, 3, B)
    r, i = (O.sigmoid(z[x].double() + bias[x].double()) for x in (0, 1))
    at = 0
    for q, m in zip(seqs, lens):
        S, last = O.gated_recurrence(u[at:at + m].double(), r[at:at + m], i[at:at + m], lam.double(), s0[q.slot].double())
        want = S.view(m, 3, n) * O.gelu(y[at:at + m].double()).view(m, 3, B)[..., :n]
        assert torch.allclose(out[at:at + m, :, :n], want, rtol=1e-5, atol=1e-5)
        assert torch.allclose(st[q.slot].double().cpu().view(3, B)[:, :n].reshape(-1), last, rtol=1e-5, atol=1e-5)
        at += m
    assert not out[..., n:].any()
    spare = ({0, 1, 2, 3, 4} - {q.slot for q in seqs}).pop()
    assert torch.equal(st[spare].cpu().view(3, B)[:, :n].reshape(-1), s0[spare])                                # nobody's slot


MEMORY = [(3, 20, 28), (2, 64, 16), (5, 96, 33), (4, 128, 128), (1, 150, 100), (2, 256, 160), (20, 32, 8), (1, 200, 256)]


def memory_inputs(H, n, e, T, g, dt):
    q, k, v, gate = (torch.randn(T, H * d, generator=g).to(dt) for d in (n, n, e, e))
    z = torch.randn(T, 2 * H, generator=g) * 3
    zb = torch.randn(2 * H, generator=g) * 2
    zb[H:] += 3
    zb[H::3] += 12                                            # heads that keep next to everything
    zb[H + 1::3] -= 25                                        # and heads that forget at once
    return q, k, v, gate, z, zb


def memory_wants(q, k, v, gate, z, zb, H, n, cap, on, eps, state=None):
    """(result, last state, the memory's output ahead of its norm)."""
    T = q.shape[0]
    z = O.capped(z.double() + zb.double(), cap)
    o, last = O.matrix_memory(q.double().view(T, H, n) * n ** -0.5, k.double().view(T, H, n), v.double().view(T, H, -1), z[:, :H], -O.softplus(-z[:, H:]), state)
    return O.rms(o, eps) * on.double().view(H, -1) * O.sigmoid(gate.double()).view(T, H, -1), last, o


def memory_views(rows, H, E, D):
    return rows[:, :H * E * D].unflatten(1, (H, E, D)), rows[:, H * E * D:H * (E + 1) * D].unflatten(1, (H, D)), rows[:, H * (E + 1) * D:H * (E + 1) * D + H]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,n,e", MEMORY)
def test_matrix_memory_in_portions(place, H, n, e):
    """Gates, recurrence, norm and output gate: single steps and chunk kernels in turns, unequal sequences, a slot that is given
    back and used again."""
    dev, eps, dt, cap = device(place), 1e-4, dtype(place), 8.0
    s = F.MlstmSpec(H, n, e, cap)
    D, E = s.D, s.E
    g = torch.Generator().manual_seed(H * n)
    x = [memory_inputs(H, n, e, m, g, dt) for m in LENS]
    zb, on = x[0][5], torch.randn(H * e, generator=g)
    want = [memory_wants(*a[:5], zb, H, n, cap, on, eps)[0] for a in x]
    kv = PagedKV([None], 60, 16, dev, max_seqs=3)
    rows = torch.full((3, 28 + H * (E + 1) * D + (H + 3) // 4 * 4), float("nan"), device=dev)[:, 28:]
    S, N, M = memory_views(rows, H, E, D)
    cols = (0, H * D, 2 * H * D, 2 * H * D + H * E)
    for again in range(2):
        seqs = [kv.new_seq() for _ in LENS]
        for q in seqs:
            rows[q.slot] = 0
        for p in range(8):
            batch, part = portions(kv, seqs, CUTS, p)

            def take(i):
                return torch.cat([x[b][i][lo:hi] for b, lo, hi in part])
            y = torch.cat([pad_heads(take(0), H, n, D), pad_heads(take(1), H, n, D), pad_heads(take(2), H, e, E), pad_heads(take(3), H, e, E)], 1)
            y = torch.nn.functional.pad(y.float() if batch.T <= F.GEMV_MAX_M else y, (0, 8)).to(dev)[:, :-8]                # a row stride of its own
            z = torch.nn.functional.pad(take(4), (0, 3)).to(dev)[:, :-3]
            out = F.mlstm(y, s, cols, z, zb.to(dev), pad_heads(on, H, e, E).to(dev), S, N, M, batch, eps=eps, dtype=dt)
            got = out.double().cpu().view(-1, H, E)
            ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
            err = (got[..., :e] - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
            assert err < (0.01 if place == "bf16" else 5e-5), (p, err)
            assert not got[..., e:].any()
        for q in seqs:
            kv.free_seq(q)


@gpu
@pytest.mark.parametrize("H,n,e", MEMORY)
@pytest.mark.parametrize("segs", [1, 2, 4])
def test_matrix_memory_chunk_kernel_keeps_32_bits(H, n, e, segs):
    """The tensor-core path from bf16 rows: memory, normaliser and maximum against the oracle's to 32-bit rounding, and the results
    to one rounding of the output; unequal sequences, full and short chunks and segments, states that are not zero."""
    from tensorsharp_b200.ops import kernels as K
    cap, eps = 12.0, 1e-5
    s = F.MlstmSpec(H, n, e, cap)
    D, E = s.D, s.E
    g = torch.Generator().manual_seed(n)
    lens = [1, 203, 64, 16, 65]
    T = sum(lens)
    q, k, v, gate, z, zb = memory_inputs(H, n, e, T, g, torch.bfloat16)
    on = torch.randn(H * e, generator=g)
    kv = PagedKV([None], 60, 16, "cuda", max_seqs=6)
    seqs = [kv.new_seq() for _ in lens]
    batch = kv.build_batch(seqs, [[0] * m for m in lens])
    s0, n0, m0 = torch.randn(6, H, e, n, generator=g), torch.randn(6, H, n, generator=g), torch.randn(6, H, generator=g)
    start = torch.zeros(6, H * (E + 1) * D + (H + 3) // 4 * 4)
    S, N, M = memory_views(start, H, E, D)
    S[:, :, :e, :n], N[:, :, :n], M[:] = s0, n0, m0
    rows = start.cuda()
    S, N, M = memory_views(rows, H, E, D)
    y = torch.cat([pad_heads(q, H, n, D), pad_heads(k, H, n, D), pad_heads(v, H, e, E), pad_heads(gate, H, e, E)], 1).cuda()
    out = K.mlstm_prompt(y, s, (0, H * D, 2 * H * D, 2 * H * D + H * E), z.cuda(), zb.cuda(), pad_heads(on, H, e, E).cuda(), S, N, M, batch, eps=eps,
                         out_dtype=torch.bfloat16, segs=segs).double().cpu().view(T, H, E)
    at = 0
    for sq, m in zip(seqs, lens):
        b, part = sq.slot, [t[at:at + m] for t in (q, k, v, gate, z)]
        want, (S1, n1, m1), _ = memory_wants(*part, zb, H, n, cap, on, eps, (s0[b].double().transpose(1, 2), n0[b].double(), m0[b].double()))
        got = S[b].double().cpu()[:, :e, :n].transpose(1, 2)
        assert torch.allclose(M[b].double().cpu(), m1, rtol=1e-5, atol=1e-5)
        for x, ref in ((got, S1), (N[b].double().cpu()[:, :n], n1)):
            size = ref.abs().amax(tuple(range(1, ref.dim())), keepdim=True)        # per head
            assert ((x - ref).abs() <= 3e-5 * size + 1e-6).all(), (b, ((x - ref).abs() / size).max())
        err = (out[at:at + m, :, :e] - want).abs()
        assert (err <= 0.01 * want.abs() + 2e-3 * want.pow(2).mean((1, 2), keepdim=True).sqrt()).double().mean() > 0.999, (b, err.max())
        assert not out[at:at + m, :, e:].any() and not S[b, :, e:].any() and not S[b, :, :, n:].any() and not N[b, :, n:].any()
        at += m
    spare = ({0, 1, 2, 3, 4, 5} - {q.slot for q in seqs}).pop()
    assert torch.equal(rows[spare].cpu(), start[spare])                                # nobody's slot


def test_what_the_memory_keeps():
    """The oracle itself: with an open forget gate a value comes back for its key however far away; with a closed one only the newest
    does; and a query that finds little is not blown up (the denominator is at least e^-m)."""
    D = 16
    g = torch.Generator().manual_seed(0)
    k = torch.eye(D, dtype=torch.float64)[:, None]
    v = torch.randn(D, 1, 5, generator=g, dtype=torch.float64)
    q = torch.zeros(D, 1, D, dtype=torch.float64)
    q[D - 1, 0, 3] = 1
    zero = torch.zeros(D, 1, dtype=torch.float64)
    assert torch.allclose(O.matrix_memory(q, k, v, zero, zero)[0][-1, 0], v[3, 0], rtol=1e-5)
    assert O.matrix_memory(q, k, v, zero, zero - 1e3)[0][-1, 0].abs().max() < 1e-5
    q[D - 1, 0] = torch.eye(D)[D - 1]
    assert torch.allclose(O.matrix_memory(q, k, v, zero, zero - 1e3)[0][-1, 0], v[-1, 0], rtol=1e-5)
    assert torch.allclose(O.matrix_memory(q, k * 1e-3, v, zero, zero)[0][-1, 0], v[-1, 0] * 1e-3, rtol=1e-5)


@pytest.mark.parametrize("place", ["cpu", pytest.param("f32", marks=gpu)])
@pytest.mark.parametrize("E,top", [(1, 1), (6, 2), (12, 12), (40, 20), (900, 32)])
def test_routing(place, E, top):
    z = torch.randn(33, E, generator=torch.Generator().manual_seed(E)) * 3
    ids, w = F.route_topk_softmax(z.to(device(place)), top)
    for t in range(33):
        want = O.choose(z[t].double(), top)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double().cpu(), torch.stack([x for _, x in want]), rtol=1e-5, atol=1e-9)


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_against_the_oracle(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    got, want = [], []
    for n in (1, 2, 9, 77, 150):
        ids = tokens(n, cfg["vocab"], n)
        s = m.new_sequence()
        got.append(m.forward_batch(m.kv.build_batch([s], [ids], rows=[list(range(n))])))
        want.append(oracle(name, cfg, w, ids))
        m.free_sequence(s)
    agree(torch.cat(got), torch.cat(want), place)
    if place != "cpu":
        m.poll_status(force=True)


def test_layers_that_share_a_cache(models):
    """Layers without keys and values of their own have no such tensors and no cache, but a state of their own."""
    folder, cfg, w = models("odd")
    assert not any(n.startswith((f"l3.mix.{x}", f"l4.mix.{x}")) for n in w for x in ("k", "v")) and "l0.mix.k.conv" in w
    m = load(folder, "cpu")
    assert m.kv.k[3] is m.kv.k[0] and m.kv.v[4] is m.kv.v[0] and m.kv.k[1] is None and m.kv.k[2] is None
    assert m.kv.k[0].shape[1:] == (2, 32) and m.kv.v[0].shape[1:] == (2, 32)
    assert [tuple(c["conv"].shape[1:]) if "conv" in c else None for c in m.carried] == [(4, 6 * 32 + 2 * 64), (1, 7 * 16), None, (4, 192), (4, 192)]
    ends = sorted((t.data_ptr() - m.state.data_ptr(), t[0].numel() * 4) for c in m.carried for t in c.values())
    assert all(a + n <= b for (a, n), (b, _) in zip(ends, ends[1:])) and ends[-1][0] + ends[-1][1] <= m.state.shape[1] * 4


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "plain", "wide", "unequal"])
@pytest.mark.parametrize("cut", [[1], [2], [3, 2, 61], [64], [23, 1, 24, 2, 70]])
def test_portions_and_token_by_token(models, place, name, cut):
    """However a prompt is cut, its logits are the same."""
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    n = 150
    ids = tokens(n, cfg["vocab"], n)
    want = oracle(name, cfg, w, ids)
    n = 90 if cut == [1] else n
    eng, got, at, i = StepEngine(m, 4), [], 0, 0
    while at < n:
        k = min(cut[i % len(cut)], n - at)
        got.append(eng.step([("a", ids[at:at + k], list(range(k)))]))
        at, i = at + k, i + 1
    agree(torch.cat(got), want[:n], place)


PLAN = [[("a", 60), ("b", 2)], [("b", 61), ("a", 5)], [("a", 1), ("b", 1), ("c", 39)], [("c", 1), ("a", 1), ("d", 1)], [("a", 62)], [("a", 1)],
        [("e", 65), ("f", 3)], [("f", 1), ("e", 1)], [("f", 1)], [("e", 2), ("f", 64)], [("e", 121), ("f", 1)], [("e", 1)]]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "far", "plain"])
def test_batches_of_unequal_requests_on_pages_and_slots_used_before(models, place, name):
    """Portions beside single tokens, a request left out of steps, requests that end and others that take their pages and
    slots; the pool holds no page to spare."""
    folder, cfg, w = models(name)
    m = load(folder, place, max_context=320, kv_pages=5)
    poison(m)
    names = {"a": 130, "b": 64, "c": 40, "d": 1, "e": 190, "f": 70}
    ids = {k: tokens(n, cfg["vocab"], ord(k)) for k, n in names.items()}
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
        agree(torch.cat(got[k]), oracle(name, cfg, w, ids[k]), place)
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
@pytest.mark.parametrize("portion", [4, 5, 7])
def test_many_short_portions(models, place, portion):
    """More rows than the small-batch paths take, in portions shorter than the prompt kernels take."""
    folder, cfg, w = models("plain")
    m = load(folder, place, max_seqs=6)
    poison(m)
    ids = [tokens(21 + i, cfg["vocab"], i) for i in range(6)]
    eng, got = StepEngine(m, 6), [[] for _ in ids]
    for at in range(0, 27, portion):
        part = [(i, t[at:at + portion]) for i, t in enumerate(ids) if at < len(t)]
        out, row = eng.step([(i, t, list(range(len(t)))) for i, t in part]), 0
        for i, t in part:
            got[i].append(out[row:row + len(t)])
            row += len(t)
    agree(torch.cat([torch.cat(g) for g in got]), torch.cat([oracle("plain", cfg, w, t) for t in ids]), place)


@gpu
@pytest.mark.parametrize("place", ["f32", "bf16"])
def test_a_large_decode_batch(models, place):
    """More sequences than a CTA of the step kernels takes, on slots in no order, beside one another and one by one."""
    folder, cfg, w = models("plain")
    m = load(folder, place, max_seqs=20)
    ids = [tokens(14 + i, cfg["vocab"], i) for i in range(19)]
    eng = StepEngine(m, 20)
    for i in torch.randperm(19, generator=torch.Generator().manual_seed(0)).tolist():
        eng.step([(i, ids[i][:-3], [])])
    rows = [eng.step([(i, [ids[i][len(ids[i]) - 3 + t]], [0]) for i in range(19)]) for t in range(3)]
    assert eng.stepper.replays == 3
    agree(torch.cat([torch.stack([r[i] for r in rows]) for i in range(19)]), torch.cat([oracle("plain", cfg, w, ids[i])[-3:] for i in range(19)]), place)


@pytest.mark.parametrize("place", PLACES)
def test_a_pool_of_one_slot(models, place):
    """The single-sequence interface, prompt and steps, twice on the same slot."""
    folder, cfg, w = models("unequal")
    m = load(folder, place, max_seqs=1)
    poison(m)
    ids = tokens(50, cfg["vocab"], 11)
    m.forward(ids[:7])
    m.reset_kv_cache()
    got = [m.forward(ids[:30])] + [m.forward([t]) for t in ids[30:]]
    agree(torch.stack(got), oracle("unequal", cfg, w, ids)[29:], place)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["memory", "plain"])
def test_wanted_rows_only(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    ids = tokens(50, cfg["vocab"], 2)
    want = oracle(name, cfg, w, ids)
    eng = StepEngine(m, 4)
    assert eng.step([("a", ids[:20], [])]) is None
    agree(eng.step([("a", ids[20:45], [24, 0, 7])]), want[[44, 20, 27]], place)
    assert eng.step([("a", ids[45:46], [])]) is None
    assert eng.step([("a", ids[46:47], [0]), ("b", ids[:1], [])]).shape == (1, cfg["vocab"])
    agree(eng.step([("b", ids[1:2], [0]), ("a", ids[47:48], [0])]), want[[1, 47]], place)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["plain", "odd"])
def test_long_decoding(models, place, name):
    """Hundreds of single steps (captured graphs on the device) after a short prompt, over several pages."""
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    n = 300
    ids = tokens(n, cfg["vocab"], 8)
    want = oracle(name, cfg, w, ids)
    eng = StepEngine(m, 2)
    got = [eng.step([("a", ids[:3], [0, 1, 2])])] + [eng.step([("a", ids[i:i + 1], [0])]) for i in range(3, n)]
    if place != "cpu":
        assert eng.stepper.replays >= n - 4
    agree(torch.cat(got), want, place)


# ------------------------------------------------------------------------------------------ generation and entry points
def greedy_is_argmax(w, cfg, prompt, out, slack):
    """Every token is the oracle's best for what precedes it, up to ``slack`` standard deviations."""
    rows = oracle(id(w), cfg, w, prompt + out)[len(prompt) - 1:-1]
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
    reqs = eng.run([GenRequest(p, 16) for p in prompts])
    assert m.kv.free_pages == m.kv.n_pages
    for p, r in zip(prompts, reqs):
        assert r.error is None and len(r.ids) == 16
        greedy_is_argmax(w, cfg, p, r.ids, slack)
        m.reset_kv_cache()
        alone = generate(m, p, 16, prefill_chunk=16)
        greedy_is_argmax(w, cfg, p, alone, slack)
        if place != "bf16":
            assert alone == r.ids
    bad = eng.run([GenRequest([], 4), GenRequest(prompts[0], 4)])
    assert bad[0].error and bad[1].error is None and bad[1].ids == reqs[0].ids[:4]


@gpu
def test_graph_decoding_advances_the_state_once(models):
    """A captured decode loop gives the tokens of the step-by-step loop: the capture's own step leaves no trace in the states."""
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


@pytest.mark.parametrize("place", ["cpu", pytest.param("b200", marks=gpu)])
def test_command_line(models, place, tmp_path):
    from tensorsharp_b200.cli.main import main
    folder, cfg, w = models("plain")
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
    full = {k: oracle("odd", cfg, w, t) for k, t in ids.items()}
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
    assert svc.architecture == "lisorax" and svc.loaded_model_name == folder.name
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
    synth.write_lisorax(str(bad), device="cpu", layers="aar", mlps="mm-", kv_from={1: 0})
    c = json.loads((bad / "config.json").read_text())
    first, second, third = c["layers"]

    def refused(error, *layers, **top):
        (bad / "config.json").write_text(json.dumps({**c, "layers": list(layers), **top}))
        with pytest.raises(error):
            ModelBase.create(str(bad), "cpu")
    mix, mlp = first["mixer"], first["mlp"]
    refused(ValueError, {**first, "type": "convolution"})
    refused(ValueError, {**first, "mlp": {**mlp, "kind": "sparse"}})
    refused(ValueError, {**first, "mixer": {**mix, "kv_heads": 3}})
    refused(ValueError, {**first, "mixer": {**mix, "heads": 6}})
    refused(ValueError, {**first, "mlp": {**mlp, "router": {"experts": 6, "top": 7}}})
    refused(ValueError, {**first, "mlp": {**mlp, "router": {"experts": 5, "top": 2}}})
    for donor in (1, 2, 5, -1):
        refused(ValueError, first, {**second, "mixer": {**second["mixer"], "kv_from": donor}}, third)
    refused(ValueError, first, {**second, "mixer": {**second["mixer"], "kv_heads": 1}}, third)
    refused(ValueError, first, second, {**third, "mixer": {**third["mixer"], "blocks": 3}})
    refused(ValueError, first, second, third, loop={"start": 0, "stop": 1, "times": 2})
    refused(KeyError, first, first, third)                 # no keys and values of its own
