"""Sogulix against the plain implementation of sogulix_oracle.py, on the CPU ops and (``-m gpu``) on the device in float32 and
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
import sogulix_oracle as O  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
PLACES = ["cpu", pytest.param("f32", marks=gpu), pytest.param("bf16", marks=gpu)]

CONFIGS = {
    "plain": dict(),
    # a loop with layers of its own before and after, odd sizes everywhere, layers without a feed-forward
    "odd": dict(layers="glgl", width=100, heads=3, dim=20, rot_dim=6, vdim=24, q_rank=28, kv_rank=36, window=70, delta_heads=3, delta_dim=20,
                decay_rank=5, ff=52, vocab=333, loop=(1, 3, 3), no_mlp=(0, 2), residual_mult=0.8, softcap=9.0, rot_base=500.0),
    "one": dict(layers="l", heads=1, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16, window=1, loop=(0, 1, 2)),
    "wide": dict(layers="lg", width=264, heads=20, dim=48, rot_dim=32, vdim=80, q_rank=136, kv_rank=200, window=64, delta_heads=2, delta_dim=128,
                 decay_rank=33, ff=200, vocab=1031, loop=(0, 2, 1), scale=0.2, eps=1e-3, residual_mult=1.0, softcap=50.0),
    "delta": dict(layers="gg", width=72, delta_heads=5, delta_dim=96, decay_rank=16, ff=40, residual_mult=0.3),
    "far": dict(layers="lgl", heads=2, dim=64, rot_dim=2, vdim=48, kv_rank=72, window=1000, delta_heads=4, delta_dim=64, loop=(0, 3, 2)),
}


def mixed():
    """No two layers alike: sizes, windows, rotations, scales and feed-forwards differ from layer to layer."""
    c = synth.sogulix_config(layers="lglg", width=96, loop=(1, 4, 2), residual_mult=0.6, softcap=15.0)
    a, b, d, e = c["layers"]
    a["mixer"].update(heads=5, dim=24, vdim=40, kv_rank=24, q_rank=40, mask={"size": 9})
    d["mixer"].update(heads=2, dim=40, rot_dim=24, rot={"dims": 24, "base": 200.0}, kv_rank=56, scale=0.3, mask={"size": 90})
    b["mixer"].update(heads=2, dim=64, decay_rank=20)
    e["mixer"].update(heads=4, dim=16, decay_rank=3)
    d["mlp"]["ff"], e["mlp"] = 120, None
    return c


CONFIGS["mixed"] = dict(config=mixed())


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
    16 bits does to these models.  A few rows may be off by more: at a sequence's first token o = (k . r) v, and the norm of o
    makes much of the rounding of k . r where that is near zero."""
    assert got.shape == want.shape
    e = errors(got, want)
    assert torch.isfinite(e).all()
    if place == "bf16":
        assert e.median() < 0.02 and (e > 0.06).sum() <= max(1, 0.02 * len(e)), (e.median(), e.max())
    else:
        assert e.max() < 3e-5, e


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            folder = tmp_path_factory.mktemp("sogulix") / name
            synth.write_sogulix(str(folder), seed=len(name), device="cpu", **CONFIGS[name])
            made[name] = (folder,) + O.read_model(folder)
        return made[name]
    return get


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def qweight(w, dev):
    t = GGMLType.BF16 if w.dtype == torch.bfloat16 else GGMLType.F32
    return QuantWeight.from_raw(w.contiguous().view(-1).view(torch.uint8), t, tuple(w.shape), dev, "w")


def portions(kv, seqs, cuts, p):
    """Batch of the p-th portion of every sequence that has one: (batch, [(sequence, from, to)])."""
    part = [(b, c[p], c[p + 1]) for b, c in enumerate(cuts) if c[p + 1] > c[p]]
    return kv.build_batch([seqs[b] for b, _, _ in part], [[0] * (hi - lo) for _, lo, hi in part]), part


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("n,lens", [(40, (1, 1, 1)), (61, (7, 1, 3, 2)), (2050, (5, 1, 40)), (24, (3000, 1, 1800))])
def test_seam_and_token_shift(place, n, lens):
    """Residual, both norms and the shift, in three portions per sequence whose cuts fall anywhere."""
    dev, D, eps = device(place), (n + 7) // 8 * 8, 1e-4
    g = torch.Generator().manual_seed(n)

    def pad(t):
        return torch.nn.functional.pad(t, (0, D - n)).to(dev).contiguous()
    w1, w2, s1, s2 = (torch.randn(n, generator=g) * 0.3 for _ in range(4))
    mix = torch.rand(n, generator=g)
    hs = [torch.randn(m, n, generator=g) * 2 for m in lens]
    y1 = [torch.randn(m, n, generator=g).to(dtype(place)) for m in lens]
    y2 = [torch.randn(m, n, generator=g).to(dtype(place)) for m in lens]
    want_h = [h.double() + s1.double() * a.double() + s2.double() * b.double() for h, a, b in zip(hs, y1, y2)]
    want_1 = [O.token_shift(O.zero_centred_norm(x, w1.double(), eps), mix.double()) for x in want_h]
    want_2 = [O.zero_centred_norm(x, w2.double(), eps) for x in want_h]
    kv = PagedKV([None], 400, 16, dev, max_seqs=4)
    seqs = [kv.new_seq() for _ in lens]
    state = torch.full((4, D + 12), float("nan"), device=dev)[:, 4:4 + D]      # a slice of wider rows
    for s in seqs:
        state[s.slot] = 0
    cuts = [[0, max(0, m - 5), max(m - 1, 0), m] for m in lens]
    for p in range(3):
        if not any(c[p + 1] > c[p] for c in cuts):
            continue
        batch, part = portions(kv, seqs, cuts, p)

        def rows(ts):
            return torch.cat([ts[b][lo:hi] for b, lo, hi in part])
        h, a1, a2 = F.parallel_seam(pad(rows(hs)), eps, n, y=(pad(rows(y1)), pad(rows(y2))), scale=(pad(s1), pad(s2)), w=(pad(1 + w1), pad(1 + w2)),
                                    dtype=dtype(place), shift=pad(mix), state=state, batch=batch)
        tol = dict(rtol=1e-2, atol=1e-2) if place == "bf16" else dict(rtol=1e-5, atol=2e-5)
        assert torch.allclose(h[:, :n].double().cpu(), rows(want_h), rtol=1e-5, atol=2e-5)
        assert torch.allclose(a1[:, :n].double().cpu(), rows(want_1), **tol) and torch.allclose(a2[:, :n].double().cpu(), rows(want_2), **tol)
        assert not h[:, n:].any() and not a1[:, n:].any() and not a2[:, n:].any()
    # plain forms: a raw copy into a slice of a wider buffer, a norm in another type, nothing added
    h = pad(hs[0])
    both = torch.full((h.shape[0], 2 * D), 7.0, dtype=dtype(place), device=dev)
    same, out, _ = F.parallel_seam(h, eps, n, out=(both[:, D:], None), outputs=1)
    assert same is h and torch.equal(both[:, D:], h.to(dtype(place))) and (both[:, :D] == 7).all()
    _, x0, _ = F.parallel_seam(h, eps, n, w=(pad(1 + w1), pad(1 + w1)), out=(None, both[:, :D]), outputs=1, dtype=torch.float32)
    assert x0.dtype == torch.float32 and torch.allclose(x0[:, :n].double().cpu(), O.zero_centred_norm(hs[0].double(), w1.double(), eps), atol=2e-5)
    assert torch.equal(both[:, :D], x0.to(dtype(place)))


def spec(H, dim, rot, vdim, rank, q_rank, window, dev, scale=0.5, base=3000.0):
    return F.LatentSpec(H, dim, rot, vdim, rank, q_rank, scale, window, base, F.rotary_freqs(rot, base, dev))


@pytest.mark.parametrize("place", PLACES)
def test_latent_rows_and_rotation(place):
    """Both latent norms and the rotated key part at near and far positions, in the cache and in padded rows."""
    dev, T, pos = device(place), 9, [0, 1, 2, 63, 64, 999, 1000, 65535, 200001]
    s = spec(1, 8, 10, 8, 21, 27, 0, dev)
    g = torch.Generator().manual_seed(5)
    x = torch.randn(T, 27 + 21 + 10, generator=g)
    qn, kn = torch.randn(27, generator=g), torch.randn(21, generator=g)
    kv = PagedKV([(1, s.row, 0)], 4, 64, dev, dtype(place), max_seqs=1)
    batch = kv.build_batch([kv.new_seq()], [[0] * T])
    batch.positions = torch.tensor(pos, dtype=torch.int32, device=dev)
    y = torch.zeros(T, s.qp + 21 + 10 + 5)
    y[:, :27], y[:, s.qp:s.qp + 31] = x[:, :27], x[:, 27:]
    cq = F.latent_cache(y.to(dev), s, qn.to(dev), kn.to(dev), kv.k[0], batch, 1e-5).b
    row = kv.k[0][batch.slots, 0].double().cpu()
    tol = dict(rtol=1e-2, atol=1e-2) if place == "bf16" else dict(rtol=1e-5, atol=1e-5)
    assert torch.allclose(cq[:, :27].double().cpu(), O.rms(x[:, :27].double(), 1e-5) * qn, **tol) and not cq[:, 27:].any()
    assert torch.allclose(row[:, :21], O.rms(x[:, 27:48].double(), 1e-5) * kn, **tol)
    assert torch.allclose(row[:, 21:31], O.rotate_half(x[:, 48:].double(), torch.tensor(pos), 3000.0), **tol) and not row[:, 31:].any()


LATENT = [(4, 32, 16, 32, 40, 24), (3, 20, 6, 24, 36, 70), (7, 64, 32, 48, 88, 33), (17, 48, 2, 16, 130, 64), (1, 16, 0, 80, 256, 1), (33, 128, 64, 128, 512, 65),
          (2, 64, 64, 48, 64, 0), (5, 8, 8, 8, 390, 16)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,dim,rot,vdim,rank,window", LATENT)
def test_latent_attention_with_keys_that_stand_out(place, H, dim, rot, vdim, rank, window):
    """Single rows stand out from all others for one query each: just inside the window, just outside of it, at page borders,
    far back, and one ahead of the query; on pages in no order, in portions and decoding.  The sinks are of the size of the
    scores."""
    dev, page = device(place), 16
    g = torch.Generator().manual_seed(H * dim + rank)
    s = spec(H, dim, rot, vdim, rank, 8, window, dev)
    lens = [150, 33, 209]
    reach = window or 10 ** 6
    kv = PagedKV([(1, s.row, 0)], 40, page, dev, dtype(place), max_seqs=3)
    kv._free = torch.randperm(40, generator=g).tolist()
    kv.k[0].fill_(float("nan"))
    seqs = [kv.new_seq() for _ in lens]
    dt = dtype(place)
    uk, uv = (torch.randn(H * d, rank, generator=g).div(rank ** 0.5).to(dt) for d in (dim, vdim))
    sinks = torch.randn(H, generator=g)
    ukh = uk.double().view(H, dim, rank)
    data = []
    for n in lens:
        c, kr = torch.randn(n, rank, generator=g) * 0.5, torch.randn(n, rot, generator=g) * 0.3
        q = torch.randn(n, H, dim + rot, generator=g) * 0.3
        pairs = []
        for i in (n - 1, n - 2, n // 2, n // 3, page, 2 * page - 1):
            pairs += [(i, j) for j in (i - reach + 1, i - reach, i - 1, 0, page - 1, page, i + 1) if 0 <= j < n]
        marks = min(rank // 2, 8)                             # latent columns that only a marked row uses
        c[:, :marks] = 0
        for m, (i, j) in enumerate(pairs[::max(1, len(pairs) // marks)][:marks]):
            c[j, m] = 6.0
            u = ukh[:, :, m]
            q[i, :, :dim] += (4.0 * u / (u * u).sum(1, keepdim=True)).float()
        c, kr, q = c.to(dt), kr.to(dt), q.to(dt)
        data.append((q, c, kr))
    want = []
    for q, c, kr in data:
        n = len(q)
        k = torch.cat([(c.double() @ uk.double().T).view(n, H, dim), kr.double()[:, None].expand(n, H, rot)], -1)
        qr = torch.cat([q.double()[..., :dim], O.rotate_half(q.double()[..., dim:], torch.arange(n), 3000.0)], -1)
        want.append(O.windowed_attention(qr, k, (c.double() @ uv.double().T).view(n, H, vdim), 0.5, window or None, sinks.double()))
    wuk = torch.nn.functional.pad(uk, (0, s.rank_p - rank)).to(dev)
    wuv = torch.zeros(H, s.Dv, s.rank_p, dtype=dt)
    wuv[:, :vdim, :rank] = uv.view(H, vdim, rank)
    ex = torch.zeros(H, s.Dk, s.row, dtype=dt)
    ex[:, :dim, :rank] = uk.view(H, dim, rank)
    ex[:, dim:dim + rot, rank:rank + rot] = torch.eye(rot)
    ev = torch.zeros(H * s.Dv, s.row, dtype=dt)
    ev[:, :s.rank_p] = wuv.view(H * s.Dv, s.rank_p)[:, :min(s.rank_p, s.row)]
    expand = qweight(torch.cat([ex.view(H * s.Dk, s.row), ev]), dev)
    cuts = [[0, 2, 17, 64, 148, 149, 150], [0, 16, 31, 32, 32, 32, 33], [0, 1, 130, 193, 207, 208, 209]]      # the last two: decoding
    for p in range(6):
        batch, part = portions(kv, seqs, cuts, p)
        assert batch.is_decode == (p >= 4)
        rows = torch.zeros(batch.T, s.row, dtype=dt)
        rows[:, :rank], rows[:, rank:rank + rot] = (torch.cat([data[b][x][lo:hi] for b, lo, hi in part]) for x in (1, 2))
        kv.k[0][batch.slots] = rows.view(batch.T, 1, s.row).to(dev)
        q = torch.zeros(batch.T, H, s.Dk, dtype=torch.bfloat16 if place == "bf16" and not batch.is_decode else torch.float32)
        q[..., :dim + rot] = torch.cat([data[b][0][lo:hi] for b, lo, hi in part])
        out = F.latent_attention(q.view(batch.T, -1).to(dev), kv.k[0], batch, s, wuk=wuk, wuv=wuv.view(H * s.Dv, s.rank_p).to(dev), expand=expand,
                                 sinks=sinks.to(dev)).view(batch.T, H, s.Dv)
        ref = torch.cat([want[b][lo:hi] for b, lo, hi in part])
        err = (out[..., :vdim].double().cpu() - ref).abs().max()
        assert err < (0.06 if place == "bf16" else 2e-4), (p, err)
        assert not out[..., vdim:].any()


DELTA = [(3, 20, 5), (2, 64, 16), (5, 96, 33), (4, 128, 64), (1, 150, 3), (2, 256, 8), (40, 32, 8)]


@gpu
@pytest.mark.parametrize("H,n", [(h, n) for h, n, _ in DELTA])
def test_delta_rule_prompt_kernels_keep_32_bits(H, n):
    """Both prompt paths, the tensor-core one included, against the oracle with 32-bit outputs: unequal sequences with full,
    short and one-token chunks, and the state they leave."""
    from tensorsharp_b200.ops import kernels as K
    D, eps = (n + 31) // 32 * 32, 1e-5
    g = torch.Generator().manual_seed(n)
    cu, T = [0, 1, 44, 52, 68, 75], 75
    x = {k: torch.randn(T, H, n, generator=g) for k in "rkvagz"}
    x["z"] = x["z"] * 3 - 2
    x["z"][:, :, ::2] -= 14                                                # half of the channels forget next to nothing
    s0 = torch.randn(6, H, n, n, generator=g)
    w0, ab, on = (torch.randn(H, n, generator=g) for _ in range(3))

    def pad(v):
        return torch.nn.functional.pad(v, (0, D - n)).reshape(*v.shape[:-2], H * D).contiguous().cuda()
    y, z = torch.cat([pad(x[k]) for k in "rkvag"], 1), pad(x["z"])
    state = torch.zeros(6, H, D, D)
    state[:, :, :n, :n] = s0
    slots = torch.tensor([4, 0, 5, 2, 1])
    outs, states = [], []
    for kind in ("scan", "wide", "chunk"):
        st = state.cuda()
        args = (y, z, pad(w0), pad(ab), pad(on), st, torch.tensor(cu, dtype=torch.int32).cuda(), slots.cuda())
        kw = dict(H=H, D=D, n=n, eps=eps, out_dtype=torch.float32)
        out = K.general_delta_chunk(*args, max_q=43, **kw) if kind == "chunk" else K.general_delta_prompt(*args, wide=kind == "wide", **kw)
        outs.append(out.cpu().double().view(T, H, D))
        states.append(st.cpu().double())
    x = {k: v.double() for k, v in x.items()}
    decay = torch.exp(-torch.exp(torch.tensor(-0.5).double()) * O.sigmoid(x["z"] + w0))
    for b, (lo, hi) in enumerate(zip(cu, cu[1:])):
        o, S = O.delta_rule(x["r"][lo:hi], x["k"][lo:hi], x["v"][lo:hi], decay[lo:hi], O.sigmoid(x["a"][lo:hi] + ab), s0[slots[b]].double().transpose(1, 2))
        want = O.rms(o, eps) * on * O.sigmoid(x["g"][lo:hi])
        for out, st in zip(outs, states):
            assert torch.allclose(out[lo:hi, :, :n], want, rtol=3e-5, atol=3e-5), (b, (out[lo:hi, :, :n] - want).abs().max())
            assert torch.allclose(st[slots[b], :, :n, :n].transpose(1, 2), S, rtol=3e-5, atol=3e-5)
            assert not out[lo:hi, :, n:].any() and not st[slots[b], :, n:].any() and not st[slots[b], :, :, n:].any()
    assert all(torch.equal(st[3], state[3].double()) for st in states)      # nobody's slot


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,n,rank", DELTA)
def test_delta_rule_in_portions(place, H, n, rank):
    """The recurrence with its decay map, norm and gate: one-kernel steps and prompt kernels in turns, unequal sequences, a
    slot that is given back and used again.  Half of the channels forget and remove next to nothing, so what is written at
    the start still shows at the end."""
    dev, eps, D, rp = device(place), 1e-4, (n + 31) // 32 * 32, (rank + 7) // 8 * 8
    g = torch.Generator().manual_seed(H * n)
    lens = [70, 19, 33]
    names = "rkvag"
    w2, w0 = torch.randn(H * n, rank, generator=g).to(dtype(place)), torch.randn(H * n, generator=g) * 2
    ab, on = torch.randn(H * n, generator=g) * 2, torch.randn(H * n, generator=g)
    w0[::2] -= 14
    ab[::2] -= 14
    x = [{k: torch.randn(m, H * n, generator=g) for k in names} for m in lens]
    low = [torch.randn(m, rank, generator=g) for m in lens]

    def heads(v):                                              # [.., H * n] -> [.., H * D]
        v = v.view(*v.shape[:-1], H, n)
        return torch.nn.functional.pad(v, (0, D - n)).reshape(*v.shape[:-2], H * D)

    want = []
    for xs, lo in zip(x, low):
        decay = torch.exp(-torch.exp(torch.tensor(-0.5).double()) * O.sigmoid(torch.tanh(lo.double()) @ w2.double().T + w0.double()))
        v = [xs[k].double().view(-1, H, n) for k in "rkv"]
        o, _ = O.delta_rule(*v, decay.view(-1, H, n), O.sigmoid(xs["a"].double() + ab.double()).view(-1, H, n))
        want.append(O.rms(o, eps).reshape(-1, H * n) * on.double() * O.sigmoid(xs["g"].double()))
    state = torch.full((3, 7 * 4 + H * D * D), float("nan"), device=dev)[:, 28:].unflatten(1, (H, D, D))
    kv = PagedKV([None], 40, 16, dev, max_seqs=3)
    w2d = torch.zeros(H, D, rp, dtype=dtype(place))
    w2d[:, :n, :rank] = w2.view(H, n, rank)
    w2d = qweight(w2d.view(H * D, rp), dev)
    vecs = [heads(v).to(dev) for v in (w0, ab, on)]
    for again in range(2):
        seqs = [kv.new_seq() for _ in lens]
        for q in seqs:
            state[q.slot] = 0
        cuts = [[0, 1, 3, 40, 69, 70], [0, 10, 17, 18, 18, 19], [0, 7, 7, 32, 32, 33]]
        for p in range(5):
            batch, part = portions(kv, seqs, cuts, p)
            assert (batch.max_q_len < F.GENERAL_DELTA_SCAN_MIN) == (p in (1, 4))
            y = torch.cat([torch.cat([heads(x[b][k][lo:hi]) for k in names] +
                                     [torch.nn.functional.pad(low[b][lo:hi], (0, rp - rank))], 1) for b, lo, hi in part])
            y = torch.nn.functional.pad(y, (0, 4)).to(dev)[:, :-4]                # a row stride of its own
            out = F.general_delta(y, w2d, *vecs, state, batch, H=H, D=D, n=n, rank=rank, eps=eps, dtype=dtype(place))
            got = out.double().cpu().view(-1, H, D)
            ref = torch.cat([want[b][lo:hi] for b, lo, hi in part]).view(-1, H, n)
            err = (got[..., :n] - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
            assert err < (0.01 if place == "bf16" else 2e-5), (p, err)
            assert not got[..., n:].any()
        for q in seqs:
            kv.free_seq(q)


def test_what_the_delta_rule_keeps():
    """The oracle itself: without decay and removal a value comes back for its key however far away; with full removal of a
    key its value is replaced."""
    g = torch.Generator().manual_seed(0)
    T, D = 50, 16
    k = torch.linalg.qr(torch.randn(D, D, generator=g, dtype=torch.float64))[0][None].repeat(4, 1, 1).reshape(-1, D)[:T]
    v = torch.randn(T, D, generator=g, dtype=torch.float64)
    one = torch.ones(T, 1, D, dtype=torch.float64)
    r = torch.zeros(T, 1, D, dtype=torch.float64)
    r[15, 0], r[T - 1, 0] = k[0], k[T - 1 - 2]
    o, _ = O.delta_rule(r, k[:, None], v[:, None], one, 0 * one)
    assert torch.allclose(o[15, 0], v[0], atol=1e-5)
    o, _ = O.delta_rule(r, k[:, None], v[:, None], one, one)
    assert torch.allclose(o[T - 1, 0], v[T - 3], atol=1e-5)                        # (the same key was written three times)


@gpu
@pytest.mark.parametrize("H,dim,rot,vdim,rank,window", [(20, 32, 16, 48, 512, 300), (40, 24, 160, 16, 64, 0), (33, 64, 64, 32, 300, 97), (64, 16, 200, 16, 500, 0),
                                                        (16, 32, 96, 32, 200, 0)])
def test_latent_decoding_of_many_heads_and_sequences(H, dim, rot, vdim, rank, window):
    """Six sequences of very different lengths in one step: every head tile, row width and split count of the decode kernel
    against the attention written out."""
    g = torch.Generator().manual_seed(H + rank)
    s = spec(H, dim, rot, vdim, rank, 8, window, "cuda", scale=0.2)
    lens = [1, 700, 64, 65, 333, 1500]
    kv = PagedKV([(1, s.row, 0)], 60, 64, "cuda", torch.bfloat16, max_seqs=6)
    kv._free = torch.randperm(60, generator=g).tolist()
    kv.k[0].fill_(float("nan"))
    seqs = [kv.new_seq() for _ in lens]
    uk, uv = (torch.randn(H * d, rank, generator=g).div(rank ** 0.5).bfloat16() for d in (dim, vdim))
    sinks = torch.randn(H, generator=g)
    rows = [torch.nn.functional.pad(torch.randn(n, rank + rot, generator=g), (0, s.row - rank - rot)).bfloat16() for n in lens]
    q = torch.randn(6, H, dim + rot, generator=g) * 0.5
    kv.build_batch([x for x, n in zip(seqs, lens) if n > 1], [[0] * (n - 1) for n in lens if n > 1])
    batch = kv.build_batch(seqs, [[0]] * 6)
    for x, r in zip(seqs, rows):
        at = torch.tensor([x.pages[j // 64] * 64 + j % 64 for j in range(len(r))])
        kv.k[0][at.cuda(), 0] = r.cuda()
    wuk = torch.nn.functional.pad(uk, (0, s.rank_p - rank)).cuda()
    wuv = torch.zeros(H, s.Dv, s.rank_p, dtype=torch.bfloat16)
    wuv[:, :vdim, :rank] = uv.view(H, vdim, rank)
    out = F.latent_attention(torch.nn.functional.pad(q, (0, s.Dk - dim - rot)).view(6, -1).cuda(), kv.k[0], batch, s, wuk=wuk,
                             wuv=wuv.view(H * s.Dv, s.rank_p).cuda(), expand=None, sinks=sinks.cuda()).view(6, H, s.Dv)
    for b, (n, r) in enumerate(zip(lens, rows)):
        lo = max(0, n - window) if window else 0
        r = r.double()[lo:]
        qr = torch.cat([q[b, :, :dim].double(), O.rotate_half(q[b, :, dim:].double()[None], torch.tensor([n - 1]), 3000.0)[0]], -1)
        k = torch.cat([(r[:, :rank] @ uk.double().T).view(-1, H, dim), r[:, None, rank:rank + rot].expand(-1, H, rot)], -1)
        v = (r[:, :rank] @ uv.double().T).view(-1, H, vdim)
        sc = torch.einsum("hd,thd->ht", qr, k) * 0.2
        e = torch.exp(sc - 20)
        want = torch.einsum("ht,thv->hv", e / (e.sum(1, keepdim=True) + torch.exp(sinks.double() - 20)[:, None]), v)
        assert (out[b, :, :vdim].double().cpu() - want).abs().max() < 0.05, b


@pytest.mark.parametrize("place", PLACES)
def test_logit_cap(place):
    z = torch.linspace(-200, 200, 999).to(device(place))
    want = 12.5 * torch.tanh(z.double().cpu() / 12.5)
    assert torch.allclose(F.softcap(z, 12.5).double().cpu(), want, atol=1e-5) and F.softcap(z, 0.0) is z


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_against_the_oracle(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    assert len(m.kv.k) == len(O.layer_runs(cfg))
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


def test_order_of_layer_runs(models):
    _, cfg, _ = models("odd")
    assert O.layer_runs(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    m = load(models("odd")[0], "cpu")
    assert m.runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert [t is None for t in m.kv.k] == [True, False, True, False, True, False, True, False]
    assert [t is None for t in m.delta_state] == [False, True] * 4 and len(m.shift_state) == 8
    # every run has rows of its own
    base, spans = m.state.data_ptr(), []
    for t in m.shift_state + [d for d in m.delta_state if d is not None]:
        spans.append(((t[0].data_ptr() - base) // 4, t[0].numel()))
    spans.sort()
    assert all(a + n <= b for (a, n), (b, _) in zip(spans, spans[1:])) and sum(n for _, n in spans) == m.state.shape[1]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "plain", "wide", "mixed"])
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
@pytest.mark.parametrize("name", ["odd", "far"])
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
def test_rings_of_pages_for_the_window(models, place, monkeypatch):
    """With a ring of pages per sequence the rows that have left the window are overwritten."""
    monkeypatch.setenv("TSB_KV_WINDOW_RING", "1")
    monkeypatch.setenv("TSB_KV_RING_CHUNK", "64")
    folder, cfg, w = models("plain")
    m = load(folder, place, max_context=320, page_size=16)
    poison(m)
    assert m.kv.ring and m.kv.ring_pages * 16 < 190
    n, eng, got = 190, StepEngine(m, 4), []
    ids = tokens(n, cfg["vocab"], 6)
    for a, b in ((0, 64), (64, 100), (100, 101), (101, 160), (160, 180)) + tuple((i, i + 1) for i in range(180, n)):
        got.append(eng.step([("a", ids[a:b], list(range(b - a)))]))
    agree(torch.cat(got), O.forward(w, cfg, ids), place)


@pytest.mark.parametrize("place", PLACES)
def test_wanted_rows_only(models, place):
    folder, cfg, w = models("delta")
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
    slack = 0.1 if place == "bf16" else 1e-3
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
    """A captured decode loop gives the tokens of the step-by-step loop: the capture's own step leaves no trace."""
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
            greedy_is_argmax(w, cfg, prompt, ids, 0.1 if place == "b200" else 1e-3)


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
    assert svc.architecture == "sogulix" and svc.loaded_model_name == folder.name
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
    synth.write_sogulix(str(bad), device="cpu", layers="l")
    c = json.loads((bad / "config.json").read_text())
    first = c["layers"][0]
    for change in ({"type": "convolution"}, {"mlp": {**first["mlp"], "kind": "moe"}},
                   {"mixer": {**first["mixer"], "rot": {"dims": 4, "base": 10.0}}}, {"mixer": {**first["mixer"], "heads": 5}}):
        (bad / "config.json").write_text(json.dumps({**c, "layers": [{**first, **change}]}))
        with pytest.raises(ValueError):
            ModelBase.create(str(bad), "cpu")
    for loop in ({"start": 0, "stop": 2, "times": 2}, {"start": 1, "stop": 0, "times": 2}):
        (bad / "config.json").write_text(json.dumps({**c, "loop": loop}))
        with pytest.raises(ValueError):
            ModelBase.create(str(bad), "cpu")
    (bad / "config.json").write_text(json.dumps({**c, "loop": {"start": 0, "stop": 1, "times": 2}}))
    with pytest.raises(KeyError):
        ModelBase.create(str(bad), "cpu")                  # no loop.in
