"""Fobolorn against the plain implementation of fobolorn_oracle.py, on the CPU ops and (``-m gpu``) on the device in float32 and
bfloat16: every mechanism alone, whole models, portions, batches, page re-use, long decoding, generation."""
import json
import os
import subprocess
import sys

import pytest
import torch

from tensorsharp_b200.models import synth
from tensorsharp_b200.models.base import ModelBase
from tensorsharp_b200.ops import functional as F
from tensorsharp_b200.runtime.batching import ContinuousBatcher, GenRequest, StepEngine
from tensorsharp_b200.runtime.engine import generate
from tensorsharp_b200.runtime.paged_kv import OutOfPagesError, PagedKV

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fobolorn_oracle as O  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
PLACES = ["cpu", pytest.param("f32", marks=gpu), pytest.param("bf16", marks=gpu)]

CONFIGS = {
    "plain": dict(),
    "odd": dict(n_layers=4, width=100, heads=3, kv_heads=1, dim=40, vdim=24, ff=40, shared_ff=100, experts=5, top=3, vocab=333,
                loop=(1, 3, 2), no_mlp=(0,), q_every=9, q_coef=0.7),
    "square": dict(n_layers=2, heads=8, kv_heads=2, dim=64, vdim=64, experts=3, top=1, shared_ff=24, loop=(0, 1, 3), q_every=7,
                   router_scale=0.6),
    "wide": dict(n_layers=2, heads=4, kv_heads=4, dim=128, vdim=128, experts=6, top=6, scale=0.05, eps=1e-3, vocab=1031),
    "group": dict(n_layers=2, width=72, heads=20, kv_heads=1, dim=16, vdim=80, loop=(0, 2, 2), no_mlp=(0, 1), q_every=1),
    "tail": dict(n_layers=3, width=136, heads=6, kv_heads=3, dim=96, vdim=32, ff=88, shared_ff=88, loop=(1, 3, 1), q_coef=0.0),
}


def device(place):
    return "cpu" if place == "cpu" else "cuda"


def dtype(place):
    return torch.bfloat16 if place == "bf16" else torch.float32


def load(folder, place, **kw):
    kw.setdefault("max_context", 512)
    kw.setdefault("max_seqs", 4)
    return ModelBase.create(str(folder), device(place), compute_dtype=dtype(place) if place != "cpu" else None, **kw)


def poison(model):
    """NaN in every cache row that nothing has been written to: a kernel that reads past a sequence's end shows."""
    for t in model.kv.k + model.kv.v:
        t.fill_(float("nan"))


def errors(got, want):
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def agree(got, want, place):
    """Logit rows against the oracle's: to rounding in float32.  In bfloat16 the bound is what rounding the inputs of all
    products to 16 bits does to these models (median 0.005 to 0.025), and a token whose router is at a close call may go to
    another expert, so a few rows may be off by more."""
    assert got.shape == want.shape
    e = errors(got, want)
    assert torch.isfinite(e).all()
    if place == "bf16":
        assert e.median() < 0.03 and (e > 0.08).sum() <= max(1, 0.1 * len(e)), e
    else:
        assert e.max() < 2e-5, e


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            folder = tmp_path_factory.mktemp("fobolorn") / name
            synth.write_fobolorn(str(folder), seed=len(name), device="cpu", **CONFIGS[name])
            made[name] = (folder,) + O.read_model(folder)
        return made[name]
    return get


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T,n,parts", [(1, 40, 1), (5, 61, 3), (320, 2050, 2)])
def test_seam_of_two_sublayers(place, T, n, parts):
    """h + post-norm of the summed expert rows (+ a vector), then the next pre-norm; the width is padded to 8 columns."""
    g = torch.Generator().manual_seed(n)
    D, eps, dev = (n + 7) // 8 * 8, 1e-4, device(place)

    def pad(t):
        return torch.nn.functional.pad(t, (0, D - n)).to(dev)
    h, y = torch.randn(T, n, generator=g) * 2 + 1, torch.randn(T * parts, n, generator=g) + 0.5
    w = torch.rand(T * parts, generator=g) + 0.1
    post, pre = [torch.randn(n, generator=g) for _ in "wb"], [torch.randn(n, generator=g) for _ in "wb"]
    add = torch.randn(n, generator=g)
    order = torch.randperm(T * parts, generator=g)
    summed = (y[order].double() * w.double()[:, None]).view(T, parts, n).sum(1)
    want_h = h.double() + O.layer_norm(summed, post[0].double(), post[1].double(), eps) + add.double()
    want_a = O.layer_norm(want_h, pre[0].double(), pre[1].double(), eps)
    hd = pad(h).contiguous()
    a = F.residual_layernorm(hd, eps, n, y=F.MoeParts(pad(y).contiguous(), parts, order.to(torch.int32).to(dev), w.to(dev)),
                             post=[pad(t) for t in post], add=pad(add), pre=[pad(t) for t in pre], dtype=dtype(place))
    assert torch.allclose(hd[:, :n].double().cpu(), want_h, atol=2e-5) and not hd[:, n:].any()
    assert torch.allclose(a.b[:, :n].double().cpu(), want_a, atol=0.05 if place == "bf16" else 5e-5) and not a.b[:, n:].any()
    before = hd.clone()
    assert F.residual_layernorm(hd, eps, n, y=None, pre=[pad(t) for t in pre], dtype=dtype(place)) is not None
    assert torch.equal(hd, before)                                        # no sublayer output: h is only read


@pytest.mark.parametrize("place", PLACES)
def test_query_temperature_and_head_norm(place):
    """Query factors on both sides of the steps, and the norm's divisor of a padded head."""
    dev, Dk, dim, Dv, every, coef = device(place), 32, 27, 16, 50, 0.8
    pos = [0, 47, 48, 49, 50, 98, 99, 100, 148, 149, 150, 50 * 700 - 2, 50 * 700 - 1, 50 * 700]
    T = len(pos)
    g = torch.Generator().manual_seed(3)
    x = torch.randn(T, 2 * dim + Dv, generator=g)
    qn, kn = torch.randn(dim, generator=g), torch.randn(dim, generator=g)

    def pad(t, n):
        return torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    y = torch.cat([pad(x[:, :dim], Dk), pad(x[:, dim:2 * dim], Dk), x[:, 2 * dim:]], 1).to(dev)
    kv = PagedKV([(1, Dk, Dv)], 4, 64, dev, dtype(place), max_seqs=1)
    batch = kv.build_batch([kv.new_seq()], [[0] * T])
    batch.positions = torch.tensor(pos, dtype=torch.int32, device=dev)
    q = F.qkv_rope_cache(y[:, :Dk].view(T, 1, Dk), y[:, Dk:2 * Dk].view(T, 1, Dk), y[:, 2 * Dk:].view(T, 1, Dv), Hq=1, Hkv=1, Dh=Dk, Dv=Dv,
                         norm_n=dim, batch=batch, k_cache=kv.k[0], v_cache=kv.v[0], rope=None, qn=pad(qn, Dk).to(dev),
                         kn=pad(kn, Dk).to(dev), eps=1e-5, q_temp=(coef, every))
    want_q = O.rms_norm(x[:, :dim].double(), qn.double(), 1e-5) * O.query_temperature(torch.tensor(pos), coef, every)[:, None]
    want_k = O.rms_norm(x[:, dim:2 * dim].double(), kn.double(), 1e-5)
    tol = dict(rtol=1e-2, atol=1e-2) if place == "bf16" else dict(rtol=2e-5, atol=2e-5)
    assert torch.allclose(q[:, 0, :dim].double().cpu(), want_q, **tol) and not q[:, 0, dim:].any()
    assert torch.allclose(kv.k[0][batch.slots, 0, :dim].double().cpu(), want_k, **tol)
    assert torch.allclose(kv.v[0][batch.slots, 0].double().cpu(), x[:, 2 * dim:].double(), **tol)
    steps = O.query_temperature(torch.tensor([48, 49, 98, 99]), coef, every)
    assert steps[0] == 1.0 and steps[1] == steps[2] > 1.0 and steps[3] > steps[2]


HEADS = [(9, 3, 64, 80), (4, 2, 32, 48), (8, 2, 64, 64), (4, 4, 128, 128), (3, 3, 16, 112), (20, 1, 208, 256), (5, 5, 96, 16),
         (17, 1, 128, 64), (24, 1, 64, 64), (2, 1, 256, 256)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,Dk,Dv", HEADS)
def test_attention_with_keys_that_stand_out(place, H, G, Dk, Dv):
    """Single keys stand out from hundreds for one query each: at a page border, the first token, far back, the query
    itself; and one key would stand out for all the queries ahead of it, which may not see it.  Prompts in portions and
    decoding."""
    dev, page = device(place), 16
    g = torch.Generator().manual_seed(H * Dk + Dv)
    lens = [150, 33, 209]
    kv = PagedKV([(G, Dk, Dv)], 40, page, dev, dtype(place), max_seqs=3)
    kv._free = torch.randperm(40, generator=g).tolist()                     # pages in no order
    kv.k[0].fill_(float("nan"))
    kv.v[0].fill_(float("nan"))
    seqs = [kv.new_seq() for _ in lens]
    data = []
    for n in lens:
        q, k, v = (torch.randn(n, h, d, generator=g) * s for h, d, s in ((H, Dk, 0.3), (G, Dk, 0.3), (G, Dv, 1.0)))
        q[:, :, :9] = 0
        for i, j in ((n - 1, 0), (n - 2, page - 1), (n - 3, page), (n - 4, n - 4), (n // 2, 1), (page, page), (page - 1, 0)):
            q[i, :, i % 7] = 9.0                                           # query i and key j meet in one column
            k[j, :, i % 7] = 9.0
        future = {150: 100, 33: 20, 209: 160}[n]                            # in the middle of a portion
        k[:, :, :9][:, :, 8] = 0
        k[future, :, 8] = 12.0
        q[:future, :, 8] = 8.0
        data.append((q.to(dtype(place)), k.to(dtype(place)), v.to(dtype(place)), torch.randn(n, H, generator=g)))
    scale = 0.5
    want = [O.head_gate(O.causal_attention(q.double(), k.double(), v.double(), scale), gt.double()) for q, k, v, gt in data]
    cuts = [[0, 2, 17, 64, 149, 150], [0, 16, 31, 32, 33, 33], [0, 1, 130, 193, 208, 209]]      # the last portions: decoding
    for p in range(5):
        part = [(b, c[p], c[p + 1]) for b, c in enumerate(cuts) if c[p + 1] > c[p]]
        batch = kv.build_batch([seqs[b] for b, _, _ in part], [[0] * (hi - lo) for _, lo, hi in part])
        assert batch.is_decode == (p == 4)
        kv.k[0][batch.slots] = torch.cat([data[b][1][lo:hi] for b, lo, hi in part]).to(dev)
        kv.v[0][batch.slots] = torch.cat([data[b][2][lo:hi] for b, lo, hi in part]).to(dev)
        gate = torch.zeros(batch.T, H + 3, device=dev)                     # a view with a row stride of its own
        gate[:, 2:2 + H] = torch.cat([data[b][3][lo:hi] for b, lo, hi in part]).to(dev)
        out = F.attention(torch.cat([data[b][0][lo:hi] for b, lo, hi in part]).to(dev), kv.k[0], kv.v[0], batch, scale=scale, Hq=H,
                          Hkv=G, Dh=Dk, Dv=Dv, gate=gate[:, 2:2 + H])
        ref = torch.cat([want[b][lo:hi] for b, lo, hi in part]).reshape(batch.T, H * Dv)
        assert torch.allclose(out.double().cpu(), ref, atol=0.03 if place == "bf16" else 2e-4), (p, (out.double().cpu() - ref).abs().max())


@pytest.mark.parametrize("place", PLACES)
def test_router(place):
    g = torch.Generator().manual_seed(1)
    for T, E, k, always in ((7, 5, 2, 0), (130, 33, 6, 3), (3, 300, 17, 1), (9, 4, 4, 0), (4, 1, 1, 2)):
        z = torch.randn(T, E + (always > 0), generator=g) * 4
        z[0, :E] += 200.0                                                  # large logits: nothing may overflow
        ids, w = F.route_softmax_renorm(z.to(device(place)), E, k, 1.7, always)
        want_ids, want_w = O.route(z[:, :E].double(), k, 1.7)
        assert ids.dtype == torch.int32 and torch.equal(ids[:, :k].cpu().long(), want_ids)
        assert torch.allclose(w[:, :k].double().cpu(), want_w, rtol=2e-5, atol=1e-7)
        if always:
            assert ids[:, k:].cpu().tolist() == [[E + i for i in range(always)]] * T
            assert torch.allclose(w[:, k:].double().cpu(), torch.sigmoid(z[:, E:].double()).expand(T, always), rtol=2e-5)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T", [1, 3, 19, 70, 1500])
def test_experts_with_a_shared_expert_in_slices(models, place, T):
    """Token counts on both sides of every path's limits; the shared expert is wider than the experts (odd) or narrower."""
    for name, layer in (("odd", 1), ("square", 0)):
        folder, cfg, w = models(name)
        m = load(folder, place)
        g = torch.Generator().manual_seed(T)
        x = torch.randn(T, cfg["width"], generator=g).to(dtype(place))
        if T > 1:                                                          # one expert gets far more tokens than the others
            x[: T // 2] = x[:1] + 0.05 * x[: T // 2]
        D = m.cfg.hidden
        a = F.Act(torch.nn.functional.pad(x, (0, D - cfg["width"])).to(device(place)).contiguous())
        parts = m.experts(a, m.layers[layer]["mlp"])
        got = (parts.sum() if isinstance(parts, F.MoeParts) else parts)[:, :cfg["width"]].double().cpu()
        want = O.moe(x.double(), w, f"l{layer}.mlp.", cfg["layers"][layer]["mlp"])
        err = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
        # (a router at a close call: see agree)
        assert (err < (0.02 if place == "bf16" else 1e-5)).float().mean() > 0.97, err.max()


@gpu
def test_pairs_sorted_by_expert_on_the_device():
    from tensorsharp_b200.ops import kernels as K
    g = torch.Generator().manual_seed(0)
    for T, k, E, bn in ((1, 1, 1, 32), (5, 3, 9, 32), (300, 5, 33, 64), (9000, 5, 33, 256), (4096, 3, 1000, 32)):
        ids = torch.randint(0, E, (T, k), generator=g, dtype=torch.int32)
        ids[: T // 2] = E - 1
        order, tiles, pos = (t.cpu().long() for t in K.moe_sort(ids.cuda(), E, bn))
        flat = ids.reshape(-1)
        assert torch.equal(pos[order], torch.arange(T * k)) and (flat[order].diff() >= 0).all()
        seen = torch.zeros(T * k)
        for e, lo, hi in tiles.tolist():
            if e >= 0:
                assert 0 < hi - lo <= bn and (flat[order[lo:hi]] == e).all()
                seen[lo:hi] += 1
        assert (seen == 1).all()


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_against_the_oracle(models, place, name):
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    loop = cfg.get("loop")
    assert len(m.kv.k) == len(cfg["layers"]) + ((loop["times"] - 1) * (loop["stop"] - loop["start"]) if loop else 0)
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


def test_residual_stream_of_every_pass(models):
    """The order of passes and the vector ahead of each: a loop in the middle, with a layer of its own before and after."""
    _, cfg, _ = models("odd")
    assert O.layer_runs(cfg) == [(0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, None, False)]
    m = load(models("odd")[0], "cpu")
    assert m.runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["odd", "square"])
@pytest.mark.parametrize("cut", [[1], [2], [3, 2, 61], [64], [63, 1, 2, 65]])
def test_portions_and_token_by_token(models, place, name, cut):
    """However a prompt is cut, its logits are the same."""
    folder, cfg, w = models(name)
    m = load(folder, place)
    poison(m)
    n = 70 if cut == [1] else 150
    ids = tokens(n, cfg["vocab"], 5)
    want = O.forward(w, cfg, ids)
    eng, got, at, i = StepEngine(m, 4), [], 0, 0
    while at < n:
        k = min(cut[i % len(cut)], n - at)
        got.append(eng.step([("a", ids[at:at + k], list(range(k)))]))
        at, i = at + k, i + 1
    agree(torch.cat(got), want, place)


@pytest.mark.parametrize("place", PLACES)
def test_batches_of_unequal_requests_on_pages_used_before(models, place):
    """Portions beside single tokens, a request left out of steps, requests that end and others that take their pages and
    slots; the pool holds no page to spare."""
    folder, cfg, w = models("odd")
    m = load(folder, place, max_context=320, kv_pages=5)
    poison(m)
    names = {"a": 130, "b": 64, "c": 40, "d": 1, "e": 190, "f": 70}
    ids = {k: tokens(n, cfg["vocab"], ord(k)) for k, n in names.items()}
    want = {k: O.forward(w, cfg, t) for k, t in ids.items()}
    at, got = {k: 0 for k in ids}, {k: [] for k in ids}
    eng = StepEngine(m, 4)
    plan = [[("a", 60), ("b", 2)], [("b", 61), ("a", 5)], [("a", 1), ("b", 1), ("c", 39)], [("c", 1), ("a", 1), ("d", 1)], [("a", 62)], [("a", 1)],
            [("e", 65), ("f", 3)], [("f", 1), ("e", 1)], [("f", 1)], [("e", 2), ("f", 64)], [("e", 121), ("f", 1)], [("e", 1)]]
    pages = set()
    for step in plan:
        entries = [(k, ids[k][at[k]:at[k] + n], list(range(n))) for k, n in step]
        out = eng.step(entries)
        row = 0
        for k, n in step:
            got[k].append(out[row:row + n])
            row, at[k] = row + n, at[k] + n
            pages |= set(eng.live[k].pages)
            if at[k] == names[k]:
                eng.end(k)
    assert at == names and not eng.live and m.kv.free_pages == 5 and pages <= set(range(5))
    for k in ids:
        agree(torch.cat(got[k]), want[k], place)
    with pytest.raises(OutOfPagesError):
        eng.step([("x", tokens(321, 333), [])])
    with pytest.raises(ValueError):
        eng.step([("y", [1, 2], [2])])


@pytest.mark.parametrize("place", PLACES)
def test_wanted_rows_only(models, place):
    folder, cfg, w = models("tail")
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
def test_long_decoding(models, place):
    """Hundreds of single steps (captured graphs on the device) after a short prompt, over several pages."""
    folder, cfg, w = models("square")
    m = load(folder, place)
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
    folder, cfg, w = models("wide" if place == "bf16" else "odd")       # (wide: every expert is chosen, no close calls)
    m = load(folder, place)
    prompts = [tokens(n, cfg["vocab"], n) for n in (5, 70, 1, 33, 12)]
    eng = ContinuousBatcher(m, 3, prefill_chunk=portion)
    reqs = eng.run([GenRequest(p, 20) for p in prompts])
    assert m.kv.free_pages == m.kv.n_pages
    for p, r in zip(prompts, reqs):
        assert r.error is None and len(r.ids) == 20
        greedy_is_argmax(w, cfg, p, r.ids, 0.1 if place == "bf16" else 1e-3)
        m.reset_kv_cache()
        alone = generate(m, p, 20, prefill_chunk=16)
        if place == "bf16":
            greedy_is_argmax(w, cfg, p, alone, 0.1)
        else:
            assert alone == r.ids
    bad = eng.run([GenRequest([], 4), GenRequest(prompts[0], 4)])
    assert bad[0].error and bad[1].error is None and bad[1].ids == reqs[0].ids[:4]


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
    folder, cfg, w = models("wide")
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


@pytest.mark.parametrize("place", ["cpu", pytest.param("f32", marks=gpu), pytest.param("bf16", marks=gpu)])
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
    assert svc.architecture == "fobolorn" and svc.loaded_model_name == folder.name
    svc.close()


def test_what_is_refused(models, tmp_path, monkeypatch):
    from tensorsharp_b200.gguf.folder import ModelFolder, write_safetensors
    from tensorsharp_b200.gguf.reader import GGUFFormatError
    folder, cfg, w = models("plain")
    with pytest.raises(ValueError):
        ModelBase.create(str(folder), "cpu", tp_rank=0, tp_size=2)
    with pytest.raises(ValueError):
        ModelBase.create(str(folder), "cpu", pp_rank=0, pp_size=2)
    monkeypatch.setenv("TSB_KV_DTYPE", "fp8")
    with pytest.raises(ValueError):
        ModelBase.create(str(folder), "cpu")
    monkeypatch.delenv("TSB_KV_DTYPE")
    bad = tmp_path / "bad"
    synth.write_fobolorn(str(bad), {**synth.fobolorn_config(n_layers=1), "architecture": "Fobolorn"}, device="cpu")
    c = json.loads((bad / "config.json").read_text())
    for change in ({"type": "convolution"}, {"mlp": {**c["layers"][0]["mlp"], "kind": "dense"}}):
        (bad / "config.json").write_text(json.dumps({**c, "layers": [{**c["layers"][0], **change}]}))
        with pytest.raises(ValueError):
            ModelBase.create(str(bad), "cpu")
    (bad / "config.json").write_text(json.dumps({**c, "loop": {"start": 0, "stop": 2, "times": 2}}))
    with pytest.raises(ValueError):
        ModelBase.create(str(bad), "cpu")
    (bad / "config.json").write_text(json.dumps(c))
    data = (bad / "model.safetensors").read_bytes()
    (bad / "model.safetensors").write_bytes(data[:-64])
    with pytest.raises(GGUFFormatError):
        ModelFolder(str(bad))
    (bad / "model.safetensors").write_bytes(b"\xff" * 64)
    with pytest.raises(GGUFFormatError):
        ModelFolder(str(bad))
    write_safetensors(str(bad / "model.safetensors"), {"embed": torch.zeros(4, 8, dtype=torch.bfloat16), "table": torch.arange(3, dtype=torch.int32)})
    f = ModelFolder(str(bad))
    assert f.tensors["embed"].shape == (4, 8) and f.tensor_bytes_view("table").view("<i4").tolist() == [0, 1, 2]
    with pytest.raises(KeyError):
        ModelBase.create(str(bad), "cpu")
