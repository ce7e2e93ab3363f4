"""Tifepel on a GPU: the kernels against the plain math, the engine in fp32 and bf16 against tests/tifepel_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import tifepel_cases as cases  # noqa: E402
import tifepel_oracle as oracle  # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
# sizes the tensor-core paths take as they come, beside the odd ones of tifepel_cases
WIDE = [cases.mamba(heads=8, groups=2, state=64, vdim=64, conv=4, norm_groups=4, mlp=cases.moe(ff=128, experts=8, top=3, identity=3, shared=256)),
        cases.attention(heads=4, kv=2, dim=64, vdim=128, scale=0.2, bias_max=150, mlp=cases.moe(ff=64, experts=4, top=2, identity=0, shared=64)),
        cases.mamba(heads=2, groups=1, state=128, vdim=128, conv=3, norm_groups=2, mlp=cases.moe(ff=136, experts=16, top=4, identity=8, shared=0)),
        cases.attention(heads=2, kv=2, dim=128, vdim=128, scale=0.1, bias_max=33),
        cases.mamba(heads=4, groups=4, state=128, vdim=32, conv=2, norm_groups=1)]
TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}


def ids(n, seed=0, vocab=61):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm())


def engine(cfg, t, dtype, max_pages=24, **kw):
    from prometorch_b200.serve.llm import LLMEngine
    e = LLMEngine(device="cuda", dtype=dtype, max_pages=max_pages, max_active=6, **kw)
    e.set_weights(cases.weights(cfg, t))
    return e


def layout(lens, starts, seed=0):
    """Page table of sequences in scattered pages, and positions, table rows and offsets of a batch of their rows."""
    g = torch.Generator().manual_seed(seed)
    per = [(s + n + 63) // 64 for s, n in zip(starts, lens)]
    pages = sum(per) + 3
    order = torch.randperm(pages, generator=g).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    for i, c in enumerate(per):
        table[i, :c] = torch.tensor([order.pop() for _ in range(c)])
    offs = [0]
    for x in lens:
        offs.append(offs[-1] + x)
    pos = torch.cat([torch.arange(s, s + m, dtype=torch.int32) for s, m in zip(starts, lens)])
    req = torch.cat([torch.full((m,), i, dtype=torch.int32) for i, m in enumerate(lens)])
    return g, pages, table, pos, req, offs


def batch(lens, starts, slots):
    from prometorch_b200.ops import recurrence as R
    offs = [0]
    for n in lens:
        offs.append(offs[-1] + n)
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return R.Sequences.of(offs, starts, slots, "cpu"), R.Sequences.of(offs, starts, slots, "cuda"), pos, req


# ------------------------------------------------------------------------------------------ into and between the sublayers
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,W", [(1, 64), (2, 176), (3, 50), (4, 2048), (6, 36)])
def test_pair_embedding_kernel(streams, W, dtype):
    from prometorch_b200.ops import paged as P, streams as H
    tab = [torch.randn(n, W).to(dtype) for n in (50, 14, 300)]
    lens, starts, slots = [150, 1, 65, 1], [0, 9, 3, 0], [4, 0, 2, 1]
    cpu, gpu, pos, req = batch(lens, starts, slots)
    x = torch.tensor(ids(sum(lens), 1, 50), dtype=torch.int32)
    lc = torch.tensor([[3], [7], [11], [5], [1]], dtype=torch.int32)
    lg = lc.cuda()
    e = H.PairEmbedding(*tab, 2_000_000_011, 90_001)
    g = H.PairEmbedding(*(t.cuda() for t in tab), 2_000_000_011, 90_001)
    want = H.pair_embed(x, e, streams, lc, pos, req, cpu)
    assert rel(H.pair_embed(x.cuda(), g, streams, lg, pos.cuda(), req.cuda(), gpu), want) < 1e-6 and torch.equal(lg.cpu(), lc)
    meta = torch.stack([torch.tensor([4, 8, 15]), torch.tensor([150, 0, 68]), torch.tensor([4, 1, 2])], 1).int()
    want = H.pair_embed(meta[:, 0], e, streams, lc, meta[:, 1], meta[:, 2])
    m = meta.cuda()
    assert rel(H.pair_embed(m[:, 0], g, streams, lg, m[:, 1], m[:, 2]), want) < 1e-6 and torch.equal(lg.cpu(), lc)
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,W,taps,n", [(2, 176, 4, 19), (1, 64, 1, 40), (3, 50, 2, 300), (4, 2048, 4, 300), (2, 5000, 3, 20), (5, 264, 6, 19), (16, 40, 4, 9)])
def test_step_kernel(streams, W, taps, n, dtype):
    from prometorch_b200.ops import experts as X, paged as P, residual as S, streams as H
    g = torch.Generator().manual_seed(streams)
    r = lambda *s: torch.randn(*s, generator=g)
    c = lambda t: None if t is None else t.cuda()
    link = lambda: H.Connection(r(streams), r(streams, streams), r(streams), r(W), r(taps, W), r(W))
    gpu = lambda k: H.Connection(*(c(t) for t in (k.way_in, k.mix, k.way_out, k.norm, k.conv, k.gate_bias)))
    a, b = link(), link()
    pick = X.ExpertRows(r(2 * n, W).to(dtype), torch.randperm(3 * n, generator=g).view(n, 3).int(), torch.rand(n, 3, generator=g), r(n, W).to(dtype))
    pick.index[pick.index >= 2 * n] = -1
    picked = X.ExpertRows(*(c(t) for t in (pick.y, pick.index, pick.weight, pick.h)))
    req, tol = torch.randperm(n, generator=g).int(), 3e-6 if dtype == torch.float32 else 6e-3
    for y, gate, rows_, pos0 in ((r(n, W + 8).to(dtype)[:, :W], r(3, n, W), None, 0), (r(2, n, W), r(n, W).to(dtype), pick, 2), (None, r(n, W), pick, 50)):
        x = r(n, streams, W)
        xg, pos = x.cuda(), torch.full((n,), pos0, dtype=torch.int32)
        state = r(n, taps - 1, W).to(dtype)
        sg = state.cuda()
        want = H.step(x, H.Output(a, S.Branch(gate), S.Branch(y) if y is not None else None, rows_), b, 1e-3, torch.float32, state.float().clone(), pos, req)
        got = H.step(xg, H.Output(gpu(a), S.Branch(c(gate)), S.Branch(c(y)) if y is not None else None, picked if rows_ else None), gpu(b), 1e-3, dtype, sg, c(pos), c(req))
        assert rel(xg, x) < 3e-6 and all(rel(v, w) < tol for v, w in zip(got, want))
        st = state.float().clone()
        H.step(x, None, b, 1e-3, torch.float32, st, pos, req)
        if taps > 1:
            live = min(taps - 1, pos0 + 1)                               # rows from before position 0 may hold anything
            assert rel(sg[:, taps - 1 - live:], st[:, taps - 1 - live:]) < tol
    index = torch.tensor([n - 1, 0, 3])
    assert rel(H.rows(xg, c(a.norm), 1e-3, c(index), dtype), H.rows(x, a.norm, 1e-3, index)) < tol
    assert H.step(xg, None, None, 1e-3, dtype, None, c(pos), c(req)) == (None, None)
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("add", [False, True])
@pytest.mark.parametrize("C,taps", [(64, 4), (50, 3), (264, 2), (40, 1), (16, 7)])
def test_convolution_with_bias_or_sum(C, taps, add, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    w, b = torch.randn(taps, C), None if add else torch.randn(C)
    for lens, starts in (([150, 1, 65], [0, 9, 3]), ([1, 2, 1], [0, 5, 64]), ([300], [0])):
        cpu, gpu, pos, req = batch(lens, starts, [4, 0, 2][:len(lens)])
        x, state = torch.randn(sum(lens), C + 8).to(dtype)[:, :C], torch.randn(5, taps - 1, C).to(dtype)
        sc, sg = state.float().clone(), state.cuda()
        want = R.short_conv(x.float(), w, sc, pos, req, cpu, bias=b, add=add)
        got = R.short_conv(x.cuda(), w.cuda(), sg, pos.cuda(), req.cuda(), gpu, bias=None if b is None else b.cuda(), add=add)
        assert rel(got, want) < (2e-6 if dtype == torch.float32 else 4e-3)
        if taps > 1:
            assert rel(sg[4], sc[4]) < 1e-6
        one = [t[:3].contiguous() for t in (torch.tensor([7, 0, 1]).int(), torch.tensor([1, 3, 2]).int())]
        want = R.short_conv(x[:3].float() if len(x) > 2 else x.float(), w, sc, *one, bias=b, add=add)
        got = R.short_conv(x[:3].cuda(), w.cuda(), sg, one[0].cuda(), one[1].cuda(), bias=None if b is None else b.cuda(), add=add)
        assert rel(got, want) < (2e-6 if dtype == torch.float32 else 4e-3)
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ attention
def biased(Hh, G, D, Dv, lens, starts, far=100, rel_rows=16, scale=None, seed=0):
    from prometorch_b200.ops import gated_attention as GA, window_attention as A
    g, pages, table, pos, req, offs = layout(lens, starts, seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    a = A.WindowAttention(Hh, G, D, Dv, A.UNBOUNDED, 0, scale or D ** -0.5, rel=GA.distance_bias(rnd(rel_rows, Hh) * 2, far, 30000).cuda())
    n, Dp = sum(lens), a.dim_stored
    k, v, q = torch.zeros(pages, G, 64, Dp), torch.zeros(pages, G, 64, a.vdim_stored), torch.zeros(n, Hh, Dp)
    k[..., :D], v[..., :Dv], q[..., :D] = rnd(pages, G, 64, D) * 1.5, rnd(pages, G, 64, Dv), rnd(n, Hh, D) * 1.5
    c = lambda t: t.bfloat16().cuda()
    return a, c(q), c(k), c(v), pos.cuda(), req.cuda(), table.cuda(), offs


SHAPES = [dict(Hh=8, G=2, D=128, Dv=128, lens=[200, 300], starts=[0, 0]), dict(Hh=16, G=4, D=128, Dv=128, far=1500, lens=[300], starts=[1900]),
          dict(Hh=6, G=3, D=48, Dv=80, far=20, lens=[90, 64, 1], starts=[0, 1, 170]), dict(Hh=12, G=12, D=64, Dv=64, far=64, lens=[90, 64], starts=[0, 1]),
          dict(Hh=5, G=1, D=80, Dv=100, far=9, lens=[90, 64], starts=[0, 1]), dict(Hh=40, G=1, D=64, Dv=128, far=128, lens=[190], starts=[201]),
          dict(Hh=3, G=3, D=16, Dv=64, rel_rows=2, far=2, lens=[70], starts=[0]), dict(Hh=4, G=2, D=256, Dv=160, lens=[120], starts=[103]),
          dict(Hh=2, G=1, D=40, Dv=600, lens=[20], starts=[103]), dict(Hh=2, G=2, D=64, Dv=64, far=20000, lens=[130], starts=[500])]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "h{Hh}g{G}d{D}v{Dv}".format(**s))
def test_biased_attention_kernels(shape):
    from prometorch_b200.ops import paged as P, window_attention as A
    a, q, k, v, pos, req, table, offs = biased(**shape)
    n, top = q.shape[0], int(pos.max()) + 1
    ref = A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())
    for splits in {A.pick_splits(n, a.kv_heads, a.most_keys(top)), A.pick_splits(1, a.kv_heads, a.most_keys(top)), max(1, -(-a.most_keys(top) // 128))}:
        assert rel(A.window_attention(q.float(), a, pos, req, table, k.float(), v.float(), splits, top), ref) < 5e-6
        assert rel(A.window_attention(q, a, pos, req, table, k, v, splits, top), ref) < 4e-3
    if A.tiles_supported(q, a):
        tiles = A.PromptTiles.of(offs, shape["starts"], list(range(len(offs) - 1)), "cuda")
        assert rel(A.window_attention_tiles(q, a, tiles, table, k, v), ref) < 1e-2
    P.check_status("cuda")


@pytest.mark.parametrize("far,rel_rows", [(40, 8), (64, 16), (65, 6), (200, 16)])
def test_a_bucket_that_stands_out(far, rel_rows):
    """One bucket's bias far above the others: rows return the mean of the values at its distances, in both kernels, across pages and tiles."""
    from prometorch_b200.ops import gated_attention as GA, window_attention as A
    n = 430
    a, q, k, v, pos, req, table, offs = biased(2, 1, 64, 64, [n], [0], scale=1e-5)
    tiles = A.PromptTiles.of(offs, [0], [0], "cuda")
    at = torch.arange(n)
    val = v[table[0, at.cuda() // 64].long(), 0, at.cuda() % 64].double().cpu()
    for b in range(rel_rows):
        a.rel = GA.distance_bias(torch.where(torch.arange(rel_rows)[:, None] == b, 60.0, 0.0).expand(rel_rows, 2), far, 1024).cuda()
        where = torch.tensor([oracle.bucket(d, rel_rows, far) == b for d in range(n)])
        for out in (A.window_attention(q, a, pos, req, table, k, v, 4, n), A.window_attention_tiles(q, a, tiles, table, k, v)):
            for i in (0, 1, 62, 63, 64, 65, 127, 128, 129, 200, 300, 429):
                there = [j for j in range(i + 1) if where[i - j]] or list(range(i + 1))
                want = val[there].mean(0)
                assert float((out[i].view(2, 64).double().cpu() - want).abs().max()) < 0.02, (b, i)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hh,G,D,Dv,every", [(4, 2, 128, 64, 16), (3, 1, 20, 28, 7), (2, 2, 7, 9, 1), (8, 4, 64, 80, None)])
def test_norm_per_head_and_pages(dtype, Hh, G, D, Dv, every):
    from prometorch_b200.ops import gated_attention as GA, paged as P, window_attention as A
    n = 37
    a = A.WindowAttention(Hh, G, D, Dv, A.UNBOUNDED, 0, 1.0)
    up = lambda x: -(-x // 8) * 8
    cols = (up(Hh * D), up(Hh * D) + up(G * D))
    p = torch.randn(n, cols[1] + up(G * Dv)).to(dtype)
    gain = torch.tensor([oracle.temperature(i, 0.7, every) for i in range(256)]) if every else None
    table = torch.tensor([[0, 0, 0], [2, 1, 3]], dtype=torch.int32)
    pos, req = torch.arange(n, dtype=torch.int32) + 100, torch.ones(n, dtype=torch.int32)
    out = []
    for dev in ("cpu", "cuda"):
        kp, vp = torch.full((4, G, 64, a.key_stored), 7.0, dtype=dtype, device=dev), torch.full((4, G, 64, a.vdim_stored), 7.0, dtype=dtype, device=dev)
        q = GA.head_norm_write(p.to(dev), a, None, None, 1e-3, pos.to(dev), req.to(dev), table.to(dev), kp, vp, cols=cols, gain=None if gain is None else gain.to(dev))
        out.append([t.cpu().float() for t in (q, kp, vp)])
    for want, got in zip(*out):
        assert rel(got, want) < (1e-6 if dtype == torch.float32 else 4e-3) and torch.equal(got == 0, want == 0) and torch.equal(got == 7, want == 7)
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ state-space recurrence
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("at,spread", [(-4.0, 0.5), (0.0, 3.0), (6.0, 4.0)], ids=["mild", "mixed", "harsh"])
@pytest.mark.parametrize("Hh,G,D,Dv", [(4, 2, 64, 64), (8, 1, 128, 64), (3, 1, 20, 36), (6, 3, 48, 80), (2, 1, 7, 5), (2, 1, 160, 96), (40, 20, 32, 64), (9, 1, 128, 128)])
def test_state_space_kernels(Hh, G, D, Dv, at, spread, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    g = torch.Generator().manual_seed(Hh + D)
    for lens, starts in (([150, 1, 65], [0, 9, 3]), ([1, 1, 1], [0, 5, 64]), ([300], [0]), ([40, 64, 128], [7, 0, 64])):
        n = sum(lens)
        cpu, gpu, pos, req = batch(lens, starts, [4, 0, 2][:len(lens)])
        rate, bias, skip = torch.rand(Hh, generator=g) + 0.3, torch.randn(Hh, generator=g) * spread + at, torch.randn(Hh, generator=g)
        cols = (Hh * Dv + G * D, Hh * Dv, 0)
        x = torch.randn(n, Hh * Dv + 2 * G * D, generator=g).to(dtype)
        a = (torch.randn(n, Hh + 3, generator=g) * spread).to(dtype)[:, 3:]
        start = torch.randn(5, Hh, D, Dv, generator=g)
        want_S = start.clone()
        want = R.state_space(x.float(), R.StateSpace(Hh, G, D, Dv, rate, bias, skip), cols, a.float(), want_S, pos, req, cpu)
        r = R.StateSpace(Hh, G, D, Dv, rate.cuda(), bias.cuda(), skip.cuda())
        for chunked in (None, False, True) if dtype == torch.bfloat16 and max(D, Dv) <= 128 else (None,):
            S = start.cuda()
            got = R.state_space(x.cuda(), r, cols, a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
            assert rel(got, want) < 1e-4 and rel(S, want_S) < 1e-4, (lens, chunked)
        if max(lens) == 1:
            S = start.cuda()
            assert rel(R.state_space(x.cuda(), r, cols, a.cuda(), S, pos.cuda(), req.cuda()), want) < 2e-5 and rel(S, want_S) < 2e-5
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("K,groups", [(256, 4), (108, 3), (2048, 1), (30, 30), (1100, 2)])
def test_gate_ahead_of_a_grouped_norm(K, groups, dtype):
    from prometorch_b200.ops import recurrence as R
    o, w, gate = torch.randn(19, K), torch.randn(K), torch.randn(19, K + 8).to(dtype)[:, 8:]
    kw = dict(act="silu", groups=groups, gate_first=True)
    want = R.group_norm_gate(o, w, gate, 1e-3, torch.float32, **kw)
    assert rel(R.group_norm_gate(o.cuda(), w.cuda(), gate.cuda(), 1e-3, dtype, **kw), want) < (2e-6 if dtype == torch.float32 else 4e-3)


# ------------------------------------------------------------------------------------------ experts
def expert_case(n, W, ff, E, identity, top, dtype, seed=0, spread=0.3, shared=0):
    from prometorch_b200.ops import experts as X
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, by=1.0: (torch.randn(*s, generator=g) * by).to(dtype)
    gate, up, down = ([r(*s, by=s[1] ** -0.5) for _ in range(E)] for s in ((ff, W), (ff, W), (W, ff)))
    three = [r(*s, by=s[1] ** -0.5) for s in ((shared, W), (shared, W), (W, shared))] if shared else None
    O = E + identity
    h, router, corr = r(n, W), r(O, W, by=2 * W ** -0.5), torch.randn(O, generator=g) * spread
    make = lambda dev, dt: X.Experts.of(*([t.to(dev, dt) for t in m] for m in (gate, up, down)), router.to(dev, dt), corr.to(dev), top, 1.0, softmax=True,
                                        shared=tuple(t.to(dev, dt) for t in three) if three else None)
    return h, make("cpu", torch.float32), make("cuda", dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,identity,top,shared", [(1, 4, 2, 2, 8), (7, 8, 0, 3, 0), (64, 64, 16, 8, 20), (65, 64, 16, 8, 16), (500, 5, 2, 7, 0), (300, 200, 100, 40, 9), (33, 1, 1, 1, 8),
                                                     (20, 250, 6, 4, 1), (64, 3, 60, 5, 0), (200, 300, 1, 2, 70)])
def test_softmax_routing_with_identities(n, E, identity, top, shared, dtype):
    """Against the plain choice from the same logits, except where the last score chosen and the next are all but equal."""
    from prometorch_b200.ops import experts as X, paged as P
    h, c, g = expert_case(n, 64, 8, E, identity, top, dtype, shared=shared)
    O, parts, K = E + identity, -(-shared // 8), top + -(-shared // 8)
    r = X.route(h.cuda(), g)
    z = h.double() @ c.router[:O].double().t()
    s = torch.softmax(z, -1)
    order = torch.sort(s + c.correction, descending=True)
    clear = order.values[:, top - 1] - order.values[:, top] > 1e-4 if top < O else torch.ones(n, dtype=torch.bool)
    off, token, index, weight = r.offsets.cpu(), r.token.cpu(), r.index.cpu(), r.weight.cpu()
    assert g.always == parts and off.shape[0] == E + parts + 1 and index.shape[1] == K
    held = (index >= 0).flatten()
    assert int(off[0]) == 0 and int(off[-1]) == int(held.sum()) and bool((off[1:] >= off[:-1]).all())
    assert sorted(index.flatten()[held].tolist()) == list(range(int(held.sum())))
    assert torch.equal(token[index.flatten()[held].long()], torch.arange(n).repeat_interleave(K).int()[held])
    expert = torch.where(index < 0, -1, torch.searchsorted(off[1:].contiguous(), index, right=True))
    assert torch.equal(expert[:, top:], torch.arange(E, E + parts).expand(n, parts)) and bool((weight[:, top:] == 1).all())
    for i in clear.nonzero()[:, 0].tolist():
        want = sorted(o if o < E else -1 for o in order.indices[i, :top].tolist())
        assert sorted(expert[i, :top].tolist()) == want
        assert torch.allclose(weight[i, :top].sort().values.double(), s[i, order.indices[i, :top]].sort().values, rtol=1e-4, atol=1e-9)
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,W,ff,E,identity,top,shared", [(1, 64, 128, 4, 2, 2, 64), (5, 192, 96, 8, 3, 4, 100), (40, 128, 200, 3, 1, 4, 0), (300, 128, 256, 6, 6, 2, 256),
                                                          (1500, 256, 136, 4, 1, 1, 520), (70, 50, 20, 7, 2, 3, 12), (200, 64, 33, 64, 16, 8, 33), (16, 520, 1032, 2, 0, 1, 2048)])
def test_expert_and_shared_products(n, W, ff, E, identity, top, shared, dtype):
    """Experts, and a shared expert both among them and by itself."""
    from prometorch_b200.ops import experts as X, paged as P
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for wide in {0, shared}:
        h, c, g = expert_case(n, W, ff, E, identity, top, dtype, spread=0.2, shared=wide)
        r = X.route(h.cuda(), g)
        cpu = X.Routing(*(t.cpu() for t in (r.index, r.weight, r.token, r.offsets)))
        live = int(cpu.offsets[-1])
        want = X.products(h.float(), c, X.Routing(cpu.index, cpu.weight, cpu.token.clamp(0, n - 1), cpu.offsets))[:live]
        for simt in (False, True):
            got = X.products(h.cuda(), g, r, simt=simt)[:live]
            assert torch.isfinite(got).all() and (live == 0 or rel(got, want) < tol), simt
        total = X.ExpertRows(X.products(h.cuda(), g, r), r.index, r.weight, h.cuda()).combine()
        assert rel(total, X.ExpertRows(X.products(h.float(), c, X.Routing(cpu.index, cpu.weight, cpu.token.clamp(0, n - 1), cpu.offsets)), cpu.index, cpu.weight, h).combine()) < tol
    if shared:
        three = [(torch.randn(*s) * s[1] ** -0.5).to(dtype) for s in ((shared, W), (shared, W), (W, shared))]
        got = X.run_shared(h.cuda(), X.SharedExpert.of(*(t.cuda() for t in three))).y
        want = X.run_shared(h.float(), X.SharedExpert.of(*(t.float() for t in three))).y
        assert rel((got.float().sum(0) if got.dim() == 3 else got)[:, :W], want[:, :W]) < tol
    P.check_status("cuda")


def test_only_identities():
    """Corrections send every token to identities: no expert has a row."""
    from prometorch_b200.ops import experts as X, paged as P
    for n in (3, 400):
        h, c, g = expert_case(n, 128, 64, 5, 3, 2, torch.bfloat16)
        for e in (c, g):
            e.correction[5:] = 50
        out = X.run(h.cuda(), g)
        assert bool((out.index == -1).all()) and rel(out.combine(), X.run(h.float(), c).combine()) < 1e-2
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ the model
def far_off(want, got):
    return float(((got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layers,loop,sizes", [(cases.MIXED, cases.MIXED_LOOP, dict()), (cases.EVEN, (0, 2, 2), dict(width=72, streams=2, taps=4)),
                                               (WIDE, (1, 3, 2), dict(width=96, streams=4, rel_rows=32)), (cases.MIXED, (0, 2, 2), dict(width=50, streams=5, taps=1)),
                                               (cases.EVEN, None, dict(width=36, streams=1, taps=6))],
                         ids=["mixed", "even", "wide", "odd-width", "one-stream"])
def test_prompt_decoding_and_portions(layers, loop, sizes, dtype):
    cfg, t = cases.model(layers, seed=1, loop=loop, **sizes)
    x = ids(210, 1)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    for cuts in ([210], [70] + [1] * 140, [100, 64, 2, 44], [1] + [1] * 100 + [109]):
        e = engine(cfg, t, dtype)
        s, at, out = e.open_sequence(), 0, []
        for n in cuts:
            out.append(e.feed([(s, x[at:at + n], range(n))]).clone())
            at += n
        assert far_off(want, torch.cat(out)) < TOL[dtype], cuts[:3]


def test_close_choices_of_experts_in_fp32():
    cfg, t = cases.model(cases.EVEN, seed=5, loop=(0, 3, 2), spaced=False)
    x = ids(100, 2)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.float32)
    assert far_off(want, e.feed([(e.open_sequence(), x, range(100))])) < TOL[torch.float32]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_batch_and_reuse(dtype):
    """Four sequences prefilled and decoded together, one ends early; then the freed pages and slots serve another run."""
    cfg, t = cases.model(WIDE[:4], seed=2, width=96, loop=(0, 3, 2))
    ref = {"config": cfg, "tensors": oracle.cast(t)}
    lens = [1, 64, 150, 33]
    xs = [ids(n + 50, 30 + n) for n in lens]
    want = [oracle.forward(ref, x) for x in xs]
    e = engine(cfg, t, dtype, max_pages=12)
    for _ in range(2):
        seqs = [e.open_sequence() for _ in xs]
        out = e.feed([(s, x[:n], [n - 1]) for s, x, n in zip(seqs, xs, lens)])
        assert rel(out, torch.stack([w[n - 1] for w, n in zip(want, lens)])) < TOL[dtype]
        live = [0, 1, 2, 3]
        for j in range(50):
            if j == 20:
                e.close_sequence(seqs[1])
                live.remove(1)
            out = e.feed([(seqs[i], [xs[i][lens[i] + j]], [0]) for i in live])
            assert rel(out, torch.stack([want[i][lens[i] + j] for i in live])) < TOL[dtype]
        for i in live:
            e.close_sequence(seqs[i])
        assert e.kv.pages_in_use == 0


def test_long_decoding():
    cfg, t = cases.model([cases.attention(heads=4, kv=2, dim=32, vdim=32, bias_max=300, mlp=cases.moe(ff=32, experts=4, top=2)),
                          cases.mamba(heads=4, groups=2, state=32, vdim=32)], seed=3, width=64)
    x = ids(450, 5)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.bfloat16, max_pages=8)
    s = e.open_sequence()
    out = [e.feed([(s, x[:128], [127])])] + [e.feed([(s, [x[j]], [0])]).clone() for j in range(128, 450)]
    assert rel(torch.cat(out), want[127:]) < TOL[torch.bfloat16]


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_scheduler(graphs):
    """fp32: the oracle's ids, with requests that queue and finish at different times (graphs captured while others are live)."""
    from prometorch_b200.serve.llm import GenerationConfig, LLMEngine, Request
    cfg, t = cases.model(cases.MIXED, seed=8, loop=cases.MIXED_LOOP)
    ref = {"config": cfg, "tensors": oracle.cast(t)}
    prompts = [ids(n, 20 + n) for n in (5, 40, 1, 37)]
    want = [oracle.generate(ref, p, 6 + i) for i, p in enumerate(prompts)]
    e = LLMEngine(device="cuda", dtype=torch.float32, max_pages=12, max_active=2, use_graphs=graphs)
    e.set_weights(cases.weights(cfg, t))
    for i, p in enumerate(prompts):
        e.submit_request(Request(i, p, GenerationConfig(max_new_tokens=6 + i, **GREEDY)))
    got = {}
    while e.num_active():
        e.step()
        got.update({r.request_id: r.token_ids for r in e.poll_responses()})
    assert [got[i] for i in range(4)] == want and e.kv.pages_in_use == 0
    b = LLMEngine(device="cuda", max_pages=12, max_active=2)             # bf16, sampled on the device
    b.set_weights(cases.weights(cfg, t))
    assert len(b.generate(prompts[1], GenerationConfig(max_new_tokens=8)).token_ids) == 8


def test_trace_replay(tmp_path):
    from prometorch_b200.serve.llm import save_safetensors
    cfg, t = cases.model(WIDE[:3], seed=12, width=96, loop=(0, 2, 2))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(t, str(tmp_path / "model.safetensors"))
    x = ids(130, 1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": x[:128], "want": [3, 127]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": x[128:129], "want": [0]}], "end": ["a"]}]
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    for dtype, tol in (("float32", TOL[torch.float32]), ("bfloat16", TOL[torch.bfloat16])):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert r.returncode == 0 and r.stdout.splitlines()[-1] == "done 1", r.stderr
        got = torch.cat([torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 61) for i in (0, 1)])
        assert rel(got, want[[3, 127, 128]]) < tol
