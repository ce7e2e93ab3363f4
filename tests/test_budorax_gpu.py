"""Budorax on a GPU: the kernels against the plain math, the engine in fp32 and bf16 against tests/budorax_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import budorax_cases as cases  # noqa: E402
import budorax_oracle as oracle  # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
# sizes the tensor-core paths take as they come, beside the odd ones of budorax_cases
WIDE = [cases.delta(heads=4, kv=2, dim=64, vdim=64, conv=4, mlp=cases.moe(ff=128, experts=8, top=3)),
        cases.attention(heads=4, kv=2, dim=64, vdim=128, scale=0.06, chunk=100, rot=32, mlp=cases.moe(ff=64, experts=4, top=2)),
        cases.latent(heads=4, dim=64, rot=32, vdim=64, q_rank=96, kv_rank=128, scale=0.08, mlp=cases.moe(ff=136, experts=16, top=4)),
        cases.attention(heads=2, kv=2, dim=128, vdim=128, scale=0.04, chunk=130, rot=128),
        cases.delta(heads=2, kv=2, dim=128, vdim=128, conv=3),
        cases.latent(heads=2, dim=128, rot=64, vdim=128, q_rank=64, kv_rank=512, scale=0.05)]
TOL = {torch.float32: 1e-4, torch.bfloat16: 4e-2}


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


# ------------------------------------------------------------------------------------------ attention with two maps in chunks
def two_maps(H, G, D, Dv, chunk, lens, starts, scale=None, seed=0):
    from prometorch_b200.ops import window_attention as A
    g, pages, table, pos, req, offs = layout(lens, starts, seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    a = A.WindowAttention(H, G, D, Dv, chunk, 0, scale or D ** -0.5, chunked=True, maps=2, mix=0.6, mix_gain=0.7, mix_eps=1e-4)
    n, Dp = sum(lens), a.dim_stored
    k, v, q = torch.zeros(pages, G, 64, 2, Dp), torch.zeros(pages, G, 64, a.vdim_stored), torch.zeros(n, 2 * H, Dp)
    k[..., :D], v[..., :Dv], q[..., :D] = rnd(pages, G, 64, 2, D) * 1.5, rnd(pages, G, 64, Dv), rnd(n, 2 * H, D) * 1.5
    c = lambda t: t.bfloat16().cuda()
    return a, c(q), c(k.view(pages, G, 64, 2 * Dp)), c(v), pos.cuda(), req.cuda(), table.cuda(), offs


SHAPES = [dict(H=8, G=2, D=128, Dv=128, chunk=100, lens=[200, 300], starts=[0, 0]), dict(H=16, G=4, D=128, Dv=128, chunk=1024, lens=[300], starts=[1900]),
          dict(H=6, G=3, D=48, Dv=80, chunk=64, lens=[90, 64, 1], starts=[0, 1, 170]), dict(H=12, G=12, D=64, Dv=64, chunk=33, lens=[90, 64], starts=[0, 1]),
          dict(H=5, G=1, D=80, Dv=100, chunk=50, lens=[90, 64], starts=[0, 1]), dict(H=40, G=1, D=64, Dv=128, chunk=90, lens=[190], starts=[201]),
          dict(H=3, G=3, D=16, Dv=64, chunk=1, lens=[70], starts=[0]), dict(H=7, G=7, D=20, Dv=72, chunk=300, lens=[270], starts=[510]),
          dict(H=4, G=2, D=256, Dv=160, chunk=90, lens=[120], starts=[103]), dict(H=2, G=1, D=40, Dv=600, chunk=90, lens=[20], starts=[103]),
          dict(H=4, G=4, D=128, Dv=64, chunk=1 << 30, lens=[400], starts=[64])]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "h{H}g{G}d{D}v{Dv}c{chunk}".format(**s))
def test_two_map_kernels(shape):
    from prometorch_b200.ops import paged as P, window_attention as A
    a, q, k, v, pos, req, table, offs = two_maps(**shape)
    n, top = q.shape[0], int(pos.max()) + 1
    ref = A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())
    for splits in {A.pick_splits(n, a.kv_heads, a.most_keys(top)), A.pick_splits(1, a.kv_heads, a.most_keys(top)), max(1, -(-a.most_keys(top) // 128))}:
        assert rel(A.window_attention(q.float(), a, pos, req, table, k.float(), v.float(), splits, top), ref) < 5e-6
        assert rel(A.window_attention(q, a, pos, req, table, k, v, splits, top), ref) < 4e-3
    if A.tiles_supported(q, a):
        tiles = A.PromptTiles.of(offs, shape["starts"], list(range(len(offs) - 1)), "cuda")
        assert rel(A.window_attention_tiles(q, a, tiles, table, k, v), ref) < 1e-2
    P.check_status("cuda")


@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("chunk", [31, 64, 65, 128, 129, 200])
def test_chunk_edges(chunk, maps):
    """A value that stands out counts from its place to the end of its chunk, in both kernels, at page and tile borders."""
    from prometorch_b200.ops import window_attention as A
    a, q, k, v, pos, req, table, offs = two_maps(4, 1, 64, 64, chunk, [430], [0], scale=0.05)
    if maps == 1:
        a.maps, q, k = 1, q[:, ::2].contiguous(), k[..., :64].contiguous()
    else:
        a.mix = 0.1
    tiles = A.PromptTiles.of(offs, [0], [0], "cuda")
    runs = [lambda x: A.window_attention(q, a, pos, req, table, k, x, 4, 430), lambda x: A.window_attention_tiles(q, a, tiles, table, k, x)]
    base = [f(v).float() for f in runs]
    for j in (0, 2, 30, 31, 63, 64, 65, 127, 128, 129, 130, 199, 200):
        v2 = v.clone()
        v2[table[0, j // 64], :, j % 64, 5] += 2e4
        want = [i for i in range(430) if oracle.same_chunk(i, j, chunk)]
        for f, b in zip(runs, base):
            assert ((f(v2).float() - b).abs().amax(1) > 0.5).nonzero()[:, 0].tolist() == want


@pytest.mark.parametrize("big", [4.0, 40.0])
def test_scores_that_stand_out(big):
    from prometorch_b200.ops import window_attention as A
    a, q, k, v, pos, req, table, offs = two_maps(8, 2, 64, 64, 70, [230], [0])
    q[40:44] *= big
    q[200:203] *= -big
    ref = A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())
    assert rel(A.window_attention(q.float(), a, pos, req, table, k.float(), v.float(), 2, 230), ref) < 2e-5
    assert rel(A.window_attention(q, a, pos, req, table, k, v, 2, 230), ref) < 4e-3
    assert rel(A.window_attention_tiles(q, a, A.PromptTiles.of(offs, [0], [0], "cuda"), table, k, v), ref) < 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,rot,maps", [(4, 2, 128, 64, 128, 2), (3, 1, 20, 28, 12, 2), (2, 2, 7, 9, 6, 2), (8, 4, 64, 128, 32, 1), (2, 1, 24, 40, 0, 2), (2, 1, 40, 8, 4, 2)])
def test_rotation_and_pages(dtype, H, G, D, Dv, rot, maps):
    from prometorch_b200.ops import paged as P, window_attention as A
    from prometorch_b200.ops.rotary import Rotary
    n = 37
    a = A.WindowAttention(H, G, D, Dv, 5, 0, 1.0, chunked=True, maps=maps)
    cols = (8, 8 + -(-maps * H * D // 8) * 8, 16 + -(-maps * H * D // 8) * 8 + -(-maps * G * D // 8) * 8)
    p = torch.randn(n, cols[2] + -(-G * Dv // 8) * 8).to(dtype)
    table = torch.tensor([[0, 0, 0], [2, 1, 3]], dtype=torch.int32)
    pos, req = torch.arange(n, dtype=torch.int32) + 100, torch.ones(n, dtype=torch.int32)
    out = []
    for dev in ("cpu", "cuda"):
        kp, vp = torch.full((4, G, 64, a.key_stored), 7.0, dtype=dtype, device=dev), torch.full((4, G, 64, a.vdim_stored), 7.0, dtype=dtype, device=dev)
        q = A.rope_write(p.to(dev), cols, a, Rotary(rot, 500.0, 256, dev), pos.to(dev), req.to(dev), table.to(dev), kp, vp)
        out.append([t.cpu().float() for t in (q, kp, vp)])
    for want, got in zip(*out):
        assert rel(got, want) < (1e-6 if dtype == torch.float32 else 4e-3) and torch.equal(got == 0, want == 0) and torch.equal(got == 7, want == 7)
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ latent attention
def latent_case(H, D, Rd, Dv, rank, lens, starts, seed=0, dtype=torch.bfloat16, scale=None):
    from prometorch_b200.ops import latent_attention as M
    from prometorch_b200.ops.rotary import Rotary
    g, pages, table, pos, req, offs = layout(lens, starts, seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    uk, uv = (rnd(H * D, rank) * rank ** -0.5).to(dtype), (rnd(H * Dv, rank) * rank ** -0.5).to(dtype)
    make = lambda dev: M.LatentAttention.of(H, D, Rd, Dv, rank, scale or (D + Rd) ** -0.5, uk.to(dev), uv.to(dev), Rotary(Rd, 5000.0, 4096, dev))
    a = make("cpu")
    kv = torch.zeros(pages, 1, 64, a.row)
    kv[..., :rank] = rnd(pages, 1, 64, rank)
    kv[..., a.rank_stored:a.rank_stored + Rd] = rnd(pages, 1, 64, Rd)
    n = sum(lens)
    q = rnd(n, -(-H * (D + Rd) // 8) * 8) * 2
    gate = rnd(n, H + 3).to(dtype)[:, :H]
    return a, make("cuda"), q.to(dtype), kv.to(dtype), pos, req, table, offs, gate


LATENT = [dict(H=4, D=64, Rd=32, Dv=64, rank=128, lens=[200, 300], starts=[0, 0]), dict(H=16, D=128, Rd=64, Dv=128, rank=512, lens=[130], starts=[900]),
          dict(H=3, D=20, Rd=6, Dv=28, rank=36, lens=[90, 64, 1], starts=[0, 1, 170]), dict(H=5, D=80, Rd=16, Dv=100, rank=200, lens=[70, 33], starts=[10, 129]),
          dict(H=40, D=32, Rd=16, Dv=32, rank=64, lens=[65], starts=[63]), dict(H=1, D=8, Rd=2, Dv=8, rank=7, lens=[70], starts=[0]),
          dict(H=2, D=128, Rd=64, Dv=128, rank=256, lens=[128, 2], starts=[0, 126]), dict(H=2, D=48, Rd=0, Dv=128, rank=96, lens=[150], starts=[0]),
          dict(H=2, D=160, Rd=64, Dv=144, rank=640, lens=[40], starts=[100])]


@pytest.mark.parametrize("shape", LATENT, ids=lambda s: "h{H}d{D}r{Rd}v{Dv}k{rank}".format(**s))
def test_latent_kernels(shape):
    from prometorch_b200.ops import latent_attention as M, paged as P
    c, g, q, kv, pos, req, table, offs, gate = latent_case(**shape)
    up = [t.cuda() for t in (pos, req, table)]
    top = int(pos.max()) + 1
    ref = M.latent_attention_reference(q.float(), c, pos, req, table, kv.float(), gate.float())
    one = latent_case(**shape, dtype=torch.float32)
    ref1 = M.latent_attention_reference(one[2], one[0], pos, req, table, one[3], one[8])
    assert rel(M.latent_attention(one[2].cuda(), one[1], *up, one[3].cuda(), top, one[8].cuda()), ref1) < 1e-5
    assert rel(M.latent_attention(q.cuda(), g, *up, kv.cuda(), top, gate.cuda()), ref) < 1.5e-2
    assert rel(M.latent_attention(q.cuda(), g, *up, kv.cuda(), top), M.latent_attention_reference(q.float(), c, pos, req, table, kv.float())) < 1.5e-2
    last = [t[-1:].contiguous() for t in up[:2]]
    assert rel(M.latent_attention(q[-1:].cuda(), g, *last, up[2], kv.cuda(), int(pos[-1]) + 1, gate[-1:].cuda()), ref[-1:]) < 1.5e-2
    if M.tiles_supported(g):
        context = M.PromptContext.of(offs, shape["starts"], list(range(len(offs) - 1)), "cuda")
        assert rel(M.latent_attention_tiles(q.cuda(), g, context, up[0], up[2], kv.cuda(), gate.cuda()), ref) < 1.5e-2
    P.check_status("cuda")


def test_latent_keys_far_and_near():
    """A latent that stands out is seen by every later row and by none before it, at page borders, in both kernels."""
    from prometorch_b200.ops import latent_attention as M
    _, g, q, kv, pos, req, table, offs, _ = latent_case(2, 32, 16, 32, 64, [330], [0], scale=1e-5)
    up = [t.cuda() for t in (pos, req, table)]
    context = M.PromptContext.of(offs, [0], [0], "cuda")
    runs = [lambda x: M.latent_attention(q.cuda(), g, *up, x, 330), lambda x: M.latent_attention_tiles(q.cuda(), g, context, up[0], up[2], x, None)]
    kv = kv.cuda()
    base = [f(kv).float() for f in runs]
    for j in (0, 1, 63, 64, 127, 128, 200, 329):
        x = kv.clone()
        x[table[0, j // 64], 0, j % 64, :64] += 300
        for f, b in zip(runs, base):
            assert ((f(x).float() - b).abs().amax(1) > 0.05).nonzero()[:, 0].tolist() == list(range(j, 330))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank,q_rank,Rd", [(512, 384, 64), (36, 20, 6), (7, 9, 2), (64, 128, 16), (24, 40, 0)])
def test_latent_write_kernel(dtype, rank, q_rank, Rd):
    from prometorch_b200.ops import latent_attention as M, paged as P
    from prometorch_b200.ops.rotary import Rotary
    n = 37
    cols = (8, 8 + -(-q_rank // 8) * 8)
    p, qw, kw = torch.randn(n, cols[1] + -(-(rank + Rd) // 8) * 8).to(dtype), torch.randn(q_rank), torch.randn(rank)
    table, pos, req = torch.tensor([[0, 0], [2, 1]], dtype=torch.int32), torch.arange(n, dtype=torch.int32) + 50, torch.ones(n, dtype=torch.int32)
    out = []
    for dev in ("cpu", "cuda"):
        a = M.LatentAttention.of(1, 4, Rd, 4, rank, 1.0, torch.zeros(4, rank, device=dev), torch.zeros(4, rank, device=dev), Rotary(Rd, 70.0, 128, dev))
        pages = torch.full((3, 1, 64, a.row), 7.0, dtype=dtype, device=dev)
        c = M.latent_write(p.to(dev), cols, a, qw.to(dev), kw.to(dev), 1e-3, pos.to(dev), req.to(dev), table.to(dev), pages)
        out.append([t.cpu().float() for t in (c, pages)])
    for want, got in zip(*out):
        assert rel(got, want) < (2e-6 if dtype == torch.float32 else 4e-3) and torch.equal(got == 7, want == 7)
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ delta rule, gate
def batch(lens, starts, slots):
    from prometorch_b200.ops import recurrence as R
    offs = [0]
    for n in lens:
        offs.append(offs[-1] + n)
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return R.Sequences.of(offs, starts, slots, "cpu"), R.Sequences.of(offs, starts, slots, "cuda"), pos, req


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("at,spread", [(-4.0, 0.5), (0.0, 3.0), (6.0, 4.0)], ids=["mild", "mixed", "harsh"])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 64), (2, 2, 128, 128), (3, 1, 20, 36), (6, 3, 48, 80), (2, 1, 7, 5), (2, 1, 160, 96), (20, 20, 32, 64)])
def test_delta_rule_with_one_decay_per_head(H, G, D, Dv, at, spread, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    g = torch.Generator().manual_seed(H + D)
    for lens, starts in (([150, 1, 65], [0, 9, 3]), ([1, 1, 1], [0, 5, 64]), ([300], [0]), ([40, 64, 128], [7, 0, 64])):
        n = sum(lens)
        cpu, gpu, pos, req = batch(lens, starts, [4, 0, 2][:len(lens)])
        rate, bias = torch.rand(H, generator=g) + 0.3, torch.randn(H, generator=g) * spread + at
        x, beta = torch.randn(n, 2 * G * D + H * Dv, generator=g).to(dtype), (torch.randn(n, H + 5, generator=g) * 2).to(dtype)[:, 5:]
        a = (torch.randn(n, H + 3, generator=g) * spread).to(dtype)[:, :H]
        start = torch.randn(5, H, D, Dv, generator=g)
        want_S = start.clone()
        want = R.delta_rule(x.float(), R.DeltaRule(H, G, D, Dv, rate, bias, True), beta.float(), a.float(), want_S, pos, req, cpu)
        r = R.DeltaRule(H, G, D, Dv, rate.cuda(), bias.cuda(), True)
        for chunked in (None, False, True) if dtype == torch.bfloat16 and max(D, Dv) <= 128 else (None,):
            S = start.cuda()
            got = R.delta_rule(x.cuda(), r, beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
            assert rel(got, want) < 1e-4 and rel(S, want_S) < 1e-4, (lens, chunked)
        if max(lens) == 1:
            S = start.cuda()
            assert rel(R.delta_rule(x.cuda(), r, beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda()), want) < 2e-5 and rel(S, want_S) < 2e-5
    P.check_status("cuda")


def test_delta_rule_repeated_keys():
    """The same key over and over with beta near 1: the triangular system of a chunk is far from the identity."""
    from prometorch_b200.ops import recurrence as R
    cpu, gpu, pos, req = batch([200], [0], [0])
    x, beta, a = torch.randn(200, 6 * 64).bfloat16(), (torch.randn(200, 2) + 6).bfloat16(), torch.randn(200, 2).bfloat16()
    x[:, 2 * 64:4 * 64] = x[:1, 2 * 64:4 * 64]
    rate, bias = torch.ones(2), torch.full((2,), -9.0)
    want_S = torch.zeros(1, 2, 64, 64)
    want = R.delta_rule(x.float(), R.DeltaRule(2, 2, 64, 64, rate, bias, True), beta.float(), a.float(), want_S, pos, req, cpu)
    for chunked in (False, True):
        S = torch.zeros(1, 2, 64, 64, device="cuda")
        got = R.delta_rule(x.cuda(), R.DeltaRule(2, 2, 64, 64, rate.cuda(), bias.cuda(), True), beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
        assert rel(got, want) < 2e-4 and rel(S, want_S) < 2e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gs,groups", [(64, 4), (36, 3), (1000, 1)])
def test_silu_gate_kernel(gs, groups, dtype):
    from prometorch_b200.ops import recurrence as R
    o, w, gate = torch.randn(19, gs * groups), torch.randn(gs), torch.randn(19, gs * groups + 8).to(dtype)[:, 8:]
    want = R.group_norm_gate(o, w, gate, 1e-3, torch.float32, act="silu")
    assert rel(R.group_norm_gate(o.cuda(), w.cuda(), gate.cuda(), 1e-3, dtype, act="silu"), want) < (2e-6 if dtype == torch.float32 else 4e-3)


# ------------------------------------------------------------------------------------------ norms, experts
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,n", [(64, 19), (2048, 19), (4096, 700), (50, 19), (264, 1500), (4104, 30)])
def test_tanh_norm_kernels(dtype, W, n):
    from prometorch_b200.ops import experts as X, residual as S, tanh_norm as T
    x, y, z, table = torch.randn(n, W), torch.randn(n, W).to(dtype), torch.randn(3, n, W), torch.randn(9, W).to(dtype)
    tok = torch.randint(0, 9, (n,), dtype=torch.int32)
    pick = X.ExpertRows(torch.randn(n * 3, W).to(dtype), torch.randperm(n * 3).view(n, 3).int(), torch.rand(n, 3))
    c = lambda t: t.cuda()
    norm = lambda a: T.TanhNorm(a, torch.randn(W), torch.randn(W))
    gpu = lambda m: T.TanhNorm(m.alpha, c(m.w), c(m.b))
    post, pre = norm(0.01), norm(1.7)                                    # small arguments keep their relative accuracy
    post.b.zero_()
    picked = X.ExpertRows(c(pick.y), c(pick.index), c(pick.weight))
    for a, b, again in ((S.Branch(y), S.Branch(c(y)), False), (S.Branch(z), S.Branch(c(z)), True), (pick, picked, False), (pick, picked, True)):
        xc, xg = torch.zeros(n, W), torch.zeros(n, W, device="cuda")
        want = T.residual(xc, a, post, pre, torch.float32, (tok, table.float()) if again else None)
        got = T.residual(xg, b, gpu(post), gpu(pre), dtype, (c(tok), c(table)) if again else None)
        assert rel(xg, xc) < 2e-6 and rel(got, want) < (2e-6 if dtype == torch.float32 else 4e-3)
        assert T.residual(xg, b, gpu(post), None, dtype) is None
    index = torch.tensor([n - 1, 0, 3])
    assert rel(T.rows(c(x), gpu(pre), c(index), dtype), T.rows(x, pre, index)) < (2e-6 if dtype == torch.float32 else 4e-3)
    assert rel(T.softcap(c(x * 20)[:, :W - 3], 7.0), T.softcap(x[:, :W - 3] * 20, 7.0)) < 1e-6


def expert_case(n, W, ff, E, top, dtype, seed=0, spread=1.0):
    from prometorch_b200.ops import experts as X
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, by=1.0: (torch.randn(*s, generator=g) * by).to(dtype)
    gate, up, down = ([r(*s, by=s[1] ** -0.5) for _ in range(E)] for s in ((ff, W), (ff, W), (W, ff)))
    h, router, corr = r(n, W), r(E, W, by=2 * W ** -0.5), torch.randn(E, generator=g) * spread
    make = lambda dev, dt: X.Experts.of(*([t.to(dev, dt) for t in m] for m in (gate, up, down)), router.to(dev, dt), corr.to(dev), top, 1.7)
    return h, make("cpu", torch.float32), make("cuda", dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,top", [(1, 4, 2), (7, 8, 3), (64, 64, 8), (65, 64, 8), (500, 5, 5), (300, 300, 40), (33, 1, 1), (20, 256, 4)])
def test_routing(n, E, top, dtype):
    """Against the plain choice from the same logits, except where the last score chosen and the next are all but equal."""
    from prometorch_b200.ops import experts as X, paged as P
    h, c, g = expert_case(n, 64, 8, E, top, dtype)
    r = X.route(h.cuda(), g)
    z = h.double() @ c.router[:E].double().t()
    s = torch.sigmoid(z)
    order = torch.sort(s + c.correction, descending=True)
    clear = order.values[:, top - 1] - order.values[:, top] > 1e-4 if top < E else torch.ones(n, dtype=torch.bool)
    at, off, token, index = r.offsets.cpu(), r.offsets.cpu(), r.token.cpu(), r.index.cpu()
    assert int(at[0]) == 0 and int(at[E]) == n * top and bool((at[1:] >= at[:-1]).all())
    assert sorted(index.flatten().tolist()) == list(range(n * top))
    assert torch.equal(token[index.flatten().long()], torch.arange(n).repeat_interleave(top).int())
    expert = torch.searchsorted(off[1:].contiguous(), index, right=True)
    for i in clear.nonzero()[:, 0].tolist():
        assert sorted(expert[i].tolist()) == sorted(order.indices[i, :top].tolist())
    w = s.gather(1, expert.long())
    assert rel(r.weight, w / w.sum(1, keepdim=True) * 1.7) < 1e-5
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,W,ff,E,top", [(1, 64, 128, 4, 2), (5, 192, 96, 8, 4), (32, 256, 64, 16, 4), (40, 128, 200, 3, 3), (300, 128, 256, 6, 2), (1500, 256, 136, 4, 1),
                                          (70, 50, 20, 7, 3), (200, 64, 33, 64, 8), (16, 520, 1032, 2, 1), (1000, 512, 384, 5, 2)])
def test_expert_products(n, W, ff, E, top, dtype):
    from prometorch_b200.ops import experts as X, paged as P
    h, c, g = expert_case(n, W, ff, E, top, dtype, spread=0.2)
    r = X.route(h.cuda(), g)
    cpu = X.Routing(*(t.cpu() for t in (r.index, r.weight, r.token, r.offsets)))
    want = X.products(h.float(), c, cpu)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for simt in (False, True):
        got = X.products(h.cuda(), g, r, simt=simt)
        assert torch.isfinite(got).all() and rel(got, want) < tol, simt
    P.check_status("cuda")


def test_all_rows_at_one_expert():
    """Corrections send every token to the same expert; the others have no rows at all."""
    from prometorch_b200.ops import experts as X
    for n in (3, 400):
        h, c, g = expert_case(n, 128, 64, 9, 1, torch.bfloat16)
        for e in (c, g):
            e.correction[5] = 50
        out = X.run(h.cuda(), g)
        assert rel(X.ExpertRows(out.y.cpu(), out.index.cpu(), out.weight.cpu()).combine(), X.run(h.float(), c).combine()) < 1e-2


# ------------------------------------------------------------------------------------------ the model
def far(want, got):
    return float(((got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layers,width,loop", [(cases.MIXED, 48, cases.MIXED_LOOP), (cases.EVEN, 64, (0, 2, 3)), (WIDE, 96, (1, 3, 2)), (cases.MIXED, 50, (0, 2, 2))],
                         ids=["mixed", "even", "wide", "odd-width"])
def test_prompt_decoding_and_portions(layers, width, loop, dtype):
    cfg, t = cases.model(layers, seed=1, width=width, loop=loop)
    x = ids(210, 1)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    for cuts in ([210], [70] + [1] * 140, [100, 64, 2, 44], [1] + [1] * 100 + [109]):
        e = engine(cfg, t, dtype)
        s, at, out = e.open_sequence(), 0, []
        for n in cuts:
            out.append(e.feed([(s, x[at:at + n], range(n))]).clone())
            at += n
        assert far(want, torch.cat(out)) < TOL[dtype], cuts[:3]


def test_close_choices_of_experts_in_fp32():
    cfg, t = cases.model(cases.EVEN, seed=5, loop=(0, 3, 2), spaced=False)
    x = ids(100, 2)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.float32)
    assert far(want, e.feed([(e.open_sequence(), x, range(100))])) < TOL[torch.float32]


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


def test_long_decoding_in_a_small_pool():
    cfg, t = cases.model([cases.attention(heads=4, kv=2, dim=32, vdim=32, chunk=100, rot=16, mlp=cases.moe(ff=32, experts=4, top=2)), cases.delta(heads=2, kv=1, dim=32, vdim=32)],
                         seed=3, width=64)
    x = ids(450, 5)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.bfloat16, max_pages=4)
    s = e.open_sequence()
    out = [e.feed([(s, x[:128], [127])])] + [e.feed([(s, [x[j]], [0])]).clone() for j in range(128, 450)]
    assert rel(torch.cat(out), want[127:]) < TOL[torch.bfloat16] and e.kv.pages_in_use <= 3


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
    for dtype, tol in (("float32", 1e-4), ("bfloat16", 4e-2)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert r.returncode == 0 and r.stdout.splitlines()[-1] == "done 1", r.stderr
        got = torch.cat([torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 61) for i in (0, 1)])
        assert rel(got, want[[3, 127, 128]]) < tol
