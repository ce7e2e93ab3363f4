"""Gelutar on a GPU: the kernels against the plain math, the engine in fp32 and bf16 against tests/gelutar_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gelutar_cases as cases  # noqa: E402
import gelutar_oracle as oracle  # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
# sizes the tensor-core paths take as they come, beside the odd ones of gelutar_cases
WIDE = [cases.parallel(heads=8, kv=2, dim=64, vdim=64, scale=0.06, window=100, keep=70, d_heads=4, d_kv=2, d_dim=64, d_vdim=64, ff=128),
        cases.lightning(heads=4, dim=64, vdim=64, ff=128),
        cases.parallel(heads=4, kv=4, dim=128, vdim=128, scale=0.04, window=130, keep=3, d_heads=2, d_kv=2, d_dim=128, d_vdim=128, conv=3, ff=0),
        cases.lightning(heads=2, dim=128, vdim=128, decay=[0.8, 0.999], ff=64)]
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


# ------------------------------------------------------------------------------------------ window attention
def attention_case(H, G, D, Dv, W, keep, lens, starts, seed=0, scale=None):
    from prometorch_b200.ops import window_attention as A
    g = torch.Generator().manual_seed(seed)
    per = [(s + n + 63) // 64 for s, n in zip(starts, lens)]
    pages = sum(per) + 3
    order = torch.randperm(pages, generator=g).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    for i, c in enumerate(per):
        table[i, :c] = torch.tensor([order.pop() for _ in range(c)])
    rnd = lambda *s: torch.randn(*s, generator=g)
    a = A.WindowAttention(H, G, D, Dv, W, keep, scale or D ** -0.5, (rnd(H) * 2).cuda())
    n = sum(lens)
    k, v, q = torch.zeros(pages, G, 64, a.dim_stored), torch.zeros(pages, G, 64, a.vdim_stored), torch.zeros(n, H, a.dim_stored)
    k[..., :D], v[..., :Dv], q[..., :D] = rnd(pages, G, 64, D) * 1.5, rnd(pages, G, 64, Dv), rnd(n, H, D) * 1.5
    offs = [0]
    for x in lens:
        offs.append(offs[-1] + x)
    pos = torch.cat([torch.arange(s, s + m, dtype=torch.int32) for s, m in zip(starts, lens)])
    req = torch.cat([torch.full((m,), i, dtype=torch.int32) for i, m in enumerate(lens)])
    gate = rnd(n, H + 3).bfloat16().cuda()[:, :H]
    return a, q.bfloat16().cuda(), k.bfloat16().cuda(), v.bfloat16().cuda(), pos.cuda(), req.cuda(), table.cuda(), offs, gate


SHAPES = [dict(H=8, G=2, D=128, Dv=128, W=100, keep=4, lens=[200, 300], starts=[0, 0]), dict(H=16, G=4, D=128, Dv=128, W=1024, keep=64, lens=[300], starts=[1900]),
          dict(H=6, G=3, D=48, Dv=80, W=64, keep=70, lens=[90, 64, 1], starts=[0, 1, 170]), dict(H=12, G=12, D=64, Dv=64, W=33, keep=1, lens=[90, 64], starts=[0, 1]),
          dict(H=5, G=1, D=80, Dv=100, W=50, keep=0, lens=[90, 64], starts=[0, 1]), dict(H=20, G=1, D=64, Dv=128, W=90, keep=20, lens=[190], starts=[201]),
          dict(H=3, G=3, D=16, Dv=64, W=1, keep=0, lens=[70], starts=[0]), dict(H=3, G=3, D=16, Dv=64, W=1, keep=130, lens=[300], starts=[0]),
          dict(H=7, G=7, D=20, Dv=72, W=300, keep=9, lens=[270], starts=[510]), dict(H=9, G=1, D=24, Dv=12, W=200, keep=5, lens=[70], starts=[329]),
          dict(H=4, G=2, D=256, Dv=160, W=90, keep=3, lens=[120], starts=[103]), dict(H=8, G=4, D=96, Dv=64, W=257, keep=128, lens=[300, 9], starts=[0, 657]),
          dict(H=4, G=4, D=128, Dv=64, W=1 << 30, keep=0, lens=[400], starts=[64])]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "h{H}g{G}d{D}v{Dv}w{W}k{keep}".format(**s))
def test_attention_kernels(shape):
    from prometorch_b200.ops import paged as P, window_attention as A
    a, q, k, v, pos, req, table, offs, gate = attention_case(**shape)
    n, top = q.shape[0], int(pos.max()) + 1
    for s in (a.sink, None):
        a.sink = s
        ref = A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float(), gate)
        for splits in {A.pick_splits(n, a.kv_heads, a.most_keys(top)), A.pick_splits(1, a.kv_heads, a.most_keys(top))}:
            assert rel(A.window_attention(q.float(), a, pos, req, table, k.float(), v.float(), splits, top, gate.float() if gate is not None else None), ref) < 2e-6
            assert rel(A.window_attention(q, a, pos, req, table, k, v, splits, top, gate), ref) < 4e-3
        if A.tiles_supported(q, a):
            tiles = A.PromptTiles.of(offs, shape["starts"], list(range(len(offs) - 1)), "cuda")
            assert rel(A.window_attention_tiles(q, a, tiles, table, k, v, gate), ref) < 6e-3
        gate = None
        assert rel(A.window_attention(q, a, pos, req, table, k, v, A.pick_splits(n, a.kv_heads, a.most_keys(top)), top),
                   A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())) < 4e-3
    P.check_status("cuda")


@pytest.mark.parametrize("W,keep", [(31, 3), (64, 0), (65, 64), (128, 65), (129, 127), (200, 130)])
def test_window_and_kept_tokens_edges(W, keep):
    """A value that stands out counts exactly where its key is seen, in both kernels, at page and tile borders."""
    from prometorch_b200.ops import window_attention as A
    a, q, k, v, pos, req, table, offs, _ = attention_case(4, 1, 64, 64, W, keep, [430], [0], scale=0.05)
    tiles = A.PromptTiles.of(offs, [0], [0], "cuda")
    runs = [lambda x: A.window_attention(q, a, pos, req, table, k, x, 4, 430)]
    if A.tiles_supported(q, a):
        runs.append(lambda x: A.window_attention_tiles(q, a, tiles, table, k, x))
    base = [f(v).float() for f in runs]
    for j in (0, 2, 3, 63, 64, 65, 100, 126, 127, 128, 129, 130, 200):
        v2 = v.clone()
        v2[table[0, j // 64], :, j % 64] += 2e4
        want = [i for i in range(430) if oracle.visible(i, j, W, keep)]
        for f, b in zip(runs, base):
            assert ((f(v2).float() - b).abs().amax(1) > 2.0).nonzero()[:, 0].tolist() == want


@pytest.mark.parametrize("big", [4.0, 40.0])
def test_scores_that_stand_out(big):
    from prometorch_b200.ops import window_attention as A
    a, q, k, v, pos, req, table, offs, gate = attention_case(8, 2, 64, 64, 70, 5, [230], [0])
    q[40:44] *= big
    q[200:203] *= -big
    ref = A.window_attention_reference(q.float(), a, pos, req, table, k.float(), v.float(), gate)
    assert rel(A.window_attention(q.float(), a, pos, req, table, k.float(), v.float(), 1, 230, gate.float()), ref) < 2e-5
    assert rel(A.window_attention(q, a, pos, req, table, k, v, 1, 230, gate), ref) < 4e-3
    if A.tiles_supported(q, a):
        assert rel(A.window_attention_tiles(q, a, A.PromptTiles.of(offs, [0], [0], "cuda"), table, k, v, gate), ref) < 6e-3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 128, 64), (3, 1, 20, 28), (2, 2, 7, 9), (32, 8, 128, 128)])
def test_projection_norm_kernel(dtype, H, G, D, Dv):
    from prometorch_b200.ops import paged as P, window_attention as A
    n, eps = 37, 1e-3
    a = A.WindowAttention(H, G, D, Dv, 5, 0, 1.0)
    up = lambda x: -(-x // 8) * 8
    cols = (8, 8 + up(H * D), 8 + up(H * D) + up(G * D))
    p = torch.randn(n, cols[2] + up(G * Dv) + 8).to(dtype)
    qw, kw = torch.randn(H * D), torch.randn(G * D)
    pos, req = torch.arange(40, 40 + n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)
    table = torch.tensor([[0, 0], [3, 1]], dtype=torch.int32)
    pages = [torch.full((4, G, 64, s), 5.0, dtype=dtype) for s in (a.dim_stored, a.vdim_stored)]
    gpu = [x.cuda() for x in pages]
    want = A.proj_norm_write(p, cols, a, qw, kw, eps, pos, req, table, *pages)
    got = A.proj_norm_write(p.cuda(), cols, a, qw.cuda(), kw.cuda(), eps, pos.cuda(), req.cuda(), table.cuda(), *gpu)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    assert rel(got, want) < tol and all(rel(x, y) < tol for x, y in zip(gpu, pages))
    P.check_status("cuda")


# ------------------------------------------------------------------------------------------ recurrences
def batch(lens, starts, slots):
    from prometorch_b200.ops import recurrence as R
    offs = [0]
    for x in lens:
        offs.append(offs[-1] + x)
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return R.Sequences.of(offs, starts, slots, "cpu"), R.Sequences.of(offs, starts, slots, "cuda"), pos, req


BATCHES = [([70], [0]), ([1, 130, 64, 2, 200], [0, 7, 0, 64, 65]), ([1, 1, 1], [0, 3, 90]), ([33, 500], [100, 0])]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,taps", [(64, 4), (37, 3), (256, 1), (40, 7)])
def test_short_convolution_kernel(C, taps, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    w = torch.randn(taps, C)
    for lens, starts in BATCHES:
        n, slots = sum(lens), [4, 0, 2, 5, 3][:len(lens)]
        cpu, gpu, pos, req = batch(lens, starts, slots)
        x = torch.randn(n, C + 8).to(dtype)[:, 8 if C % 8 == 0 else 3:][:, :C]
        state = torch.randn(6, taps - 1, C).to(dtype)
        sg = state.cuda()
        for seqs in ((cpu, gpu), (None, None)) if max(lens) == 1 else ((cpu, gpu),):
            want = R.short_conv(x, w, state, pos, req, seqs[0])
            got = R.short_conv(x.cuda(), w.cuda(), sg, pos.cuda(), req.cuda(), seqs[1])
            assert rel(got, want) < (1e-6 if dtype == torch.float32 else 3e-3) and torch.equal(sg.cpu(), state)
    P.check_status("cuda")


def delta_inputs(H, G, D, Dv, n, dtype, shift=-2.0, spread=2.0, seed=0):
    from prometorch_b200.ops import recurrence as R
    g = torch.Generator().manual_seed(seed)
    r = R.DeltaRule(H, G, D, Dv, torch.rand(H, generator=g) * 2 + 0.1, torch.randn(H * D, generator=g) * spread + shift)
    x, beta = torch.randn(n, 2 * G * D + H * Dv, generator=g).to(dtype), (torch.randn(n, H, generator=g) * 2).to(dtype)
    return r, x, beta, torch.randn(n, H * D + 8, generator=g)[:, :H * D]


def on_gpu(r):
    import dataclasses
    return dataclasses.replace(r, **{k: v.cuda() for k, v in vars(r).items() if torch.is_tensor(v)})


def modes(dtype, lens):
    """(chunked, tolerance): token by token, and in chunks for bf16 prompts."""
    return [(False, 2e-5)] + ([(True, 1e-4)] if dtype == torch.bfloat16 and max(lens) > 1 else [])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 64), (2, 2, 128, 128), (3, 1, 20, 36), (2, 1, 48, 80), (1, 1, 8, 5), (2, 2, 96, 32), (1, 1, 300, 40)])
def test_delta_rule_kernels(H, G, D, Dv, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    for lens, starts in BATCHES:
        n, slots = sum(lens), [4, 0, 2, 5, 3][:len(lens)]
        cpu, gpu, pos, req = batch(lens, starts, slots)
        r, x, beta, a = delta_inputs(H, G, D, Dv, n, dtype)
        start = torch.randn(6, H, D, Dv)
        want_S = start.clone()
        want = R.delta_rule(x, r, beta, a, want_S, pos, req, cpu)
        for chunked, tol in modes(dtype, lens):
            S = start.cuda()
            got = R.delta_rule(x.cuda(), on_gpu(r), beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
            assert rel(got, want) < tol and rel(S, want_S) < tol, (lens, chunked)
        if max(lens) == 1:
            S = start.cuda()
            got = R.delta_rule(x.cuda(), on_gpu(r), beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda())
            assert rel(got, want) < 2e-5 and rel(S, want_S) < 2e-5
    P.check_status("cuda")


@pytest.mark.parametrize("shift,spread", [(-12.0, 1.0), (0.0, 0.5), (8.0, 6.0), (60.0, 40.0)])
def test_delta_rule_decays(shift, spread):
    """From nearly none to states that are gone within one token, with both kinds of channel side by side."""
    from prometorch_b200.ops import recurrence as R
    lens, starts = [150, 65], [0, 9]
    cpu, gpu, pos, req = batch(lens, starts, [1, 0])
    r, x, beta, a = delta_inputs(2, 1, 64, 64, sum(lens), torch.bfloat16, shift, spread)
    start = torch.randn(2, 2, 64, 64)
    want_S = start.clone()
    want = R.delta_rule(x, r, beta, a, want_S, pos, req, cpu)
    for chunked in (False, True):
        S = start.cuda()
        got = R.delta_rule(x.cuda(), on_gpu(r), beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
        assert torch.isfinite(got).all() and rel(got, want) < 1e-4 and rel(S, want_S) < 1e-4


@pytest.mark.parametrize("H,G,D,Dv,rank", [(4, 2, 64, 64, 24), (2, 2, 128, 128, 128), (3, 1, 20, 36, 8), (2, 1, 96, 48, 256), (2, 1, 96, 48, 264)])
def test_delta_rule_low_rank_decays(H, G, D, Dv, rank):
    """The decays' projection given as its two factors."""
    from prometorch_b200.ops import recurrence as R
    lens, starts = [150, 1, 65], [0, 9, 3]
    cpu, gpu, pos, req = batch(lens, starts, [1, 0, 2])
    r, x, beta, _ = delta_inputs(H, G, D, Dv, sum(lens), torch.bfloat16)
    low, w = torch.randn(sum(lens), rank + 16).bfloat16()[:, 8:8 + rank], (torch.randn(-(-H * D // 8) * 8, rank) * rank ** -0.5).bfloat16()
    start = torch.randn(3, H, D, Dv)
    want_S = start.clone()
    want = R.delta_rule(x, r, beta, (low, w), want_S, pos, req, cpu)
    for chunked in (False, True):
        S = start.cuda()
        got = R.delta_rule(x.cuda(), on_gpu(r), beta.cuda(), (low.cuda(), w.cuda()), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
        assert rel(got, want) < 1e-4 and rel(S, want_S) < 1e-4


def test_delta_rule_repeated_keys():
    """The same key over and over with beta near 1: the triangular system of a chunk is far from the identity."""
    from prometorch_b200.ops import recurrence as R
    lens, starts = [200], [0]
    cpu, gpu, pos, req = batch(lens, starts, [0])
    r, x, beta, a = delta_inputs(2, 2, 64, 64, 200, torch.bfloat16, -9.0, 0.5)
    x[:, 2 * 64:4 * 64] = x[:1, 2 * 64:4 * 64]
    beta += 6
    want_S = torch.zeros(1, 2, 64, 64)
    want = R.delta_rule(x, r, beta, a, want_S, pos, req, cpu)
    for chunked in (False, True):
        S = torch.zeros(1, 2, 64, 64, device="cuda")
        got = R.delta_rule(x.cuda(), on_gpu(r), beta.cuda(), a.cuda(), S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
        assert rel(got, want) < 2e-4 and rel(S, want_S) < 2e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,Dv", [(4, 64, 64), (2, 128, 128), (3, 20, 36), (5, 48, 80), (1, 8, 5), (2, 96, 32)])
def test_decay_attention_kernels(H, D, Dv, dtype):
    from prometorch_b200.ops import paged as P, recurrence as R
    for lens, starts in BATCHES:
        n, slots = sum(lens), [4, 0, 2, 5, 3][:len(lens)]
        cpu, gpu, pos, req = batch(lens, starts, slots)
        r = R.DecayAttention(H, D, Dv, torch.tensor([1.0, 0.0, 0.999, 0.6, 0.95][:H]))
        up = lambda v: -(-v // 8) * 8
        cols = (8, 8 + up(H * D), 8 + 2 * up(H * D))
        x = torch.randn(n, cols[2] + up(H * Dv)).to(dtype)
        start = torch.randn(6, H, D, Dv)
        want_S = start.clone()
        want = R.decay_attention(x, r, cols, want_S, pos, req, cpu)
        for chunked, tol in modes(dtype, lens):
            S = start.cuda()
            got = R.decay_attention(x.cuda(), on_gpu(r), cols, S, pos.cuda(), req.cuda(), gpu, chunked=chunked)
            assert rel(got, want) < tol and rel(S, want_S) < tol, (lens, chunked)
        if max(lens) == 1:
            S = start.cuda()
            got = R.decay_attention(x.cuda(), on_gpu(r), cols, S, pos.cuda(), req.cuda())
            assert rel(got, want) < 2e-5 and rel(S, want_S) < 2e-5
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gs,groups", [(64, 4), (128, 16), (36, 3), (2048, 1), (1000, 1), (5, 2)])
def test_group_norm_gate_kernel(gs, groups, dtype):
    from prometorch_b200.ops import recurrence as R
    o, w = torch.randn(19, gs * groups), torch.randn(gs)
    for gt in (torch.float32, torch.bfloat16):
        gate = torch.randn(19, gs * groups + 8).to(gt)[:, 8:]
        want = R.group_norm_gate(o, w, gate, 1e-3, torch.float32)
        assert rel(R.group_norm_gate(o.cuda(), w.cuda(), gate.cuda(), 1e-3, dtype), want) < (2e-6 if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,n", [(64, 19), (2048, 19), (4096, 19), (9000, 19), (50, 19), (264, 1500), (2048, 1100), (4096, 2500), (4104, 1030)])
def test_residual_norm_kernel(dtype, W, n):
    from prometorch_b200.ops import residual as S
    x, y, z = torch.randn(n, W), torch.randn(n, W).to(dtype), torch.randn(3, n, W)
    w = [torch.randn(W) for _ in range(3)]
    c = lambda t: t.cuda()
    for make in (lambda f: [S.Branch(f(y))], lambda f: [S.Branch(f(y), 0.5, f(w[0])), S.Branch(f(y), 0.25, f(w[1]))], lambda f: [S.Branch(f(y), 0.5, f(w[0])), S.Branch(f(z), 0.25, f(w[1]))], lambda f: [S.Branch(f(z))], lambda f: [S.Branch(f(y), 1.0), S.Branch(f(y), 2.0, f(w[0]))]):
        xc, xg = x.clone(), x.cuda()
        want = S.residual_norm(xc, make(lambda t: t), 1e-3, w[2], torch.float32)
        got = S.residual_norm(xg, make(c), 1e-3, c(w[2]), dtype)
        assert rel(xg, xc) < 1e-6 and rel(got, want) < (2e-6 if dtype == torch.float32 else 4e-3)
        assert S.residual_norm(xg, make(c), 1e-3) is None


@pytest.mark.parametrize("M", [1, 5, 40, 100, 300])
def test_projections_around_the_stream(M):
    from prometorch_b200.ops import gemm, residual as S
    K, Nn = 256, 512
    a, w, up = torch.randn(M, K).bfloat16(), (torch.randn(Nn, K) * K ** -0.5).bfloat16(), (torch.randn(192, K) * K ** -0.5).bfloat16()
    x = torch.randn(M, Nn)
    g = torch.randn(Nn)
    with torch.no_grad():
        xg = x.cuda()
        h = S.residual_norm(xg, [S.linear_branch(a.cuda(), w.cuda(), 0.5, g.cuda()), S.linear_branch(a.cuda(), w.cuda())], 1e-4, g.cuda(), torch.bfloat16)
        y = a.double() @ w.double().t()
        want = x.double() + y + 0.5 * oracle.plain_norm(y, g.double(), 1e-4)
        assert rel(xg, want) < 3e-3 and rel(h, oracle.plain_norm(want, g.double(), 1e-4)) < 6e-3
        assert rel(gemm.linear_relu2(a.cuda(), up.cuda()), torch.relu(a.double() @ up.double().t()) ** 2) < 4e-3


# ------------------------------------------------------------------------------------------ the model
def far(want, got):
    return float(((got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layers,width", [(cases.MIXED, 48), (cases.EVEN, 64), (WIDE, 96), (cases.MIXED, 50)], ids=["mixed", "even", "wide", "odd-width"])
def test_prompt_decoding_and_portions(layers, width, dtype):
    cfg, t = cases.model(layers, seed=1, width=width)
    x = ids(210, 1)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    for cuts in ([210], [70] + [1] * 140, [100, 64, 2, 44], [1] + [1] * 100 + [109]):
        e = engine(cfg, t, dtype)
        s, at, out = e.open_sequence(), 0, []
        for n in cuts:
            out.append(e.feed([(s, x[at:at + n], range(n))]))
            at += n
        assert far(want, torch.cat(out)) < TOL[dtype], cuts[:3]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_batch_and_reuse(dtype):
    """Four sequences prefilled and decoded together, one ends early; then the freed pages and slots serve another run."""
    cfg, t = cases.model(WIDE, seed=2, width=96)
    ref = {"config": cfg, "tensors": oracle.cast(t)}
    lens = [1, 64, 150, 33]
    xs = [ids(n + 70, 30 + n) for n in lens]
    want = [oracle.forward(ref, x) for x in xs]
    e = engine(cfg, t, dtype, max_pages=12)
    for _ in range(2):
        seqs = [e.open_sequence() for _ in xs]
        out = e.feed([(s, x[:n], [n - 1]) for s, x, n in zip(seqs, xs, lens)])
        assert rel(out, torch.stack([w[n - 1] for w, n in zip(want, lens)])) < TOL[dtype]
        live = [0, 1, 2, 3]
        for j in range(70):
            if j == 20:
                e.close_sequence(seqs[1])
                live.remove(1)
            out = e.feed([(seqs[i], [xs[i][lens[i] + j]], [0]) for i in live])
            assert rel(out, torch.stack([want[i][lens[i] + j] for i in live])) < TOL[dtype]
        for i in live:
            e.close_sequence(seqs[i])
        assert e.kv.pages_in_use == 0


def test_long_decoding_in_a_small_pool():
    cfg, t = cases.model([cases.parallel(heads=4, kv=2, dim=32, vdim=32, window=50, keep=5, d_heads=2, d_kv=1, d_dim=32, d_vdim=32, ff=64), cases.lightning(heads=2, dim=32, vdim=32)], seed=3)
    x = ids(500, 5)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.bfloat16, max_pages=4)
    s = e.open_sequence()
    out = [e.feed([(s, x[:128], [127])])] + [e.feed([(s, [x[j]], [0])]) for j in range(128, 500)]
    assert rel(torch.cat(out), want[127:]) < TOL[torch.bfloat16] and e.kv.pages_in_use <= 3


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_scheduler(graphs):
    """fp32: the oracle's ids, with requests that queue and finish at different times (graphs captured while others are live)."""
    from prometorch_b200.serve.llm import GenerationConfig, LLMEngine, Request
    cfg, t = cases.model(cases.MIXED, seed=8)
    ref = {"config": cfg, "tensors": oracle.cast(t)}
    prompts = [ids(n, 20 + n) for n in (5, 70, 1, 64)]
    want = [oracle.generate(ref, p, 10 + i) for i, p in enumerate(prompts)]
    e = LLMEngine(device="cuda", dtype=torch.float32, max_pages=12, max_active=2, use_graphs=graphs)
    e.set_weights(cases.weights(cfg, t))
    for i, p in enumerate(prompts):
        e.submit_request(Request(i, p, GenerationConfig(max_new_tokens=10 + i, **GREEDY)))
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
    cfg, t = cases.model(WIDE, seed=12, width=96)
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
