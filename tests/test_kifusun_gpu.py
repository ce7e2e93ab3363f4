"""Kifusun on a GPU: the kernels against the plain math, the engine in fp32 and bf16 against tests/kifusun_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kifusun_cases as cases  # noqa: E402
import kifusun_oracle as oracle  # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
# sizes the tensor-core paths take as they come, beside the odd ones of kifusun_cases
WIDE = [cases.layer(heads=8, kv=2, dim=64, vdim=64, window=100, ff=128, dmax=60, scale=0.12, cap=20.0, v_mix=v) for v in (False, True, True)]
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


def attention_case(H, G, D, Dv, W, lens, starts, talk=True, cap=30.0, seed=0):
    from prometorch_b200.ops import gated_attention as A
    g = torch.Generator().manual_seed(seed)
    per = [(s + n + 63) // 64 for s, n in zip(starts, lens)]
    pages = sum(per) + 3
    order = torch.randperm(pages, generator=g).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    for i, c in enumerate(per):
        table[i, :c] = torch.tensor([order.pop() for _ in range(c)])
    rnd = lambda *s: torch.randn(*s, generator=g)
    a = A.GatedAttention(H, G, D, Dv, W, D ** -0.5, cap, A.distance_bias(rnd(12, H), 60, W, rnd(H) - 2).cuda(),
                         (rnd(H, H) * 0.3).bfloat16().float().cuda() if talk else None)
    n = sum(lens)
    k, v, q = torch.zeros(pages, G, 64, a.dim_stored), torch.zeros(pages, G, 64, a.vdim_stored), torch.zeros(n, H, a.dim_stored)
    k[..., :D], v[..., :Dv], q[..., :D] = rnd(pages, G, 64, D) * 1.5, rnd(pages, G, 64, Dv), rnd(n, H, D) * 1.5
    offs = [0]
    for x in lens:
        offs.append(offs[-1] + x)
    pos = torch.cat([torch.arange(s, s + m, dtype=torch.int32) for s, m in zip(starts, lens)])
    req = torch.cat([torch.full((m,), i, dtype=torch.int32) for i, m in enumerate(lens)])
    return a, q.bfloat16().cuda(), k.bfloat16().cuda(), v.bfloat16().cuda(), pos.cuda(), req.cuda(), table.cuda(), offs


SHAPES = [dict(H=8, G=2, D=128, Dv=128, W=100, lens=[200, 300], starts=[0, 0]), dict(H=16, G=4, D=128, Dv=128, W=1024, lens=[300], starts=[900]),
          dict(H=32, G=8, D=128, Dv=128, W=130, lens=[150, 17], starts=[0, 90]), dict(H=6, G=3, D=48, Dv=80, W=64, lens=[90, 64, 1], starts=[0, 1, 70]),
          dict(H=12, G=12, D=64, Dv=64, W=33, lens=[90, 64], starts=[0, 1]), dict(H=5, G=1, D=80, Dv=100, W=50, lens=[90, 64], starts=[0, 1], talk=False),
          dict(H=40, G=8, D=64, Dv=128, W=90, lens=[90, 64], starts=[0, 1]), dict(H=64, G=8, D=96, Dv=96, W=90, lens=[120], starts=[0], cap=0.0),
          dict(H=8, G=4, D=256, Dv=256, W=90, lens=[120], starts=[3]), dict(H=3, G=3, D=16, Dv=64, W=1, lens=[70], starts=[0]),
          dict(H=7, G=7, D=20, Dv=72, W=300, lens=[270], starts=[10]), dict(H=9, G=1, D=24, Dv=12, W=200, lens=[70], starts=[129]),
          dict(H=16, G=1, D=64, Dv=64, W=150, lens=[75, 33], starts=[300, 0]), dict(H=32, G=1, D=80, Dv=64, W=40, lens=[97], starts=[64]),
          dict(H=8, G=4, D=96, Dv=64, W=257, lens=[300, 9], starts=[0, 257]), dict(H=24, G=6, D=128, Dv=64, W=500, lens=[200], starts=[450]),
          dict(H=28, G=14, D=64, Dv=128, W=70, lens=[130], starts=[7], cap=0.0)]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "h{H}g{G}d{D}v{Dv}w{W}".format(**s))
def test_attention_kernels(shape):
    from prometorch_b200.ops import gated_attention as A, paged as P
    a, q, k, v, pos, req, table, offs = attention_case(**shape)
    n, top = q.shape[0], int(pos.max()) + 1
    ref = A.gated_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())
    for splits in {A.pick_splits(n, a.window, top), A.pick_splits(1, a.window, top)}:
        assert rel(A.gated_attention(q.float(), a, pos, req, table, k.float(), v.float(), splits, top), ref) < 2e-6
        assert rel(A.gated_attention(q, a, pos, req, table, k, v, splits, top), ref) < 4e-3
    if A.tiles_supported(q, a):
        tiles = A.PromptTiles.of(offs, shape["starts"], list(range(len(offs) - 1)), "cuda")
        for tc in (True, False):
            assert rel(A.gated_attention_tiles(q, a, tiles, table, k, v, tensor_cores=tc), ref) < 5e-3
    P.check_status("cuda")


@pytest.mark.parametrize("big", [3.0, 12.0, 60.0])
def test_large_scores(big):
    """Scores far into the soft cap's bend and past it, one standing out among small ones."""
    from prometorch_b200.ops import gated_attention as A
    a, q, k, v, pos, req, table, offs = attention_case(8, 2, 64, 64, 70, [130], [0], cap=3.0)
    q[40:44] *= big
    ref = A.gated_attention_reference(q.float(), a, pos, req, table, k.float(), v.float())
    assert rel(A.gated_attention(q.float(), a, pos, req, table, k.float(), v.float(), 1, 130), ref) < 2e-6
    assert rel(A.gated_attention(q, a, pos, req, table, k, v, 1, 130), ref) < 4e-3
    for tc in (True, False):
        assert rel(A.gated_attention_tiles(q, a, A.PromptTiles.of(offs, [0], [0], "cuda"), table, k, v, tensor_cores=tc), ref) < 5e-3


@pytest.mark.parametrize("W", [31, 32, 33, 64, 65, 128])
def test_window_edges(W):
    """A value that stands out counts from its own place to W - 1 places later, in both kernels, at page and tile borders."""
    from prometorch_b200.ops import gated_attention as A
    a, q, k, v, pos, req, table, offs = attention_case(4, 1, 64, 64, W, [230], [0])
    tiles = A.PromptTiles.of(offs, [0], [0], "cuda")
    for j in (0, 31, 32, 63, 64, 100):
        v2 = v.clone()
        v2[table[0, j // 64], :, j % 64] += 200.0
        for run in (lambda x: A.gated_attention(q, a, pos, req, table, k, x, 2, 230), lambda x: A.gated_attention_tiles(q, a, tiles, table, k, x),
                    lambda x: A.gated_attention_tiles(q, a, tiles, table, k, x, tensor_cores=False)):
            d = (run(v2).float() - run(v).float()).abs().amax(1)
            assert (d > 0.05).nonzero()[:, 0].tolist() == list(range(j, min(230, j + W)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 128, 64), (3, 1, 20, 28), (2, 2, 7, 9), (8, 1, 256, 16)])
def test_head_norm_kernel(dtype, H, G, D, Dv):
    from prometorch_b200.ops import gated_attention as A, paged as P
    n, eps = 37, 1e-3
    a = A.GatedAttention(H, G, D, Dv, 5, 1.0, 0.0, torch.zeros(H, 1), None)
    qkv, first = (torch.randn(n, w).to(dtype) for w in (H * D + G * (D + Dv), G * Dv + 3))
    qw, kw = torch.randn(D), torch.randn(D)
    pos, req = torch.arange(40, 40 + n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)
    table = torch.tensor([[0, 0], [3, 1]], dtype=torch.int32)
    pages = [torch.full((4, G, 64, s), 5.0, dtype=dtype) for s in (a.dim_stored, a.vdim_stored)]
    gpu = [p.cuda() for p in pages]
    args = (qw, kw, eps, pos, req, table)
    want = A.head_norm_write(qkv, a, *args, *pages, first[:, :G * Dv], 0.3)
    got = A.head_norm_write(qkv.cuda(), a, *[x.cuda() if torch.is_tensor(x) else x for x in args], *gpu, first.cuda()[:, :G * Dv], 0.3)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    assert rel(got, want) < tol and all(rel(x, y) < tol for x, y in zip(gpu, pages))
    P.check_status("cuda")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [64, 2048, 9000, 50])
def test_residual_kernels(dtype, W):
    from prometorch_b200.ops import residual as S
    n = 19
    x, y = torch.randn(n, W), torch.randn(n, W).to(dtype)
    for w in (None, torch.randn(W)):
        xc, xg = x.clone(), x.cuda()
        sc = (xc, xc if dtype == torch.float32 else torch.empty(n, W, dtype=dtype))
        sg = (xg, xg if dtype == torch.float32 else torch.empty(n, W, dtype=dtype, device="cuda"))
        S.post_norm_add(y, sc, 1.3, 1e-3, w)
        S.post_norm_add(y.cuda(), sg, 1.3, 1e-3, w.cuda() if w is not None else None)
        assert rel(sg[0], sc[0]) < 1e-6 and rel(sg[1], sc[1]) < (1e-6 if dtype == torch.float32 else 4e-3)
        i = torch.tensor([n - 1, 0, 4])
        assert rel(S.row_norm(sg, 0.7, 1e-3, w.cuda() if w is not None else None, i.cuda()), S.row_norm(sc, 0.7, 1e-3, w, i)) < 5e-3
    t, k = torch.randn(30, W).to(dtype), torch.randint(0, 30, (n,), dtype=torch.int32)
    assert rel(S.embed_residual(k.cuda(), t.cuda(), 2.5)[0], S.embed_residual(k, t, 2.5)[0]) < 1e-6


@pytest.mark.parametrize("M", [1, 5, 40, 100, 300])
def test_projection_then_norm_and_logits(M):
    from prometorch_b200.ops import residual as S
    K, Nn = 256, 512
    a, w, head = torch.randn(M, K).bfloat16(), (torch.randn(Nn, K) * K ** -0.5).bfloat16(), (torch.randn(1000, K) * K ** -0.5).bfloat16()
    x = torch.randn(M, Nn)
    with torch.no_grad():
        got = S.linear_post_norm_add(a.cuda(), w.cuda(), (x.cuda(), torch.empty(M, Nn, dtype=torch.bfloat16, device="cuda")), 1.2, 1e-4)
        want = x.double() + oracle.scalar_norm(a.double() @ w.double().t(), 1.2, 1e-4)
        assert rel(got[0], want) < 3e-3 and rel(got[1], want) < 6e-3
        assert rel(S.linear_f32(a.cuda(), head.cuda()), a.double() @ head.double().t()) < 1e-5


# ------------------------------------------------------------------------------------------ the model
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
        got = torch.cat(out)
        err = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert float(err.max()) < TOL[dtype], (cuts[:3], float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_batch_and_page_reuse(dtype):
    """Four sequences prefilled and decoded together, one ends early; then the freed pages serve another run."""
    cfg, t = cases.model(WIDE, seed=2, width=96)
    ref = {"config": cfg, "tensors": oracle.cast(t)}
    lens = [1, 64, 150, 33]
    xs = [ids(n + 70, 30 + n) for n in lens]
    want = [oracle.forward(ref, x) for x in xs]
    e = engine(cfg, t, dtype, max_pages=10)
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
    cfg, t = cases.model([cases.layer(heads=4, kv=2, dim=32, vdim=32, window=50, ff=64) for _ in range(2)], seed=3)
    x = ids(500, 5)
    want = oracle.forward({"config": cfg, "tensors": oracle.cast(t)}, x)
    e = engine(cfg, t, torch.bfloat16, max_pages=4)
    s = e.open_sequence()
    out = [e.feed([(s, x[:128], [127])])] + [e.feed([(s, [x[j]], [0])]) for j in range(128, 500)]
    assert rel(torch.cat(out), want[127:]) < TOL[torch.bfloat16] and e.kv.pages_in_use <= 2


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_scheduler(graphs):
    """fp32: the oracle's ids, with requests that queue and finish at different times."""
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
