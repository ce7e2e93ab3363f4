"""Budorax on CPU: each mechanism and the whole model in the batching engine against tests/budorax_oracle.py."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import budorax_cases as cases  # noqa: E402
import budorax_oracle as oracle  # noqa: E402

from prometorch_b200.models.budorax import BudoraxConfig, BudoraxWeights  # noqa: E402
from prometorch_b200.models.paged import known_models, resolve_architecture  # noqa: E402
from prometorch_b200.ops import experts as X, latent_attention as M, recurrence as R, residual as S, tanh_norm as T, window_attention as A  # noqa: E402
from prometorch_b200.ops.rotary import Rotary  # noqa: E402
from prometorch_b200.serve.llm import PAGE, GenerationConfig, LLMEngine, Request, save_safetensors  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
MODELS = {"mixed": (cases.MIXED, cases.MIXED_LOOP), "even": (cases.EVEN, (0, 2, 3)), "single": (cases.SINGLE, None)}


def ids(n, seed=0, vocab=61):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def reference(cfg, t):
    return {"config": cfg, "tensors": oracle.cast(t)}


def build(name, seed=0, **kw):
    layers, loop = MODELS[name]
    return cases.model(layers, seed=seed, loop=loop, **kw)


def engine(cfg, t, max_pages=16, max_active=6, **kw):
    e = LLMEngine(device="cpu", dtype=torch.float32, max_pages=max_pages, max_active=max_active, **kw)
    e.set_weights(cases.weights(cfg, t))
    return e


def close(a, b, tol=2e-5):
    a, b = a.double(), b.double()
    return float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max()))


def rows(n, first=0):
    return torch.arange(first, first + n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)


def scattered(pages=8, seed=1):
    g = torch.Generator().manual_seed(seed)
    table = torch.zeros(2, pages, dtype=torch.int32)
    table[1] = torch.randperm(pages, generator=g).int()
    return table


# ------------------------------------------------------------------------------------------ norms, rotation
def test_tanh_norm_around_the_stream():
    n, W = 5, 24
    x, y, z = torch.randn(n, W), torch.randn(n, W), torch.randn(3, n, W)
    post, pre = (T.TanhNorm(a, torch.randn(W), torch.randn(W)) for a in (0.6, 1.7))
    ref = lambda v, m: oracle.tanh_norm(v, m.alpha, m.w.double(), m.b.double())
    want = x.double() + ref(y.double(), post)
    h = T.residual(x, S.Branch(y), post, pre)
    assert close(x, want) and close(h, ref(want, pre))
    want = want + ref(z.double().sum(0), post)
    assert T.residual(x, S.Branch(z), post, None) is None and close(x, want)
    table, ids_ = torch.randn(7, W), torch.tensor([3, 0, 6, 3, 1], dtype=torch.int32)
    rows_ = X.ExpertRows(torch.randn(2 * n, W), torch.randperm(2 * n).view(n, 2).int(), torch.rand(n, 2))
    mixed = torch.stack([sum(rows_.weight[i, k].double() * rows_.y[rows_.index[i, k]].double() for k in range(2)) for i in range(n)])
    want = want + ref(mixed, post) + table[ids_.long()].double()
    h = T.residual(x, rows_, post, pre, again=(ids_, table))
    assert close(x, want) and close(h, ref(want, pre))
    assert close(T.rows(x, pre, torch.tensor([4, 1])), ref(want[[4, 1]], pre))
    assert close(T.softcap(x * 30, 7.0), torch.tanh(want * 30 / 7) * 7)


@pytest.mark.parametrize("dims,size", [(0, 6), (2, 6), (8, 8), (6, 11)])
def test_rotation(dims, size):
    rot = Rotary(dims, 300.0, 5000)
    x, pos = torch.randn(4, 3, size), torch.tensor([0, 1, 63, 4999], dtype=torch.int32)
    assert close(rot.apply(x, pos), oracle.rotate_rows(x.double(), dims, 300.0, pos.tolist()))


# ------------------------------------------------------------------------------------------ attention with two maps
def two_map_case(H, G, D, Dv, chunk, n, diff=0.3, rot=4, seed=1, eps=1e-3, scale=0.4):
    a = A.WindowAttention(H, G, D, Dv, chunk, 0, scale, chunked=True, maps=2, mix=0.45, mix_gain=1 - diff, mix_eps=eps)
    g = torch.Generator().manual_seed(seed)
    p = torch.randn(n, 3 + 2 * H * D + 2 * G * D + G * Dv + 2, generator=g) * 1.5
    cols = (3, 3 + 2 * H * D, 3 + 2 * H * D + 2 * G * D)
    kp, vp = torch.zeros(8, G, PAGE, a.key_stored), torch.zeros(8, G, PAGE, a.vdim_stored)
    return a, p, cols, Rotary(rot, 100.0, 1024), scattered(), kp, vp


def two_map_oracle(a, p, cols, rot, diff=0.3):
    n, H, G, D, Dv = p.shape[0], a.heads, a.kv_heads, a.dim, a.vdim
    x = p.double()
    q = oracle.rotate_rows(x[:, cols[0]:cols[0] + 2 * H * D].view(n, H, 2, D), rot.dims, rot.base)
    k = oracle.rotate_rows(x[:, cols[1]:cols[1] + 2 * G * D].view(n, G, 2, D), rot.dims, rot.base)
    v = x[:, cols[2]:cols[2] + G * Dv].view(n, G, Dv)
    return oracle.two_maps_rows(q, k, v, a.scale, a.window, a.mix, diff, a.mix_eps)


@pytest.mark.parametrize("H,G,D,Dv,chunk,rot", [(4, 2, 12, 20, 20, 8), (3, 3, 8, 6, 70, 0), (2, 1, 10, 8, 1, 10), (2, 2, 16, 16, 64, 2), (2, 1, 8, 8, 500, 4)])
def test_two_maps_in_chunks(H, G, D, Dv, chunk, rot):
    n = 140
    a, p, cols, r, table, kp, vp = two_map_case(H, G, D, Dv, chunk, n, rot=rot)
    q = A.rope_write(p, cols, a, r, *rows(n), table, kp, vp)
    got = A.window_attention(q, a, *rows(n), table, kp, vp, 1, n).view(n, H, Dv)
    assert close(got, two_map_oracle(a, p, cols, r))


@pytest.mark.parametrize("chunk", [5, 63, 64, 65, 100])
def test_chunk_edges(chunk):
    """A value that stands out counts from its own place to the end of its chunk: the chunks lie by position in the sequence, also when
    the rows are a later portion."""
    n = 170
    a, p, cols, r, table, kp, vp = two_map_case(2, 1, 16, 16, chunk, n, scale=0.05)
    a.mix = 0.1
    q = A.rope_write(p, cols, a, r, *rows(n), table, kp, vp)
    for j in (0, 3, 62, 63, 64, 65, 99, 100, 129):
        vp2 = vp.clone()
        vp2[table[1, j // PAGE], :, j % PAGE, 0] += 1e4
        for first in (0, 50, 101):
            part = [x[first:] for x in rows(n)]
            d = (A.window_attention(q[first:], a, *part, table, kp, vp2, 1, n) - A.window_attention(q[first:], a, *part, table, kp, vp, 1, n)).abs().amax(1)
            assert [first + i for i in (d > 1e-2).nonzero()[:, 0].tolist()] == [i for i in range(first, n) if oracle.same_chunk(i, j, chunk)]


def test_a_score_that_stands_out_carries_its_value():
    """One key of the first map turned towards one query: the head returns that value's direction, scaled to the norm."""
    n, D = 40, 16
    a, p, cols, r, table, kp, vp = two_map_case(1, 1, D, 16, 100, n, rot=0, eps=1e-9)
    p[33, 3:3 + D] = p[7, cols[1]:cols[1] + D] * 40
    a.mix = 0.0
    q = A.rope_write(p, cols, a, r, *rows(n), table, kp, vp)
    out = A.window_attention(q, a, *rows(n), table, kp, vp, 1, n)
    v = p[7, cols[2]:cols[2] + 16].double()
    assert close(out[33], oracle.rms(v, 1e-9) * 0.7, 1e-4)


def test_factor_of_the_second_map():
    cfg, t = cases.model([cases.attention(dim=6, rot=4, diff=0.3)], seed=3)
    e = engine(cfg, t)
    a, m = e.model.prep[0]["attn"], reference(cfg, t)["tensors"]
    want = oracle.mix_factor(*(m["l0.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")), 0.3)
    assert abs(a.mix - want) < 1e-6 and abs(a.mix_gain - 0.7) < 1e-9


# ------------------------------------------------------------------------------------------ latent attention
def latent_case(H=3, D=10, Rd=6, Dv=7, rank=20, q_rank=9, n=150, seed=2):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    uk, uv = r(H * D, rank) * 0.4, r(H * Dv, rank)
    a = M.LatentAttention.of(H, D, Rd, Dv, rank, 0.3, uk, uv, Rotary(Rd, 400.0, 1024))
    p = r(n, 2 + q_rank + rank + Rd + 1)
    return a, uk, uv, p, (2, 2 + q_rank), r(q_rank) * 0.2 + 1, r(rank) * 0.2 + 1.3, r(n, H * (D + Rd) + 3)


@pytest.mark.parametrize("sizes", [dict(), dict(H=1, D=8, Rd=2, Dv=16, rank=16, q_rank=16), dict(H=4, D=5, Rd=16, Dv=3, rank=33, q_rank=1)])
def test_latent_attention(sizes):
    a, uk, uv, p, cols, qw, kw, q = latent_case(**sizes)
    n, H, D, Rd, Dv, rank, eps = q.shape[0], a.heads, a.dim, a.rot_dim, a.vdim, a.rank, 1e-3
    table, pages = scattered(), torch.zeros(8, 1, PAGE, a.row)
    gate = torch.randn(n, H)
    c = M.latent_write(p, cols, a, qw, kw, eps, *rows(n), table, pages)
    x = p.double()
    assert close(c, oracle.plain_norm(x[:, cols[0]:cols[0] + len(qw)], qw.double(), eps))
    got = M.latent_attention(q, a, *rows(n), table, pages, n, gate).view(n, H, Dv)
    lat = oracle.plain_norm(x[:, cols[1]:cols[1] + rank], kw.double(), eps)
    shared = oracle.rotate_rows(x[:, cols[1] + rank:cols[1] + rank + Rd], Rd, 400.0)
    qd = q[:, :H * (D + Rd)].double().view(n, H, D + Rd)
    qd = torch.cat([qd[..., :D], oracle.rotate_rows(qd[..., D:], Rd, 400.0)], -1)
    k = torch.cat([(lat @ uk.double().t()).view(n, H, D), shared[:, None].expand(n, H, Rd)], -1)
    want = oracle.latent_rows(qd, k, (lat @ uv.double().t()).view(n, H, Dv), 0.3)
    assert close(got, want * oracle.sigmoid(gate.double())[..., None])
    # a later portion and single rows see the same keys
    for lo, hi in ((64, 150), (149, 150), (100, 102)):
        part = [v[lo:hi] for v in rows(n)]
        assert close(M.latent_attention(q[lo:hi], a, *part, table, pages, hi, gate[lo:hi]), got[lo:hi].reshape(hi - lo, -1))


# ------------------------------------------------------------------------------------------ delta rule, gate
def seqs_of(lens, starts, slots):
    offs = [0]
    for n in lens:
        offs.append(offs[-1] + n)
    s = R.Sequences.of(offs, starts, slots, "cpu")
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return s, pos, req


@pytest.mark.parametrize("dim", [1, 12])
def test_delta_rule_with_one_decay_per_head(dim):
    H, G, D, Dv, n = 4, 2, dim, 20, 40
    g = torch.Generator().manual_seed(4)
    r = R.DeltaRule(H, G, D, Dv, torch.rand(H, generator=g) + 0.3, torch.randn(H, generator=g) - 1, head_decay=True)
    x, beta, a = (torch.randn(n, w, generator=g) for w in (2 * G * D + H * Dv, H, H))
    f = x.double()
    q, k = oracle.unit(f[:, :G * D].view(n, G, D)) * D ** -0.5, oracle.unit(f[:, G * D:2 * G * D].view(n, G, D))
    v, b = f[:, 2 * G * D:].view(n, H, Dv), oracle.sigmoid(beta.double())
    decay = oracle.head_decay(a.double(), r.rate.double().log(), r.dt_bias.double())
    want, last = torch.zeros(n, H, Dv, dtype=torch.float64), []
    for h in range(H):
        st = torch.zeros(D, Dv, dtype=torch.float64)
        for i in range(n):
            st, want[i, h] = oracle.delta_step(st, q[i, h // 2], k[i, h // 2], v[i, h], decay[i, h], b[i, h])
        last.append(st)
    for cuts in ([40], [2] * 20, [1, 38, 1], [17, 23]):
        state, at, out = torch.full((3, H, D, Dv), 5.0), 0, []
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [1])
            out.append(R.delta_rule(x[at:at + m], r, beta[at:at + m], a[at:at + m], state, pos, req, s if m > 1 else None))
            at += m
        assert close(torch.cat(out), want.view(n, -1)) and close(state[1], torch.stack(last)) and float(state[0].min()) == 5.0


def test_norm_per_head_and_silu_gate():
    o, gate, w = torch.randn(5, 24), torch.randn(5, 40), torch.randn(8)
    want = oracle.plain_norm(o.double().view(5, -1, 8), w.double(), 1e-2).reshape(5, 24) * oracle.silu(gate[:, 9:33].double())
    assert close(R.group_norm_gate(o, w, gate[:, 9:33], 1e-2, torch.float32, act="silu"), want)


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,top,ff", [(6, 2, 20), (3, 3, 8), (9, 1, 7)])
def test_experts(E, top, ff):
    W, n = 24, 30
    g = torch.Generator().manual_seed(5)
    r = lambda *s: torch.randn(*s, generator=g)
    gate, up, down = ([r(*s) * 0.3 for _ in range(E)] for s in ((ff, W), (ff, W), (W, ff)))
    router, corr, h = r(E, W) * 0.2, r(E), r(n, W)
    e = X.Experts.of(gate, up, down, router, corr, top, 1.7)
    out = X.run(h, e)
    t = {"router": router.double(), "correction": corr.double()}
    for i in range(E):
        t.update({f"e{i}.gate": gate[i].double(), f"e{i}.up": up[i].double(), f"e{i}.down": down[i].double()})
    want = oracle.experts(h.double(), t, "", {"router": {"top": top, "scale": 1.7}})
    assert close(out.combine(), want)
    assert sorted(out.index.flatten().tolist()) == list(range(n * top)) and close(out.weight.sum(1), torch.full((n,), 1.7))


def test_the_correction_chooses_and_does_not_weigh():
    W, E = 8, 4
    eye = [torch.eye(W) * (i + 1) for i in range(E)]
    e = X.Experts.of(eye, eye, eye, torch.zeros(E, W), torch.tensor([0.0, 3.0, -1.0, 2.0]), 2, 1.0)
    out = X.run(torch.randn(3, W), e)
    assert close(out.weight, torch.full((3, 2), 0.5))                   # equal scores, whatever the corrections
    r = X.route(torch.randn(3, W), e)
    assert r.offsets.tolist() == [0, 0, 3, 3, 6]


# ------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompt(name):
    cfg, t = build(name)
    x = ids(130)
    e = engine(cfg, t)
    assert close(e.feed([(e.open_sequence(), x, range(130))]), oracle.forward(reference(cfg, t), x))


def test_every_layer():
    """A model cut off after each of its layers."""
    for k in range(len(cases.MIXED) + 1):
        cfg, t = cases.model(cases.MIXED[:k], seed=20)
        x = ids(40, 3)
        e = engine(cfg, t)
        assert close(e.feed([(e.open_sequence(), x, range(40))]), oracle.forward(reference(cfg, t), x)), k


@pytest.mark.parametrize("loop", [None, (0, 1, 2), (1, 3, 3), (0, 3, 2), (2, 3, 4), (1, 1, 5), (0, 3, 1)])
def test_loops(loop):
    """Every pass of a looped run has entries of its own, and the embedding joins once ahead of every pass but the first."""
    cfg, t = cases.model(cases.EVEN, seed=21, loop=loop)
    x = ids(40, 5)
    e = engine(cfg, t)
    runs = len(oracle.run_order(cfg))
    assert len(e.kv.k) == len(e.kv.state) == runs
    s = e.open_sequence()
    got = [e.feed([(s, x[:30], range(30))])] + [e.feed([(s, [x[j]], [0])]) for j in range(30, 40)]
    assert close(torch.cat(got), oracle.forward(reference(cfg, t), x))


@pytest.mark.parametrize("name", ["mixed", "single"])
@pytest.mark.parametrize("start", [1, 60])
def test_token_by_token(name, start):
    """Decoding through cache and state, over page and chunk borders, equals the whole prompt."""
    cfg, t = build(name, seed=1)
    x = ids(135, 1)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    got = [e.feed([(s, x[:start], range(start))])] + [e.feed([(s, [x[j]], [0])]) for j in range(start, len(x))]
    assert close(torch.cat(got), want)


@pytest.mark.parametrize("portion", [2, 7, 64, 65])
def test_portions(portion):
    cfg, t = build("mixed", seed=2)
    x = ids(131, 2)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    got = [e.feed([(s, x[lo:lo + portion], range(len(x[lo:lo + portion])))]) for lo in range(0, len(x), portion)]
    assert close(torch.cat(got), want)


def test_unequal_batch_against_each_alone():
    cfg, t = build("mixed", seed=3)
    lens = [1, 64, 90, 3]
    xs = [ids(n + 45, 10 + n) for n in lens]
    want = [oracle.forward(reference(cfg, t), x) for x in xs]
    e = engine(cfg, t)
    seqs = [e.open_sequence() for _ in xs]
    out = e.feed([(s, x[:n], [n - 1, 0]) for s, x, n in zip(seqs, xs, lens)])
    assert close(out, torch.cat([w[[n - 1, 0]] for w, n in zip(want, lens)]))
    live = list(range(4))
    for j in range(45):                                                  # the first sequence ends early
        if j == 20:
            e.close_sequence(seqs[0])
            live.remove(0)
        out = e.feed([(seqs[i], [xs[i][lens[i] + j]], [0]) for i in live])
        assert close(out, torch.stack([want[i][lens[i] + j] for i in live]))


def test_portions_of_one_beside_the_first_tokens_of_another():
    """One batch: a sequence that goes on by three tokens, one by a single token, and one that starts."""
    cfg, t = build("mixed", seed=4)
    x, y, z = ids(80, 1), ids(40, 2), ids(70, 3)
    want = [oracle.forward(reference(cfg, t), v) for v in (x, y, z)]
    e = engine(cfg, t)
    a, b, c = (e.open_sequence() for _ in range(3))
    e.feed([(a, x[:77], []), (b, y[:39], [])])
    out = e.feed([(a, x[77:], [0, 2]), (b, y[39:], [0]), (c, z, [69])])
    assert close(out, torch.stack([want[0][77], want[0][79], want[1][39], want[2][69]]))


def test_what_a_layer_still_sees():
    """A changed token is seen to the end of its chunk and no further by the chunked layer, by everything behind it through the latent one."""
    x = ids(60, 4)
    for layer, seen in ((cases.attention(chunk=16), lambda j: list(range(j, (j // 16 + 1) * 16))), (cases.latent(), lambda j: list(range(j, 60)))):
        cfg, t = cases.model([layer], seed=4)
        for j in (15, 16, 17, 31):
            y = list(x)
            y[j] = (x[j] + 1) % 61
            e = engine(cfg, t)
            a, b = e.open_sequence(), e.open_sequence()
            out = e.feed([(a, x[:25], range(25)), (b, y[:25], range(25))])
            diff = [(out[i] - out[25 + i]).abs().max().item() for i in range(25)]
            for i in range(25, 60):
                out = e.feed([(a, [x[i]], [0]), (b, [y[i]], [0])])
                diff.append((out[0] - out[1]).abs().max().item())
            assert [i for i, d in enumerate(diff) if d > 1e-7] == [i for i in seen(j) if i < 60]


def test_pages_of_finished_chunks_and_slots_come_back():
    """Without a latent layer the pages behind the chunk return while the request runs; freed pages and state slots serve another one,
    whose first tokens see nothing of the old state."""
    cfg, t = cases.model([cases.attention(chunk=50), cases.delta(), cases.attention(chunk=80, heads=2, kv=1)], seed=6, loop=(0, 2, 2))
    x, y = ids(300, 6), ids(120, 7)
    want, want_y = (oracle.forward(reference(cfg, t), z) for z in (x, y))
    e = engine(cfg, t, max_pages=4, max_active=1)
    s = e.open_sequence()
    got = [e.feed([(s, x[:100], [99])])]
    for j in range(100, 300):
        got.append(e.feed([(s, [x[j]], [0])]))
        assert e.kv.pages_in_use <= 3
    assert close(torch.cat(got), want[99:]) and s.pages[0] == -1
    e.close_sequence(s)
    assert e.kv.pages_in_use == 0
    s = e.open_sequence()
    got = [e.feed([(s, y[:70], range(70))])] + [e.feed([(s, [y[j]], [0])]) for j in range(70, 120)]
    assert close(torch.cat(got), want_y)
    e.close_sequence(s)
    s = e.open_sequence()
    assert close(e.feed([(s, y[:1], [0])]), want_y[:1])                  # a prompt of one token
    with pytest.raises(RuntimeError):
        e.feed([(s, ids(400), [])])                                      # more than the pool holds at once


def test_a_latent_layer_keeps_every_page():
    cfg, t = cases.model(cases.EVEN, seed=7)
    e = engine(cfg, t, max_pages=5, max_active=1)
    s = e.open_sequence()
    e.feed([(s, ids(300), [])])
    assert e.kv.pages_in_use == 5 and e.model.cache_window() is None


def test_greedy_generation_through_the_scheduler():
    cfg, t = build("mixed", seed=8, width=40)
    ref = reference(cfg, t)
    prompts = [ids(n, 20 + n) for n in (5, 40, 1, 37)]
    want = [oracle.generate(ref, p, 8) for p in prompts]
    e = engine(cfg, t, max_active=2)                                     # two at a time: the others wait
    assert e.generate(prompts[0], GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want[0]
    for i, p in enumerate(prompts):
        e.submit_request(Request(100 + i, p, GenerationConfig(max_new_tokens=8, **GREEDY)))
    got = {}
    while e.num_active():
        e.step()
        got.update({r.request_id: r.token_ids for r in e.poll_responses()})
    assert [got[100 + i] for i in range(4)] == want
    assert e.kv.pages_in_use == 0 and sorted(e.free_rows) == [0, 1]
    stop = want[1][3]
    assert e.generate(prompts[1], GenerationConfig(max_new_tokens=8, stop_tokens=[stop], **GREEDY)).token_ids == want[1][:want[1].index(stop) + 1]
    emb = e.embed(prompts[1])
    assert emb.shape == (40,) and abs(float(emb.norm()) - 1) < 1e-5


def test_proposals_are_taken_back_where_no_state_runs():
    """Speculative decoding needs a model that can take a token back: one without recurrent layers."""
    rep = (ids(5, 1) * 6)[:24]
    for layers, rewinds in (([cases.attention(chunk=30), cases.latent(mlp=cases.moe())], True), ([cases.delta(), cases.attention()], False)):
        cfg, t = cases.model(layers, seed=8)
        e = engine(cfg, t, spec_tokens=3)
        assert e.generate(rep, GenerationConfig(max_new_tokens=14, **GREEDY)).token_ids == oracle.generate(reference(cfg, t), rep, 14)
        assert e.model.rewinds == rewinds and (e.spec_drafted > 0) == rewinds


def test_sampled_generation_and_text():
    cfg, t = cases.model(cases.EVEN, seed=9, vocab=300)
    e = engine(cfg, t)
    r = e.generate("abc", GenerationConfig(max_new_tokens=6, temperature=1.0, top_k=20))
    assert len(r.token_ids) == 6 and all(0 <= i < 300 for i in r.token_ids)
    assert e._encode("abc") == [ord(c) + 3 for c in "abc"]               # the design has no begin-of-text id


# ------------------------------------------------------------------------------------------ configuration, loading, tools
def save(path, cfg, t):
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(t, os.path.join(path, "model.safetensors"))


def test_configuration_and_registry():
    cfg, t = build("mixed")
    assert "budorax" in known_models() and resolve_architecture(cfg).config is BudoraxConfig
    c = BudoraxConfig.from_dict(cfg)
    assert BudoraxConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    for edit in (lambda d: d["layers"][0].update(type="lightning"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                 lambda d: d["layers"][0]["mixer"].update(heads=5, kv_heads=2), lambda d: d["layers"][0]["mlp"]["router"].update(top=9),
                 lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), lambda d: d["layers"][0]["mixer"]["rot"].update(dims=14),
                 lambda d: d["layers"][1]["mixer"]["rot"].update(dims=2), lambda d: d["loop"].update(stop=9), lambda d: d["layers"][2]["mixer"].update(conv=0)):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(ValueError):
            BudoraxConfig.from_dict(bad)
    wrong = dict(t)
    wrong["l1.mix.uk"] = torch.zeros(3, 3)
    with pytest.raises(ValueError):
        cases.weights(cfg, wrong)
    back = cases.weights(cfg, t).state_dict()
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    w = BudoraxWeights.random(c, seed=3)
    assert w.num_parameters() > 0 and all(math.isfinite(float(v.float().sum())) for v in w.state_dict().values())
    e = LLMEngine(device="cpu", max_pages=8, max_active=1)
    c.max_position_embeddings = 512
    e.set_weights(w)
    assert e.weights.num_parameters() == w.num_parameters() and torch.isfinite(e.feed([(e.open_sequence(), ids(30), [29])])).all()


def test_no_loop_and_no_cap():
    cfg, t = cases.model(cases.SINGLE, seed=13, cap=1e9)
    x = ids(20)
    want = oracle.forward(reference(cfg, t), x)
    cfg["logit_softcap"], cfg["loop"] = None, None
    e = engine(cfg, t)
    assert close(e.feed([(e.open_sequence(), x, range(20))]), want, 1e-4)


def test_load_and_serve(tmp_path):
    from prometorch_b200.serve import PagedBackend
    cfg, t = cases.model(cases.EVEN, seed=10, loop=(1, 3, 2))
    save(tmp_path, cfg, t)
    e = LLMEngine(device="cpu", max_pages=8, max_active=2)
    assert e.load(str(tmp_path)) and e.model.architecture == "budorax"
    p = ids(9, 3)
    want = oracle.generate(reference(cfg, t), p, 8)
    assert e.generate(p, GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want
    b = PagedBackend(str(tmp_path), "m", "cpu", max_active=2, max_pages=8)
    out = []
    b.generate(p, {"num_predict": 8, "temperature": 0.0, "repeat_penalty": 1.0}, lambda tok: out.append(tok) or True)
    assert out == want and b.architecture == "budorax"
    b.server.close()


def test_generate_command(tmp_path, capsys):
    from prometorch_b200 import generate
    cfg, t = cases.model(cases.EVEN, seed=11, vocab=300)
    save(tmp_path, cfg, t)
    assert generate.main([str(tmp_path), "hey", "--device", "cpu", "--greedy", "--max-tokens", "5"]) == 0
    assert "budorax" in capsys.readouterr().out
    assert generate.main([str(tmp_path), "--info", "--tensors"]) == 0
    out = capsys.readouterr().out
    assert "l1.mix.lq1" in out and "architecture = 'Budorax'" in out


def test_trace_replay(tmp_path):
    """bin/trace_run on CPU: prompts and decoding of two requests, one of which ends early; logits against the oracle."""
    cfg, t = build("mixed", seed=12)
    save(tmp_path, cfg, t)
    x, y = ids(80, 1), ids(10, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": x[:75], "want": [74, 3]}, {"id": "b", "tokens": y[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": x[75:76], "want": []}, {"id": "b", "tokens": y[8:9], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": x[76:77], "want": [0]}], "end": []}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "128",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = oracle.forward(reference(cfg, t), x[:77])
    got = torch.frombuffer(bytearray((out / "0.f32").read_bytes()), dtype=torch.float32).view(2, -1)
    assert close(got, want[[74, 3]]) and not (out / "1.f32").exists()
    assert close(torch.frombuffer(bytearray((out / "2.f32").read_bytes()), dtype=torch.float32), want[76])
