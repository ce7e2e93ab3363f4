"""Tifepel on CPU: each mechanism and the whole model in the batching engine against tests/tifepel_oracle.py."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import tifepel_cases as cases  # noqa: E402
import tifepel_oracle as oracle  # noqa: E402

from prometorch_b200.models.paged import known_models, resolve_architecture  # noqa: E402
from prometorch_b200.models.tifepel import TifepelConfig, TifepelWeights  # noqa: E402
from prometorch_b200.ops import experts as X, gated_attention as GA, recurrence as R, residual as S, streams as H, window_attention as A  # noqa: E402
from prometorch_b200.serve.llm import PAGE, GenerationConfig, LLMEngine, Request, save_safetensors  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
MODELS = {"mixed": (cases.MIXED, cases.MIXED_LOOP, dict()), "even": (cases.EVEN, (0, 2, 3), dict(streams=2, taps=4)),
          "single": (cases.SINGLE, None, dict(streams=1, taps=1, buckets=1)), "wide": (cases.EVEN[:2], None, dict(streams=5, taps=6, width=20))}


def ids(n, seed=0, vocab=61):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def reference(cfg, t):
    return {"config": cfg, "tensors": oracle.cast(t)}


def build(name, seed=0, **kw):
    layers, loop, sizes = MODELS[name]
    return cases.model(layers, seed=seed, loop=loop, **{**sizes, **kw})


def engine(cfg, t, max_pages=16, max_active=6, **kw):
    e = LLMEngine(device="cpu", dtype=torch.float32, max_pages=max_pages, max_active=max_active, **kw)
    e.set_weights(cases.weights(cfg, t))
    return e


def close(a, b, tol=1e-4):
    a, b = a.double(), b.double()
    return float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max()))


def rows(n, first=0):
    return torch.arange(first, first + n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)


def seqs_of(lens, starts, slots):
    offs = [0]
    for n in lens:
        offs.append(offs[-1] + n)
    s = R.Sequences.of(offs, starts, slots, "cpu")
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return s, pos, req


# ------------------------------------------------------------------------------------------ into and between the sublayers
def test_pair_embedding():
    """A sequence in portions and token by token, a slot that another sequence used before, ids whose products pass 32 bits."""
    W, V = 6, 50
    c = {"embedding": {"bigram": {"buckets": 13, "mul_prev": 2_000_000_011, "mul_cur": 90_001}}}
    t = {"embed": torch.randn(V, W), "bigram": torch.randn(14, W), "pos": torch.randn(40, W)}
    e = H.PairEmbedding(t["embed"], t["bigram"], t["pos"], 2_000_000_011, 90_001)
    x = ids(20, 1, V)
    want = oracle.embed(t, c, x)
    last = torch.full((3, 1), 7, dtype=torch.int32)
    for cuts in ([20], [1] * 20, [3, 1, 9, 7]):
        at, out = 0, []
        for n in cuts:
            s, pos, req = seqs_of([n], [at], [2])
            out.append(H.pair_embed(torch.tensor(x[at:at + n], dtype=torch.int32), e, 4, last, pos, req, s if n > 1 else None))
            at += n
        out = torch.cat(out)
        assert out.shape == (20, 4, W) and all(torch.allclose(out[:, k], want) for k in range(4))
        assert last.flatten().tolist() == [7, 7, x[-1]]
    s, pos, req = seqs_of([4, 1, 3], [0, 6, 2], [0, 1, 2])               # three sequences of one batch, two of them going on
    y = x[:4] + [5] + x[4:7]
    out = H.pair_embed(torch.tensor(y, dtype=torch.int32), e, 1, last, pos, req, s)[:, 0]
    assert torch.allclose(out[:4], want[:4])
    assert torch.allclose(out[4], t["embed"][5] + t["bigram"][(7 * 2_000_000_011 + 5 * 90_001) % 13] + t["pos"][6])
    assert torch.allclose(out[5], t["embed"][x[4]] + t["bigram"][(x[-1] * 2_000_000_011 + x[4] * 90_001) % 13] + t["pos"][2])


@pytest.mark.parametrize("streams", [1, 2, 3, 7])
def test_step_between_sublayers(streams):
    n, W, taps, eps = 9, 20, 4, 1e-2
    g = torch.Generator().manual_seed(streams)
    r = lambda *s: torch.randn(*s, generator=g)
    link = lambda: H.Connection(r(streams), r(streams, streams), r(streams), r(W), r(taps, W), r(W))
    a, b = link(), link()
    x, y, z, rg = r(n, streams, W), r(2, n, W), r(n, W), r(3, n, W)
    pick = X.ExpertRows(r(2 * n, W), torch.randperm(3 * n, generator=g).view(n, 3).int(), torch.rand(n, 3, generator=g), z)
    pick.index[pick.index >= 2 * n] = -1
    start = x.double()
    f = y.double().sum(0)
    for i in range(n):
        for k in range(3):
            f[i] += pick.weight[i, k].double() * (pick.y[pick.index[i, k]] if pick.index[i, k] >= 0 else z[i]).double()
    f = f * oracle.sigmoid(rg.double().sum(0) + a.gate_bias.double())
    want = torch.stack([sum(a.mix[s, t].double() * start[:, s] for s in range(streams)) + a.way_out[t].double() * f for t in range(streams)], 1)
    u = sum(b.way_in[s].double() * want[:, s] for s in range(streams))
    h = oracle.layer_norm(u, b.norm.double(), eps)
    state = torch.zeros(2, taps - 1, W)
    got, read = H.step(x, H.Output(a, S.Branch(rg), S.Branch(y), pick), b, eps, torch.float32, state, *rows(n), seqs_of([n], [0], [1])[0])
    assert close(x, want) and close(got, h) and close(read, h + oracle.causal_conv(h, b.conv.double().t()))
    assert close(state[1], h[-(taps - 1):])
    state.fill_(9.0)                                                      # row by row: the state carries the inputs from token to token
    for i in range(n):
        one, two = H.step(want[i:i + 1].float().clone(), None, b, eps, torch.float32, state, *(v[i:i + 1] for v in rows(n)))
        assert close(one, h[i:i + 1]) and close(two, read[i:i + 1])
    assert H.step(x, None, None, eps, torch.float32, None, *rows(n)) == (None, None)
    assert close(H.rows(x, a.norm, eps, torch.tensor([5, 0])), oracle.layer_norm(want[[5, 0]].sum(1), a.norm.double(), eps))


# ------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("n_rows,far", [(16, 110), (16, 128), (32, 1000), (10, 37), (7, 50), (2, 9), (5, 2.5), (64, 64.5)])
def test_bias_by_distance(n_rows, far):
    table = torch.arange(2 * n_rows).view(n_rows, 2)
    got = GA.distance_bias(table, far, 6000)
    for n in list(range(min(300, 3 * int(far)))) + [int(far) - 1, int(far), int(far) + 1, 5000]:
        assert got[1, min(n, got.shape[1] - 1)] == 2 * oracle.bucket(n, n_rows, far) + 1, n
    assert got.shape[1] <= far + 2 and int(got[0, -1]) == 2 * (n_rows - 1)


def attention_case(Hh, G, D, Dv, n, rel_rows=8, far=30, scale=0.4, seed=1, every=10, coef=0.5):
    g = torch.Generator().manual_seed(seed)
    rel = torch.randn(rel_rows, Hh, generator=g) * 2
    a = A.WindowAttention(Hh, G, D, Dv, A.UNBOUNDED, 0, scale, rel=GA.distance_bias(rel, far, 1024))
    kc, vc = Hh * D + 3, Hh * D + 3 + G * D
    p = torch.randn(n, vc + G * Dv + 2, generator=g) * 1.5
    gain = torch.tensor([oracle.temperature(i, coef, every) for i in range(256)])
    table = torch.zeros(2, 8, dtype=torch.int32)
    table[1] = torch.randperm(8, generator=g).int()
    return a, rel, p, (kc, vc), gain, table, torch.zeros(8, G, PAGE, a.key_stored), torch.zeros(8, G, PAGE, a.vdim_stored)


@pytest.mark.parametrize("Hh,G,D,Dv,far", [(4, 2, 12, 20, 30), (3, 3, 8, 6, 500), (6, 1, 16, 16, 5)])
def test_attention(Hh, G, D, Dv, far):
    n, eps = 140, 1e-2
    a, rel, p, cols, gain, table, kp, vp = attention_case(Hh, G, D, Dv, n, far=far)
    q = GA.head_norm_write(p, a, None, None, eps, *rows(n), table, kp, vp, cols=cols, gain=gain)
    x = p.double()
    qd = oracle.rms(x[:, :Hh * D].view(n, Hh, D), eps)
    qd = torch.stack([r * oracle.temperature(i, 0.5, 10) for i, r in enumerate(qd)])
    assert close(q[..., :D], qd)
    kd, vd = oracle.rms(x[:, cols[0]:cols[0] + G * D].view(n, G, D), eps), x[:, cols[1]:cols[1] + G * Dv].view(n, G, Dv)
    want = oracle.biased_rows(qd, kd, vd, a.scale, rel.double(), far)
    assert close(A.window_attention(q, a, *rows(n), table, kp, vp, 1, n).view(n, Hh, Dv), want)
    for lo, hi in ((64, 140), (139, 140), (100, 102)):                   # a later portion and single rows
        got = A.window_attention(q[lo:hi], a, *(v[lo:hi] for v in rows(n)), table, kp, vp, 1, hi)
        assert close(got.view(hi - lo, Hh, Dv), want[lo:hi])


def test_a_bucket_that_stands_out():
    """One bucket's bias far above the others: every query returns the mean of the values at that bucket's distances."""
    n, D = 120, 8
    a, rel, p, cols, gain, table, kp, vp = attention_case(1, 1, D, D, n, rel_rows=8, far=40, scale=1e-4)
    q = GA.head_norm_write(p, a, None, None, 1e-6, *rows(n), table, kp, vp, cols=cols, gain=gain)
    v = p[:, cols[1]:cols[1] + D].double()
    for b in range(8):
        a.rel = GA.distance_bias(torch.where(torch.arange(8)[:, None] == b, 60.0, 0.0), 40, 1024)
        out = A.window_attention(q, a, *rows(n), table, kp, vp, 1, n)
        for i in range(n):
            there = [j for j in range(i + 1) if oracle.bucket(i - j, 8, 40) == b] or list(range(i + 1))
            assert close(out[i], v[there].mean(0), 2e-3), (b, i)


def test_a_far_key_that_stands_out():
    n, D = 100, 16
    a, rel, p, cols, gain, table, kp, vp = attention_case(1, 1, D, D, n, scale=40.0)
    p[93, :D] = p[2, cols[0]:cols[0] + D]
    q = GA.head_norm_write(p, a, None, None, 1e-9, *rows(n), table, kp, vp, cols=cols, gain=gain)
    out = A.window_attention(q, a, *rows(n), table, kp, vp, 1, n)
    assert close(out[93], p[2, cols[1]:cols[1] + D], 1e-3)


def test_factor_on_queries():
    cfg, t = cases.model([cases.attention(coef=0.7, every=5)], seed=3, max_positions=200)
    gain = engine(cfg, t).model.prep[0]["gain"]
    assert close(gain, torch.tensor([oracle.temperature(p, 0.7, 5) for p in range(200)], dtype=torch.float64), 1e-7)
    assert gain[3] == 1 and gain[4] > 1


# ------------------------------------------------------------------------------------------ state-space recurrence
@pytest.mark.parametrize("Hh,G,N,Dv", [(4, 2, 12, 20), (3, 1, 1, 5), (2, 2, 16, 1)])
def test_state_space_steps(Hh, G, N, Dv):
    n = 40
    g = torch.Generator().manual_seed(4)
    r = R.StateSpace(Hh, G, N, Dv, torch.rand(Hh, generator=g) + 0.3, torch.randn(Hh, generator=g) - 1, torch.randn(Hh, generator=g))
    cols = (Hh * Dv + G * N, Hh * Dv, 0)
    x, a = torch.randn(n, Hh * Dv + 2 * G * N, generator=g), torch.randn(n, Hh + 2, generator=g)[:, 2:]
    f = x.double()
    v, B, C = f[:, :Hh * Dv].view(n, Hh, Dv), f[:, cols[1]:cols[0]].view(n, G, N), f[:, cols[0]:].view(n, G, N)
    dt = oracle.softplus(a.double() + r.dt_bias.double())
    want, last = torch.zeros(n, Hh, Dv, dtype=torch.float64), []
    for h in range(Hh):
        st = torch.zeros(N, Dv, dtype=torch.float64)
        for i in range(n):
            st, want[i, h] = oracle.ssm_step(st, v[i, h], B[i, h // (Hh // G)], C[i, h // (Hh // G)], dt[i, h], r.rate[h].double().log(), r.skip[h].double())
        last.append(st)
    for cuts in ([40], [2] * 20, [1, 38, 1], [17, 23]):
        state, at, out = torch.full((3, Hh, N, Dv), 5.0), 0, []
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [1])
            out.append(R.state_space(x[at:at + m], r, cols, a[at:at + m], state, pos, req, s if m > 1 else None))
            at += m
        assert close(torch.cat(out), want.view(n, -1)) and close(state[1], torch.stack(last)) and float(state[0].min()) == 5.0


def test_convolution_with_a_bias():
    x, w, b = torch.randn(11, 6), torch.randn(6, 4), torch.randn(6)
    want = oracle.silu(oracle.causal_conv(x.double(), w.double()) + b.double())
    for cuts in ([11], [1] * 11, [2, 9]):
        state, at, out = torch.full((2, 3, 6), 3.0), 0, []
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [1])
            out.append(R.short_conv(x[at:at + m], w.t().contiguous(), state, pos, req, s if m > 1 else None, bias=b))
            at += m
        assert close(torch.cat(out), want)


@pytest.mark.parametrize("groups", [1, 3, 24])
def test_gate_ahead_of_a_grouped_norm(groups):
    o, gate, w = torch.randn(5, 24), torch.randn(5, 40), torch.randn(24)
    want = oracle.gated_norm(o.double(), gate[:, 9:33].double(), w.double(), groups, 1e-2)
    assert close(R.group_norm_gate(o, w, gate[:, 9:33], 1e-2, torch.float32, act="silu", groups=groups, gate_first=True), want)


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,identity,top,ff,shared", [(6, 2, 2, 20, 12), (3, 0, 3, 8, 0), (2, 7, 4, 7, 33), (1, 1, 2, 8, 8)])
def test_experts(E, identity, top, ff, shared):
    W, n = 24, 30
    g = torch.Generator().manual_seed(5)
    r = lambda *s: torch.randn(*s, generator=g)
    gate, up, down = ([r(*s) * 0.3 for _ in range(E)] for s in ((ff, W), (ff, W), (W, ff)))
    router, corr, h = r(E + identity, W) * 0.2, r(E + identity) * 0.2, r(n, W)
    e = X.Experts.of(gate, up, down, router, corr, top, 1.0, softmax=True)
    out = X.run(h, e)
    t = {"router": router.double(), "correction": corr.double()}
    for i in range(E):
        t.update({f"e{i}.gate": gate[i].double(), f"e{i}.up": up[i].double(), f"e{i}.down": down[i].double()})
    got, m = out.combine(), {"router": {"top": top, "experts": E, "identity": identity}}
    if shared:
        three = [r(*s) * 0.3 for s in ((shared, W), (shared, W), (W, shared))]
        t.update({"shared." + k: v.double() for k, v in zip(("gate", "up", "down"), three)})
        m["shared"] = {"ff": shared}
        got = got + X.run_shared(h, X.SharedExpert.of(*three)).y
        joined = X.run(h, X.Experts.of(gate, up, down, router, corr, top, 1.0, softmax=True, shared=tuple(three)))       # as more experts of the same products
        assert close(joined.combine(), oracle.moe(h.double(), t, "", m)) and joined.index.shape[1] == top + -(-shared // ff)
    assert close(got, oracle.moe(h.double(), t, "", m))
    held = out.index[out.index >= 0]
    assert sorted(held.tolist()) == list(range(held.numel())) and (identity > 0) == bool((out.index < 0).any())
    assert int(X.route(h, e).offsets[-1]) == held.numel()


def test_identities_return_the_input_and_weights_are_plain_scores():
    W, E = 8, 3
    eye = [torch.eye(W)] * E
    e = X.Experts.of(eye, eye, eye, torch.zeros(E + 2, W), torch.tensor([0.0, -1.0, -1.0, 3.0, 2.0]), 2, 1.0, softmax=True)
    h = torch.randn(4, W)
    out = X.run(h, e)
    assert close(out.weight, torch.full((4, 2), 0.2)) and bool((out.index == -1).all())     # equal scores, whatever the corrections
    assert close(out.combine(), 0.4 * h) and X.route(h, e).offsets.tolist() == [0, 0, 0, 0]


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
    """Every pass of a looped run has entries of its own."""
    cfg, t = cases.model(cases.EVEN, seed=21, loop=loop)
    x = ids(40, 5)
    e = engine(cfg, t)
    runs = len(oracle.run_order(cfg))
    assert len(e.kv.k) == runs and len(e.kv.state) == runs + 1
    s = e.open_sequence()
    got = [e.feed([(s, x[:30], range(30))])] + [e.feed([(s, [x[j]], [0])]) for j in range(30, 40)]
    assert close(torch.cat(got), oracle.forward(reference(cfg, t), x))


@pytest.mark.parametrize("name", ["mixed", "single", "wide"])
@pytest.mark.parametrize("start", [1, 60])
def test_token_by_token(name, start):
    """Decoding through cache and states, over page borders, equals the whole prompt."""
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
    xs = [ids(n + 30, 10 + n) for n in lens]
    want = [oracle.forward(reference(cfg, t), x) for x in xs]
    e = engine(cfg, t)
    seqs = [e.open_sequence() for _ in xs]
    out = e.feed([(s, x[:n], [n - 1, 0]) for s, x, n in zip(seqs, xs, lens)])
    assert close(out, torch.cat([w[[n - 1, 0]] for w, n in zip(want, lens)]))
    live = list(range(4))
    for j in range(30):                                                  # the first sequence ends early
        if j == 12:
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


def test_what_a_changed_token_reaches():
    """Everything behind it and nothing ahead of it, through a layer of either kind, in prompts and in decoding."""
    x = ids(40, 4)
    for layer in (cases.attention(), cases.mamba()):
        cfg, t = cases.model([layer], seed=4)
        for j in (0, 1, 15, 24):
            y = list(x)
            y[j] = (x[j] + 1) % 61
            e = engine(cfg, t)
            a, b = e.open_sequence(), e.open_sequence()
            out = e.feed([(a, x[:25], range(25)), (b, y[:25], range(25))])
            diff = [(out[i] - out[25 + i]).abs().max().item() for i in range(25)]
            for i in range(25, 40):
                out = e.feed([(a, [x[i]], [0]), (b, [y[i]], [0])])
                diff.append((out[0] - out[1]).abs().max().item())
            assert all(d < 5e-6 for d in diff[:j]) and all(d > 5e-5 for d in diff[j:])


def test_pages_and_slots_that_are_used_again():
    cfg, t = build("mixed", seed=6)
    x, y = ids(150, 6), ids(120, 7)
    want, want_y = (oracle.forward(reference(cfg, t), z) for z in (x, y))
    e = engine(cfg, t, max_pages=3, max_active=1)
    s = e.open_sequence()
    got = [e.feed([(s, x[:100], [99])])] + [e.feed([(s, [x[j]], [0])]) for j in range(100, 150)]
    assert close(torch.cat(got), want[99:]) and e.kv.pages_in_use == 3
    e.close_sequence(s)
    assert e.kv.pages_in_use == 0
    s = e.open_sequence()                                                 # its first tokens see nothing of the old states
    got = [e.feed([(s, y[:70], range(70))])] + [e.feed([(s, [y[j]], [0])]) for j in range(70, 120)]
    assert close(torch.cat(got), want_y)
    e.close_sequence(s)
    s = e.open_sequence()
    assert close(e.feed([(s, y[:1], [0])]), want_y[:1])                  # a prompt of one token
    with pytest.raises(RuntimeError):
        e.feed([(s, ids(400), [])])                                      # more than the pool holds


def test_without_attention_the_pages_come_back():
    cfg, t = cases.model([cases.mamba(mlp=cases.moe()), cases.mamba(heads=2, groups=1)], seed=7)
    x = ids(300, 6)
    e = engine(cfg, t, max_pages=6, max_active=1)
    s = e.open_sequence()
    got = [e.feed([(s, x[:290], [289])])]
    assert e.kv.pages_in_use <= 1 and e.model.cache_window() == 1
    got += [e.feed([(s, [x[j]], [0])]) for j in range(290, 300)]
    assert close(torch.cat(got), oracle.forward(reference(cfg, t), x)[289:])


def test_positions_end_with_their_table():
    cfg, t = cases.model(cases.SINGLE, seed=14, max_positions=40)
    e = engine(cfg, t)
    s = e.open_sequence()
    x = ids(40)
    got = [e.feed([(s, x[:39], [38])]), e.feed([(s, x[39:], [0])])]
    assert close(torch.cat(got), oracle.forward(reference(cfg, t), x)[38:])
    with pytest.raises(ValueError):
        e.feed([(s, [1], [0])])


def test_greedy_generation_through_the_scheduler():
    cfg, t = build("mixed", seed=8, width=40)
    ref = reference(cfg, t)
    prompts = [ids(n, 20 + n) for n in (5, 40, 1, 37)]
    want = [oracle.generate(ref, p, 8) for p in prompts]
    e = engine(cfg, t, max_active=2, spec_tokens=2)                       # two at a time: the others wait
    assert e.generate(prompts[0], GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want[0]
    for i, p in enumerate(prompts):
        e.submit_request(Request(100 + i, p, GenerationConfig(max_new_tokens=8, **GREEDY)))
    got = {}
    while e.num_active():
        e.step()
        got.update({r.request_id: r.token_ids for r in e.poll_responses()})
    assert [got[100 + i] for i in range(4)] == want
    assert e.kv.pages_in_use == 0 and sorted(e.free_rows) == [0, 1]
    assert not e.model.rewinds and e.spec_drafted == 0                   # convolutions cannot take a token back
    stop = want[1][3]
    assert e.generate(prompts[1], GenerationConfig(max_new_tokens=8, stop_tokens=[stop], **GREEDY)).token_ids == want[1][:want[1].index(stop) + 1]
    emb = e.embed(prompts[1])
    assert emb.shape == (40,) and abs(float(emb.norm()) - 1) < 1e-5


def test_sampled_generation_and_text():
    cfg, t = cases.model(cases.EVEN, seed=9, vocab=300)
    e = engine(cfg, t)
    r = e.generate("abc", GenerationConfig(max_new_tokens=6, temperature=1.0, top_k=20))
    assert len(r.token_ids) == 6 and all(0 <= i < 300 for i in r.token_ids)


# ------------------------------------------------------------------------------------------ configuration, loading, tools
def save(path, cfg, t):
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(t, os.path.join(path, "model.safetensors"))


def test_configuration_and_registry():
    cfg, t = build("mixed")
    assert "tifepel" in known_models() and resolve_architecture(cfg).config is TifepelConfig
    c = TifepelConfig.from_dict(cfg)
    assert TifepelConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    for edit in (lambda d: d["layers"][0].update(type="lightning"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                 lambda d: d["layers"][1]["mixer"].update(heads=5, kv_heads=2), lambda d: d["layers"][0]["mlp"]["router"].update(top=11),
                 lambda d: d["layers"][0]["mixer"].update(groups=4), lambda d: d["layers"][0]["mixer"].update(norm_groups=7),
                 lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=0), lambda d: d["loop"].update(stop=9), lambda d: d["layers"][2]["mixer"].update(conv=0),
                 lambda d: d.update(streams=0), lambda d: d["canon"].update(taps=0)):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(ValueError):
            TifepelConfig.from_dict(bad)
    wrong = dict(t)
    wrong["l0.mix.in"] = torch.zeros(3, 3)
    with pytest.raises(ValueError):
        cases.weights(cfg, wrong)
    back = cases.weights(cfg, t).state_dict()
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    w = TifepelWeights.random(c, seed=3)
    assert w.num_parameters() > 0 and all(math.isfinite(float(v.float().sum())) for v in w.state_dict().values())
    e = LLMEngine(device="cpu", max_pages=8, max_active=1)
    e.set_weights(w)
    assert e.weights.num_parameters() == w.num_parameters() and torch.isfinite(e.feed([(e.open_sequence(), ids(30), [29])])).all()


def test_what_a_configuration_may_leave_out():
    cfg, t = cases.model([cases.attention(coef=0.0, mlp=cases.moe(identity=0, shared=0)), cases.mamba()], seed=13)
    x = ids(20)
    want = oracle.forward(reference(cfg, t), x)
    del cfg["layers"][0]["mixer"]["q_temp"], cfg["layers"][0]["mlp"]["shared"], cfg["layers"][0]["mlp"]["router"]["identity"], cfg["layers"][1]["mlp"]
    cfg["loop"] = None
    e = engine(cfg, t)
    assert close(e.feed([(e.open_sequence(), x, range(20))]), want)


def test_load_and_serve(tmp_path):
    from prometorch_b200.serve import PagedBackend
    cfg, t = cases.model(cases.EVEN, seed=10, loop=(1, 3, 2))
    save(tmp_path, cfg, t)
    e = LLMEngine(device="cpu", max_pages=8, max_active=2)
    assert e.load(str(tmp_path)) and e.model.architecture == "tifepel"
    p = ids(9, 3)
    want = oracle.generate(reference(cfg, t), p, 8)
    assert e.generate(p, GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want
    b = PagedBackend(str(tmp_path), "m", "cpu", max_active=2, max_pages=8)
    out = []
    b.generate(p, {"num_predict": 8, "temperature": 0.0, "repeat_penalty": 1.0}, lambda tok: out.append(tok) or True)
    assert out == want and b.architecture == "tifepel"
    b.server.close()


def test_generate_command(tmp_path, capsys):
    from prometorch_b200 import generate
    cfg, t = cases.model(cases.EVEN, seed=11, vocab=300)
    save(tmp_path, cfg, t)
    assert generate.main([str(tmp_path), "hey", "--device", "cpu", "--greedy", "--max-tokens", "5"]) == 0
    assert "tifepel" in capsys.readouterr().out
    assert generate.main([str(tmp_path), "--info", "--tensors"]) == 0
    out = capsys.readouterr().out
    assert "l1.mix.A_log" in out and "architecture = 'Tifepel'" in out


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
