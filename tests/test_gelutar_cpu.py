"""Gelutar on CPU: each mechanism and the whole model in the batching engine against tests/gelutar_oracle.py."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gelutar_cases as cases  # noqa: E402
import gelutar_oracle as oracle  # noqa: E402

from prometorch_b200.models.gelutar import GelutarConfig, GelutarWeights  # noqa: E402
from prometorch_b200.models.paged import RowPack, known_models, resolve_architecture  # noqa: E402
from prometorch_b200.ops import gemm, recurrence as R, residual as S, window_attention as A  # noqa: E402
from prometorch_b200.serve.llm import PAGE, GenerationConfig, LLMEngine, Request, save_safetensors  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, repetition_penalty=1.0, top_k=1)
MODELS = {"mixed": cases.MIXED, "even": cases.EVEN, "single": cases.SINGLE}


def ids(n, seed=0, vocab=61):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def reference(cfg, t):
    return {"config": cfg, "tensors": oracle.cast(t)}


def engine(cfg, t, max_pages=16, max_active=6, **kw):
    e = LLMEngine(device="cpu", dtype=torch.float32, max_pages=max_pages, max_active=max_active, **kw)
    e.set_weights(cases.weights(cfg, t))
    return e


def close(a, b, tol=2e-5):
    a, b = a.double(), b.double()
    return float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max()))


# ------------------------------------------------------------------------------------------ window attention
def paged(a, n, seed=1, pages=8):
    """q, k, v of n tokens; k and v in scattered pages of one sequence (page-table row 1)."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(n, h, d, generator=g) for h, d in ((a.heads, a.dim), (a.kv_heads, a.dim), (a.kv_heads, a.vdim)))
    order = torch.randperm(pages, generator=g)
    table = torch.zeros(2, pages, dtype=torch.int32)
    table[1] = order.int()
    kp, vp = torch.zeros(pages, a.kv_heads, PAGE, a.dim_stored), torch.zeros(pages, a.kv_heads, PAGE, a.vdim_stored)
    for j in range(n):
        kp[order[j // PAGE], :, j % PAGE, :a.dim], vp[order[j // PAGE], :, j % PAGE, :a.vdim] = k[j], v[j]
    qs = torch.zeros(n, a.heads, a.dim_stored)
    qs[..., :a.dim] = q
    return q, k, v, qs, table, kp, vp


def rows(n):
    return torch.arange(n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)


@pytest.mark.parametrize("H,G,D,Dv,W,keep", [(3, 3, 20, 28, 9, 2), (6, 2, 16, 12, 70, 0), (4, 1, 8, 8, 1, 5), (2, 2, 16, 16, 64, 64), (2, 1, 8, 8, 500, 3)])
def test_window_attention(H, G, D, Dv, W, keep):
    sink = torch.linspace(-2, 3, H)
    a = A.WindowAttention(H, G, D, Dv, W, keep, 0.4, sink)
    n = 150
    q, k, v, qs, table, kp, vp = paged(a, n)
    gate = torch.randn(n, H)
    got = A.window_attention(qs, a, *rows(n), table, kp, vp, 1, n, gate).view(n, H, Dv)
    want = oracle.attention_rows(q.double(), k.double(), v.double(), 0.4, W, keep, sink.double())
    assert close(got, want * torch.sigmoid(gate.double())[..., None])


@pytest.mark.parametrize("W,keep", [(5, 3), (63, 1), (64, 64), (65, 70), (100, 0)])
def test_window_and_kept_tokens_edges(W, keep):
    """A value that stands out counts for W places, for all later ones if it is among the kept tokens, and never before its own."""
    a = A.WindowAttention(2, 1, 16, 16, W, keep, 0.3, torch.zeros(2))
    n = 170
    q, k, v, qs, table, kp, vp = paged(a, n)
    base = A.window_attention(qs, a, *rows(n), table, kp, vp, 1, n)
    for j in (0, 2, 3, 13, 63, 64, 69, 70):
        vp2 = vp.clone()
        vp2[table[1, j // PAGE], :, j % PAGE] += 1e4
        d = (A.window_attention(qs, a, *rows(n), table, kp, vp2, 1, n) - base).abs().amax(1)
        assert (d > 1e-2).nonzero()[:, 0].tolist() == [i for i in range(n) if oracle.visible(i, j, W, keep)]


def test_sink_takes_its_share():
    a = A.WindowAttention(1, 1, 8, 8, 4, 0, 1.0, torch.tensor([50.0]))
    q, k, v, qs, table, kp, vp = paged(a, 20)
    assert float(A.window_attention(qs, a, *rows(20), table, kp, vp, 1, 20).abs().max()) < 1e-6          # the sink has everything
    a.sink = torch.tensor([0.0])
    one = A.window_attention(qs[:1] * 0, a, *rows(1), table, kp, vp, 1, 1)
    assert close(one[0], v[0, 0] / 2)                                                                    # one key with score 0 beside exp(0)
    a.sink = None
    assert close(A.window_attention(qs[:1], a, *rows(1), table, kp, vp, 1, 1)[0], v[0, 0])


def test_projection_norm_and_pages():
    a = A.WindowAttention(4, 2, 12, 20, 5, 0, 1.0)
    n, eps = 70, 1e-3
    p, cols = torch.randn(n, 48 + 24 + 40 + 9), (3, 56, 81)
    qw, kw = torch.randn(48), torch.randn(24)
    kp, vp = torch.full((3, 2, PAGE, 16), 7.0), torch.full((3, 2, PAGE, 32), 7.0)
    table = torch.tensor([[0, 0], [2, 1]], dtype=torch.int32)
    pos, req = torch.arange(n, dtype=torch.int32) + 10, torch.ones(n, dtype=torch.int32)
    q = A.proj_norm_write(p, cols, a, qw, kw, eps, pos, req, table, kp, vp)
    x = p.double()
    assert close(q[..., :12], oracle.plain_norm(x[:, 3:51], qw.double(), eps).view(n, 4, 12)) and float(q[..., 12:].abs().max()) == 0
    k, v = oracle.plain_norm(x[:, 56:80], kw.double(), eps).view(n, 2, 12), x[:, 81:].view(n, 2, 20)
    for i in (0, 5, 53, 54, 69):                                         # 54 + 10 = the first slot of the second page
        page, slot = int(table[1, (i + 10) // PAGE]), (i + 10) % PAGE
        assert close(kp[page, :, slot, :12], k[i]) and close(vp[page, :, slot, :20], v[i])
    assert float(kp[0].min()) == 7.0 and float(kp[2, :, :10].min()) == 7.0


# ------------------------------------------------------------------------------------------ recurrences
def seqs_of(lens, starts, slots):
    offs = [0]
    for n in lens:
        offs.append(offs[-1] + n)
    s = R.Sequences.of(offs, starts, slots, "cpu")
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in zip(starts, lens)])
    req = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in zip(slots, lens)])
    return s, pos, req


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_short_convolution_in_portions(taps):
    """Whole, cut into portions shorter than the taps, and token by token; the slot's old content does not leak into position 0."""
    C, n = 10, 23
    x, w = torch.randn(n, C), torch.randn(taps, C)
    want = oracle.silu(oracle.causal_conv(x.double(), w.t().double()))
    for cuts in ([23], [1, 2, 1, 3, 16], [1] * 23):
        state, at = torch.full((3, taps - 1, C), 9.0), 0
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [2])
            y = R.short_conv(x[at:at + m], w, state, pos, req, s if m > 1 else None)
            assert close(y, want[at:at + m])
            at += m
        assert taps == 1 or close(state[2], x[n - taps + 1:]) and float(state[:2].min()) == 9.0


def delta_case(H=4, G=2, D=12, Dv=20, n=40, seed=0):
    g = torch.Generator().manual_seed(seed)
    r = R.DeltaRule(H, G, D, Dv, torch.rand(H, generator=g) + 0.3, torch.randn(H * D, generator=g) - 1)
    x, beta, a = (torch.randn(n, w, generator=g) for w in (2 * G * D + H * Dv, H, H * D))
    return r, x, beta, a


def delta_oracle(r, x, beta, a):
    n, H, G, D, Dv = x.shape[0], r.heads, r.kv_heads, r.dim, r.vdim
    x = x.double()
    q, k = oracle.unit(x[:, :G * D].view(n, G, D)) * D ** -0.5, oracle.unit(x[:, G * D:2 * G * D].view(n, G, D))
    v = x[:, 2 * G * D:].view(n, H, Dv)
    g = oracle.delta_decay(a.double().view(n, H, D), r.rate.double().log(), r.dt_bias.double().view(H, D))
    out, S = torch.zeros(n, H, Dv, dtype=torch.float64), [torch.zeros(D, Dv, dtype=torch.float64)] * H
    for i in range(n):
        for h in range(H):
            S[h], out[i, h] = oracle.delta_step(S[h], q[i, h // (H // G)], k[i, h // (H // G)], v[i, h], g[i, h], oracle.sigmoid(beta[i, h].double()))
    return out.view(n, H * Dv), torch.stack(S)


def test_delta_rule_in_portions():
    r, x, beta, a = delta_case()
    want, S = delta_oracle(r, x, beta, a)
    for cuts in ([40], [2] * 20, [1, 38, 1], [17, 23]):
        state, at, out = torch.full((3, 4, 12, 20), 5.0), 0, []
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [1])
            out.append(R.delta_rule(x[at:at + m], r, beta[at:at + m], a[at:at + m], state, pos, req, s if m > 1 else None))
            at += m
        assert close(torch.cat(out), want) and close(state[1], S) and float(state[0].min()) == 5.0


def test_delta_rule_takes_factors_of_its_decays():
    r, x, beta, _ = delta_case()
    low, w = torch.randn(40, 6), torch.randn(48, 6)
    s, pos, req = seqs_of([40], [0], [0])
    want, S = delta_oracle(r, x, beta, low @ w.t())
    state = torch.zeros(1, 4, 12, 20)
    assert close(R.delta_rule(x, r, beta, (low, w), state, pos, req, s), want) and close(state[0], S)


def test_delta_rule_overwrites_a_key():
    """Two tokens with one key: with beta near 1 and no decay the second value replaces the first."""
    r = R.DeltaRule(1, 1, 4, 3, torch.tensor([1e-6]), torch.zeros(4))
    k = torch.tensor([0.0, 3.0, 0.0, 0.0])
    x = torch.stack([torch.cat([k, k, torch.tensor(v)]) for v in ([1.0, 2.0, 3.0], [-4.0, 5.0, 6.0])])
    s, pos, req = seqs_of([2], [0], [0])
    o = R.delta_rule(x, r, torch.full((2, 1), 30.0), torch.zeros(2, 4), torch.zeros(1, 1, 4, 3), pos, req, s)
    assert close(o * 2, x[:, 8:], 1e-4)                                 # q carries dim ** -0.5


def test_decay_attention_in_portions():
    H, D, Dv, n = 3, 8, 12, 30
    r = R.DecayAttention(H, D, Dv, torch.tensor([0.0, 0.7, 1.0]))
    x, cols = torch.randn(n, 2 * H * D + H * Dv + 5), (5, 5 + H * D, 5 + 2 * H * D)
    f = x.double()
    q, k, v = (oracle.silu(f[:, c:c + H * d]).view(n, H, d) for c, d in zip(cols, (D, D, Dv)))
    want = torch.zeros(n, H, Dv, dtype=torch.float64)
    for h in range(H):
        S = torch.zeros(D, Dv, dtype=torch.float64)
        for i in range(n):
            S, want[i, h] = oracle.lightning_step(S, q[i, h], k[i, h], v[i, h], float(r.decay[h]))
    for cuts in ([30], [2] * 15, [1] * 30):
        state, at, out = torch.full((2, H, D, Dv), 5.0), 0, []
        for m in cuts:
            s, pos, req = seqs_of([m], [at], [1])
            out.append(R.decay_attention(x[at:at + m], r, cols, state, pos, req, s if m > 1 else None))
            at += m
        assert close(torch.cat(out), want.view(n, -1)) and float(state[0].min()) == 5.0


def test_group_norm_and_gate():
    o, gate = torch.randn(5, 24), torch.randn(5, 40)
    for gs in (8, 24):
        w = torch.randn(gs)
        want = oracle.plain_norm(o.double().view(5, -1, gs), w.double(), 1e-2).reshape(5, 24) * oracle.sigmoid(gate[:, 9:33].double())
        assert close(R.group_norm_gate(o, w, gate[:, 9:33], 1e-2, torch.float32), want)


# ------------------------------------------------------------------------------------------ around the mixers
def test_residual_norm():
    x, y, z, eps = torch.randn(5, 24), torch.randn(5, 24), torch.randn(3, 5, 24), 1e-2
    w = [torch.randn(24) for _ in range(3)]
    want = x.double() + 0.5 * oracle.plain_norm(y.double(), w[0].double(), eps) + 0.25 * oracle.plain_norm(z.double().sum(0), w[1].double(), eps)
    h = S.residual_norm(x, [S.Branch(y, 0.5, w[0]), S.Branch(z, 0.25, w[1])], eps, w[2], torch.float32)
    assert close(x, want) and close(h, oracle.plain_norm(want, w[2].double(), eps))
    assert S.residual_norm(x, [S.Branch(y)], eps) is None and close(x, want + y.double())


def test_squared_relu_and_row_pack():
    x, w = torch.randn(4, 8), torch.randn(6, 8)
    assert close(gemm.linear_relu2(x, w), torch.relu(x.double() @ w.double().t()) ** 2)
    p = RowPack({"a": 3, "b": 8, "c": 9})
    parts = {n: torch.randn(k, 8) for n, k in p.sizes.items()}
    m = p.pack(parts)
    assert m.shape[0] == p.rows == 32 and p.at == {"a": 0, "b": 8, "c": 16}
    assert all(close(p.cols(x @ m.t(), n), x @ t.t()) for n, t in parts.items()) and p.cols(x @ m.t(), "c", padded=True).shape[1] == 16


# ------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompt(name):
    cfg, t = cases.model(MODELS[name])
    x = ids(150)
    e = engine(cfg, t)
    assert close(e.feed([(e.open_sequence(), x, range(150))]), oracle.forward(reference(cfg, t), x))


def test_every_layer():
    """A model cut off after each of its layers."""
    for k in range(len(cases.MIXED) + 1):
        cfg, t = cases.model(cases.MIXED[:k], seed=20)
        x = ids(40, 3)
        e = engine(cfg, t)
        assert close(e.feed([(e.open_sequence(), x, range(40))]), oracle.forward(reference(cfg, t), x)), k


@pytest.mark.parametrize("name", ["mixed", "single"])
@pytest.mark.parametrize("start", [1, 60])
def test_token_by_token(name, start):
    """Decoding through cache and state, over page borders and past every window, equals the whole prompt."""
    cfg, t = cases.model(MODELS[name], seed=1)
    x = ids(145, 1)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    got = [e.feed([(s, x[:start], range(start))])] + [e.feed([(s, [x[j]], [0])]) for j in range(start, len(x))]
    assert close(torch.cat(got), want)


@pytest.mark.parametrize("portion", [2, 7, 64, 65])
def test_portions(portion):
    cfg, t = cases.model(cases.MIXED, seed=2)
    x = ids(140, 2)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    got = [e.feed([(s, x[lo:lo + portion], range(len(x[lo:lo + portion])))]) for lo in range(0, len(x), portion)]
    assert close(torch.cat(got), want)


def test_unequal_batch_against_each_alone():
    cfg, t = cases.model(cases.MIXED, seed=3)
    lens = [1, 64, 90, 3]
    xs = [ids(n + 70, 10 + n) for n in lens]
    want = [oracle.forward(reference(cfg, t), x) for x in xs]
    e = engine(cfg, t)
    seqs = [e.open_sequence() for _ in xs]
    out = e.feed([(s, x[:n], [n - 1, 0]) for s, x, n in zip(seqs, xs, lens)])
    assert close(out, torch.cat([w[[n - 1, 0]] for w, n in zip(want, lens)]))
    live = list(range(4))
    for j in range(70):                                                  # the first sequence ends early
        if j == 20:
            e.close_sequence(seqs[0])
            live.remove(0)
        out = e.feed([(seqs[i], [xs[i][lens[i] + j]], [0]) for i in live])
        assert close(out, torch.stack([want[i][lens[i] + j] for i in live]))


def test_portions_of_one_beside_the_first_tokens_of_another():
    """One batch: a sequence that goes on by three tokens, one by a single token, and one that starts."""
    cfg, t = cases.model(cases.MIXED, seed=4)
    x, y, z = ids(80, 1), ids(40, 2), ids(70, 3)
    want = [oracle.forward(reference(cfg, t), v) for v in (x, y, z)]
    e = engine(cfg, t)
    a, b, c = (e.open_sequence() for _ in range(3))
    e.feed([(a, x[:77], []), (b, y[:39], [])])
    out = e.feed([(a, x[77:], [0, 2]), (b, y[39:], [0]), (c, z, [69])])
    assert close(out, torch.stack([want[0][77], want[0][79], want[1][39], want[2][69]]))


def test_a_layer_forgets_what_left_its_window():
    """Without the recurrent half a token is seen window - 1 places later and no further unless it is kept; in a prompt and in
    decoding."""
    W, keep = 11, 2
    cfg, t = cases.model([cases.parallel(window=W, keep=keep, ff=0)], seed=4)
    t["l0.mix.right.out"] = torch.zeros_like(t["l0.mix.right.out"])
    x = ids(40, 4)
    for j, seen in ((15, list(range(15, 15 + W))), (1, list(range(1, 40))), (2, list(range(2, 2 + W)))):
        y = list(x)
        y[j] = (x[j] + 1) % 61
        e = engine(cfg, t)
        a, b = e.open_sequence(), e.open_sequence()
        out = e.feed([(a, x[:22], range(22)), (b, y[:22], range(22))])
        diff = [(out[i] - out[22 + i]).abs().max().item() for i in range(22)]
        for i in range(22, 40):
            out = e.feed([(a, [x[i]], [0]), (b, [y[i]], [0])])
            diff.append((out[0] - out[1]).abs().max().item())
        assert [i for i, d in enumerate(diff) if d > 1e-5] == seen


def test_pages_and_slots_come_back_and_are_reused():
    """A pool smaller than the sequence: pages between the kept tokens and every window return while it runs; freed pages and state
    slots serve another one, whose first tokens see nothing of the old state."""
    cfg, t = cases.model([cases.parallel(window=20, keep=3, heads=4, kv=2), cases.lightning(), cases.parallel(window=50, keep=66, heads=4, kv=2)], seed=6)
    x, y = ids(400, 6), ids(120, 7)
    want, want_y = (oracle.forward(reference(cfg, t), z) for z in (x, y))
    e = engine(cfg, t, max_pages=5, max_active=1)
    s = e.open_sequence()
    got = [e.feed([(s, x[:100], [99])])]
    for j in range(100, 400):
        got.append(e.feed([(s, [x[j]], [0])]))
        assert e.kv.pages_in_use <= 4                                    # two kept pages and at most two of the window
    assert close(torch.cat(got), want[99:]) and s.pages[0] >= 0 and s.pages[1] >= 0 and s.pages[2] == -1
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


def test_greedy_generation_through_the_scheduler():
    cfg, t = cases.model(cases.MIXED, seed=8)
    ref = reference(cfg, t)
    prompts = [ids(n, 20 + n) for n in (5, 70, 1, 64)]
    want = [oracle.generate(ref, p, 12) for p in prompts]
    e = engine(cfg, t, max_active=2)                                     # two at a time: the others wait
    assert e.generate(prompts[0], GenerationConfig(max_new_tokens=12, **GREEDY)).token_ids == want[0]
    for i, p in enumerate(prompts):
        e.submit_request(Request(100 + i, p, GenerationConfig(max_new_tokens=12, **GREEDY)))
    got = {}
    while e.num_active():
        e.step()
        got.update({r.request_id: r.token_ids for r in e.poll_responses()})
    assert [got[100 + i] for i in range(4)] == want
    assert e.kv.pages_in_use == 0 and sorted(e.free_rows) == [0, 1]
    stop = want[1][3]
    assert e.generate(prompts[1], GenerationConfig(max_new_tokens=12, stop_tokens=[stop], **GREEDY)).token_ids == want[1][:want[1].index(stop) + 1]
    spec = engine(cfg, t, spec_tokens=3)                                 # a recurrent state cannot take proposals back: plain decoding
    rep = (prompts[0] * 6)[:30]
    assert spec.generate(rep, GenerationConfig(max_new_tokens=12, **GREEDY)).token_ids == oracle.generate(ref, rep, 12)
    assert spec.spec_drafted == 0
    emb = e.embed(prompts[1])
    assert emb.shape == (48,) and abs(float(emb.norm()) - 1) < 1e-5


def test_layers_without_pages():
    """A model of recurrent layers alone holds no keys."""
    cfg, t = cases.model([cases.lightning(), cases.lightning(heads=2, dim=5, vdim=7, decay=[0.2, 0.999], ff=0)], seed=9)
    x = ids(150, 9)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    got = [e.feed([(s, x[:90], range(90))])] + [e.feed([(s, [x[j]], [0])]) for j in range(90, 150)]
    assert close(torch.cat(got), want) and all(k.numel() == 0 for k in e.kv.k)


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
    cfg, t = cases.model(cases.MIXED)
    assert "gelutar" in known_models() and resolve_architecture(cfg).config is GelutarConfig
    c = GelutarConfig.from_dict(cfg)
    assert GelutarConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    for edit in (lambda d: d["layers"][0].update(type="attention"), lambda d: d["layers"][0]["mlp"].update(kind="sparse"),
                 lambda d: d["layers"][1]["mixer"]["left"].update(heads=5, kv_heads=2), lambda d: d["layers"][0]["mixer"]["decay"].pop(),
                 lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(size=0)):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(ValueError):
            GelutarConfig.from_dict(bad)
    wrong = dict(t)
    wrong["l1.mix.right.a2"] = torch.zeros(3, 3)
    with pytest.raises(ValueError):
        cases.weights(cfg, wrong)
    back = cases.weights(cfg, t).state_dict()
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    w = GelutarWeights.random(c, seed=3, rank=5)
    assert w.num_parameters() > 0 and all(math.isfinite(float(v.float().sum())) for v in w.state_dict().values())
    e = LLMEngine(device="cpu", max_pages=8, max_active=1)
    e.set_weights(w)
    assert e.weights.num_parameters() == w.num_parameters() and torch.isfinite(e.feed([(e.open_sequence(), ids(30), [29])])).all()


def test_load_and_serve(tmp_path):
    from prometorch_b200.serve import PagedBackend
    cfg, t = cases.model(cases.EVEN, seed=10)
    save(tmp_path, cfg, t)
    e = LLMEngine(device="cpu", max_pages=8, max_active=2)
    assert e.load(str(tmp_path)) and e.model.architecture == "gelutar"
    p = ids(9, 3)
    want = oracle.generate(reference(cfg, t), p, 8)
    assert e.generate(p, GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want
    b = PagedBackend(str(tmp_path), "m", "cpu", max_active=2, max_pages=8)
    out = []
    b.generate(p, {"num_predict": 8, "temperature": 0.0, "repeat_penalty": 1.0}, lambda tok: out.append(tok) or True)
    assert out == want and b.architecture == "gelutar"
    b.server.close()


def test_generate_command(tmp_path, capsys):
    from prometorch_b200 import generate
    cfg, t = cases.model(cases.EVEN, seed=11, vocab=300)
    save(tmp_path, cfg, t)
    assert generate.main([str(tmp_path), "hey", "--device", "cpu", "--greedy", "--max-tokens", "5"]) == 0
    assert "gelutar" in capsys.readouterr().out
    assert generate.main([str(tmp_path), "--info", "--tensors"]) == 0
    out = capsys.readouterr().out
    assert "l1.mix.norm" in out and "architecture = 'Gelutar'" in out


def test_trace_replay(tmp_path):
    """bin/trace_run on CPU: prompts and decoding of two requests, one of which ends early; logits against the oracle."""
    cfg, t = cases.model(cases.MIXED, seed=12)
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
