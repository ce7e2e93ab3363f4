"""Kifusun on CPU: each mechanism and the whole model in the batching engine against tests/kifusun_oracle.py."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kifusun_cases as cases  # noqa: E402
import kifusun_oracle as oracle  # noqa: E402

from prometorch_b200.models.kifusun import KifusunConfig, KifusunWeights  # noqa: E402
from prometorch_b200.models.paged import known_models, resolve_architecture  # noqa: E402
from prometorch_b200.ops import gated_attention as A  # noqa: E402
from prometorch_b200.ops import residual as S  # noqa: E402
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


# ------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("rows,dmax,window", [(10, 50, 90), (8, 64, 70), (32, 256, 300), (7, 33, 40), (16, 100.5, 200), (2, 9, 12), (32, 120, 20)])
def test_distance_buckets(rows, dmax, window):
    got = A.distance_buckets(rows, dmax, window).tolist()
    assert got == [oracle.distance_bucket(n, rows, dmax) for n in range(window)]
    assert max(got) <= rows - 1 and got == sorted(got)


def test_distance_buckets_on_an_edge():
    """half = 4, (64 / 4)^(k / 4) = 2^k: the buckets change exactly at 4, 8, 16 and 32."""
    b = A.distance_buckets(8, 64, 80).tolist()
    assert [n for n in range(1, 80) if b[n] != b[n - 1]] == [1, 2, 3, 4, 8, 16, 32]
    with pytest.raises(ValueError):
        A.distance_buckets(16, 8, 20)


def test_distance_bias_folds_the_head_number():
    rel, pb = torch.randn(10, 3), torch.randn(3)
    t = A.distance_bias(rel, 50, 200, pb)
    for n in (0, 1, 4, 5, 7, 20, 49, 50, 199):
        want = rel[oracle.distance_bucket(n, 10, 50)] + pb
        assert torch.allclose(t[:, min(n, t.shape[1] - 1)], want)
    assert A.distance_bias(rel, 50, 3).shape == (3, 3)                   # no longer than the window


def gated(H=3, G=3, D=20, Dv=28, W=9, talk=True, cap=4.0, seed=0, rows=10, dmax=50):
    g = torch.Generator().manual_seed(seed)
    rel, pb = torch.randn(rows, H, generator=g), torch.randn(H, generator=g) - 1
    T = torch.randn(H, H, generator=g) * 0.5 + torch.eye(H)
    a = A.GatedAttention(H, G, D, Dv, W, 0.3, cap, A.distance_bias(rel, dmax, W, pb), T if talk else None)
    return a, dict(scale=0.3, cap=cap if cap else 1e9, window=W, rel=rel.double(), dmax=dmax, pb=pb.double(), talk=T.double() if talk else torch.eye(H).double())


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


@pytest.mark.parametrize("kw", [dict(), dict(H=6, G=2, W=70, talk=True), dict(H=4, G=1, W=1), dict(H=2, G=2, D=16, Dv=16, W=64, talk=False, cap=0.0)])
def test_gated_attention_against_the_oracle(kw):
    a, o = gated(**kw)
    n = 150
    q, k, v, qs, table, kp, vp = paged(a, n)
    pos, req = torch.arange(n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)
    got = A.gated_attention(qs, a, pos, req, table, kp, vp, 1, n).view(n, a.heads, a.vdim)
    assert close(got, oracle.attention_rows(q.double(), k.double(), v.double(), **o))


@pytest.mark.parametrize("W", [5, 63, 64, 65, 100])
def test_window_edges(W):
    """A key whose score stands out counts at distance W - 1 and not at W, also across a page border."""
    a, o = gated(H=2, G=1, D=16, Dv=16, W=W, cap=30.0)
    n = 140
    q, k, v, qs, table, kp, vp = paged(a, n)
    for j in (0, 13, 63, 64):
        vp2 = vp.clone()
        vp2[table[1, j // PAGE], :, j % PAGE] += 50.0
        pos, req = torch.arange(n, dtype=torch.int32), torch.ones(n, dtype=torch.int32)
        d = (A.gated_attention(qs, a, pos, req, table, kp, vp2, 1, n) - A.gated_attention(qs, a, pos, req, table, kp, vp, 1, n)).abs().amax(1)
        touched = (d > 1e-3).nonzero()[:, 0].tolist()
        assert touched == list(range(j, min(n, j + W)))


def test_oracle_weights_one_by_one():
    """The two forms of the oracle agree: weights pair by pair, then mixed, and whole rows."""
    a, o = gated(H=4, G=2, W=6)
    q, k, v, *_ = paged(a, 20)
    q, k, v = q.double(), k.double(), v.double()
    rows = oracle.attention_rows(q, k, v, **o)
    for i in (0, 3, 6, 19):
        w = oracle.attention_weights(q[i], k, i, list(range(20)), o["scale"], o["cap"], o["window"], o["rel"], o["dmax"], o["pb"])
        w = oracle.mix_heads(w, o["talk"])
        assert close(torch.stack([w[h] @ v[:, h // 2] for h in range(4)]), rows[i], 1e-12)


def test_head_norm_and_value_mixing_into_pages():
    a, _ = gated(H=4, G=2, D=12, Dv=20)
    n, eps = 70, 1e-3
    qkv, first = torch.randn(n, 4 * 12 + 2 * 32), torch.randn(n, 40)
    qw, kw = torch.randn(12), torch.randn(12)
    kp, vp = torch.full((3, 2, PAGE, 16), 7.0), torch.full((3, 2, PAGE, 32), 7.0)
    table = torch.tensor([[0, 0], [2, 1]], dtype=torch.int32)
    pos, req = torch.arange(n, dtype=torch.int32) + 10, torch.ones(n, dtype=torch.int32)
    q = A.head_norm_write(qkv, a, qw, kw, eps, pos, req, table, kp, vp, first, 0.3)
    x = qkv.double()
    assert close(q[..., :12], oracle.head_norm(x[:, :48].view(n, 4, 12), qw.double(), eps)) and float(q[..., 12:].abs().max()) == 0
    k = oracle.head_norm(x[:, 48:72].view(n, 2, 12), kw.double(), eps)
    v = oracle.mix_values(x[:, 72:].view(n, 2, 20), first.double().view(n, 2, 20), 0.3)
    for i in (0, 5, 53, 54, 69):                                         # 54 + 10 = the first slot of the second page
        page, slot = int(table[1, (i + 10) // PAGE]), (i + 10) % PAGE
        assert close(kp[page, :, slot, :12], k[i]) and close(vp[page, :, slot, :20], v[i])
    assert float(kp[0].min()) == 7.0 and float(kp[2, :, :10].min()) == 7.0


def test_residual_stream():
    x, y, g, eps = torch.randn(5, 24), torch.randn(5, 24), 1.3, 1e-2
    want = x.double() + oracle.scalar_norm(y.double(), g, eps)
    s = S.post_norm_add(y, (x, x), g, eps)
    assert s[0] is s[1] and close(s[0], want)
    xb = torch.empty(5, 24, dtype=torch.bfloat16)
    x2, b2 = S.post_norm_add(y.bfloat16(), (want.float(), xb), g, eps)
    assert x2.dtype == torch.float32 and torch.equal(b2, x2.bfloat16())
    assert close(S.row_norm((x, x), g, eps, index=torch.tensor([4, 1])), oracle.scalar_norm(x[[4, 1]].double(), g, eps))
    emb = torch.randn(9, 24)
    assert close(S.embed_residual(torch.tensor([3, 8], dtype=torch.int32), emb, 2.5)[0], emb[[3, 8]].double() * 2.5)


# ------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompt(name):
    cfg, t = cases.model(MODELS[name])
    x = ids(150)
    want = oracle.forward(reference(cfg, t), x)
    e = engine(cfg, t)
    s = e.open_sequence()
    assert close(e.feed([(s, x, range(150))]), want)


@pytest.mark.parametrize("name", ["mixed", "single"])
@pytest.mark.parametrize("start", [1, 60])
def test_token_by_token(name, start):
    """Decoding through the cache, over page borders and past every window, equals the whole prompt."""
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
    got = []
    for lo in range(0, len(x), portion):
        part = x[lo:lo + portion]
        got.append(e.feed([(s, part, range(len(part)))]))
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


def test_one_layer_sees_exactly_its_window():
    """A token is seen window - 1 places later and no further, in a prompt and in decoding."""
    W = 11
    cfg, t = cases.model([cases.layer(window=W, ff=0, v_mix=False)], seed=4)
    x = ids(40, 4)
    y = list(x)
    y[15] = (x[15] + 1) % 61
    e = engine(cfg, t)
    a, b = e.open_sequence(), e.open_sequence()
    out = e.feed([(a, x[:22], range(22)), (b, y[:22], range(22))])
    diff = [(out[i] - out[22 + i]).abs().max().item() for i in range(22)]
    for j in range(22, 40):
        out = e.feed([(a, [x[j]], [0]), (b, [y[j]], [0])])
        diff.append((out[0] - out[1]).abs().max().item())
    assert [i for i, d in enumerate(diff) if d > 1e-4] == list(range(15, 15 + W))


def test_value_mixing_takes_the_first_marked_layer():
    """Without the mixing, or with another source layer, the logits move."""
    cfg, t = cases.model(cases.MIXED, seed=5)
    x = ids(30, 5)
    base = oracle.forward(reference(cfg, t), x)
    zero = dict(t)
    for i in (2, 4):
        zero[f"l{i}.mix.vmix"] = torch.zeros((), dtype=torch.bfloat16)
    assert (oracle.forward(reference(cfg, zero), x) - base).abs().max() > 1e-2
    unused = dict(t)
    unused["l1.mix.vmix"] = torch.tensor(0.9, dtype=torch.bfloat16)     # the first marked layer's own number has no effect
    e = engine(cfg, unused)
    assert close(e.feed([(e.open_sequence(), x, range(30))]), base)


def test_pages_come_back_and_are_reused():
    """A pool smaller than the sequence: pages behind every window return while it runs, and freed pages serve another one."""
    cfg, t = cases.model([cases.layer(window=20, heads=4, kv=2), cases.layer(window=50, heads=4, kv=2)], seed=6)
    x, y = ids(300, 6), ids(120, 7)
    want, want_y = (oracle.forward(reference(cfg, t), z) for z in (x, y))
    e = engine(cfg, t, max_pages=4)
    s = e.open_sequence()
    got = [e.feed([(s, x[:100], [99])])]
    for j in range(100, 300):
        got.append(e.feed([(s, [x[j]], [0])]))
        assert e.kv.pages_in_use <= 2
    assert close(torch.cat(got), want[99:])
    e.close_sequence(s)
    assert e.kv.pages_in_use == 0
    s = e.open_sequence()
    got = [e.feed([(s, y[:70], range(70))])] + [e.feed([(s, [y[j]], [0])]) for j in range(70, 120)]
    assert close(torch.cat(got), want_y)
    with pytest.raises(RuntimeError):
        e.feed([(e.open_sequence(), ids(300), [])])                      # more than the pool holds at once


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
    spec = engine(cfg, t, spec_tokens=3)                                 # proposals verified as extra rows of a pass
    rep = (prompts[0] * 6)[:30]
    assert spec.generate(rep, GenerationConfig(max_new_tokens=12, **GREEDY)).token_ids == oracle.generate(ref, rep, 12)
    emb = e.embed(prompts[1])
    assert emb.shape == (48,) and abs(float(emb.norm()) - 1) < 1e-5


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


def test_configuration_and_registry(tmp_path):
    cfg, t = cases.model(cases.MIXED)
    assert "kifusun" in known_models() and resolve_architecture(cfg).config is KifusunConfig
    assert resolve_architecture({"model_type": "llama"}).name == "llama" and resolve_architecture({}).name == "llama"
    with pytest.raises(ValueError):
        resolve_architecture({"architecture": "unheard-of"})
    c = KifusunConfig.from_dict(cfg)
    assert KifusunConfig.from_dict(c.to_dict()) == c and c.to_dict() == cfg
    for edit in (lambda d: d["layers"][0].update(type="recurrent"), lambda d: d["layers"][0]["mlp"].update(kind="sparse"),
                 lambda d: d["layers"][0]["mixer"].update(heads=5, kv_heads=2)):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(ValueError):
            KifusunConfig.from_dict(bad)
    wrong = dict(t)
    wrong["l0.mix.talk"] = torch.zeros(3, 3)
    with pytest.raises(ValueError):
        cases.weights(cfg, wrong)
    back = cases.weights(cfg, t).state_dict()
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    w = KifusunWeights.random(c, seed=3)
    assert w.num_parameters() > 0 and all(math.isfinite(float(v.float().sum())) for v in w.state_dict().values())


def test_load_and_serve(tmp_path):
    from prometorch_b200.serve import PagedBackend
    cfg, t = cases.model(cases.EVEN, seed=10)
    save(tmp_path, cfg, t)
    e = LLMEngine(device="cpu", max_pages=8, max_active=2)
    assert e.load(str(tmp_path)) and e.model.architecture == "kifusun"
    p = ids(9, 3)
    want = oracle.generate(reference(cfg, t), p, 8)
    assert e.generate(p, GenerationConfig(max_new_tokens=8, **GREEDY)).token_ids == want
    b = PagedBackend(str(tmp_path), "m", "cpu", max_active=2, max_pages=8)
    out = []
    b.generate(p, {"num_predict": 8, "temperature": 0.0, "repeat_penalty": 1.0}, lambda tok: out.append(tok) or True)
    assert out == want and b.architecture == "kifusun"
    b.server.close()


def test_generate_command(tmp_path, capsys):
    from prometorch_b200 import generate
    cfg, t = cases.model(cases.EVEN, seed=11, vocab=300)
    save(tmp_path, cfg, t)
    assert generate.main([str(tmp_path), "hey", "--device", "cpu", "--greedy", "--max-tokens", "5"]) == 0
    assert "kifusun" in capsys.readouterr().out
    assert generate.main([str(tmp_path), "--info", "--tensors"]) == 0
    out = capsys.readouterr().out
    assert "l1.mix.talk" in out and "architecture = 'Kifusun'" in out


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
