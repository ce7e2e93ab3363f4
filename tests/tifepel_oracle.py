"""Plain, slow Tifepel: one function per mechanism, written from the equations with a loop over tokens wherever a state or a mask is
involved.  Shares no code with the package; the tests compare the framework with it.

A model is a dict: ``config`` (the parsed config.json) and ``tensors`` (name -> tensor).  Everything is computed in the dtype
of :func:`cast` (float64 unless a test asks for something else)."""
import math

import torch


def cast(tensors, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in tensors.items()}


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------- into the model
def bigram_rows(ids, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token: the pair's hash, the last row for a token that has none before it."""
    return [buckets if i == 0 else (ids[i - 1] * mul_prev + ids[i] * mul_cur) % buckets for i in range(len(ids))]


def embed(t, c, ids):
    b = c["embedding"]["bigram"]
    rows = bigram_rows(ids, b["buckets"], b["mul_prev"], b["mul_cur"])
    return torch.stack([t["embed"][i] + t["bigram"][r] + t["pos"][p] for p, (i, r) in enumerate(zip(ids, rows))])


# ---------------------------------------------------------------- convolution over time
def causal_conv(x, w):
    """x [T, C], w [C, taps]: channel c of token i is the sum of w[c, taps - 1 - n] x[i - n, c], zeros before the first token."""
    T, C = x.shape
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    return torch.stack([sum(w[:, n] * full[i + n] for n in range(taps)) for i in range(T)])


# ---------------------------------------------------------------- attention
def bucket(n, rows, far):
    """Row of the bias table for a key n tokens back: one row per distance in the first half, logarithmic steps up to ``far`` in the other."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9))


def temperature(p, coef, every):
    return 1 + coef * math.log((p + 1) // every + 1)


def biased_row(q, i, k, v, k_pos, scale, rel, far):
    """One query of one head: q [dim] at position i over k [S, dim], v [S, vdim]; rel [rows]."""
    see = [n for n, j in enumerate(k_pos) if j <= i]
    bias = rel[[bucket(i - k_pos[n], len(rel), far) for n in see]]
    s = k[see] @ q * scale + bias
    e = torch.exp(s - s.max())
    return (e / e.sum()) @ v[see]


def biased_rows(q, k, v, scale, rel, far, q_pos=None, k_pos=None):
    """q [T, H, dim], k [S, G, dim], v [S, G, vdim], rel [rows, H] -> [T, H, vdim]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    q_pos = list(range(T)) if q_pos is None else list(q_pos)
    k_pos = list(range(k.shape[0])) if k_pos is None else list(k_pos)
    return torch.stack([torch.stack([biased_row(q[t, h], i, k[:, h // (H // G)], v[:, h // (H // G)], k_pos, scale, rel[:, h], far) for h in range(H)])
                        for t, i in enumerate(q_pos)])


def attention_mixer(h, t, p, m, eps):
    T, H, G, D, Dv, qt = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["q_temp"]
    q = rms((h @ t[p + "q"].t()).view(T, H, D), eps)
    q = torch.stack([r * temperature(i, qt["coef"], qt["every"]) for i, r in enumerate(q)])
    k = rms((h @ t[p + "k"].t()).view(T, G, D), eps)
    v = (h @ t[p + "v"].t()).view(T, G, Dv)
    return biased_rows(q, k, v, m["scale"], t[p + "rel"], m["bias_max"]).reshape(T, H * Dv) @ t[p + "o"].t()


# ---------------------------------------------------------------- state-space recurrence
def ssm_step(S, x, B, C, dt, A_log, D):
    """One token of one head: S [N, vdim], x [vdim], B / C [N], dt a number -> (S, y)."""
    S = torch.exp(-torch.exp(A_log) * dt) * S + dt * torch.outer(B, x)
    return S, S.t() @ C + D * x


def gated_norm(y, z, w, groups, eps):
    """The gate first, then every one of ``groups`` equal parts by its own root mean square."""
    g = y * silu(z)
    return rms(g.view(g.shape[0], groups, -1), eps).reshape(g.shape) * w


def mamba2_mixer(h, t, p, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = (h @ t[p + "in"].t()).split([inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, t[p + "conv"]) + t[p + "conv.b"])
    x, B, C = xbc.split([inner, G * N, G * N], -1)
    x, B, C = x.view(T, H, P), B.view(T, G, N), C.view(T, G, N)
    dt = softplus(dt + t[p + "dt_bias"])
    y = torch.zeros(T, H, P, dtype=h.dtype)
    for n in range(H):
        S, g = torch.zeros(N, P, dtype=h.dtype), n // (H // G)
        for i in range(T):
            S, y[i, n] = ssm_step(S, x[i, n], B[i, g], C[i, g], dt[i, n], t[p + "A_log"][n], t[p + "D"][n])
    return gated_norm(y.reshape(T, inner), z, t[p + "norm"], m["norm_groups"], eps) @ t[p + "o"].t()


# ---------------------------------------------------------------- mixture of experts
def route(z, correction, top):
    """Router logits z [experts + identity] -> (chosen outputs, their weights): the correction has a say in the choice and none in the weights."""
    e = torch.exp(z - z.max())
    s = e / e.sum()
    chosen = sorted(range(len(z)), key=lambda n: (-float(s[n] + correction[n]), n))[:top]
    return chosen, s[chosen]


def expert(h, gate, up, down):
    return (silu(h @ gate.t()) * (h @ up.t())) @ down.t()


def moe(h, t, p, m):
    r = m["router"]
    three = lambda name: [t[f"{p}{name}.{n}"] for n in ("gate", "up", "down")]
    out = expert(h, *three("shared")) if m.get("shared") else torch.zeros_like(h)
    for i in range(h.shape[0]):
        chosen, w = route(t[p + "router"] @ h[i], t[p + "correction"], r["top"])
        for e, f in zip(chosen, w):
            out[i] += f * (expert(h[i], *three(f"e{e}")) if e < r["experts"] else h[i])
    return out


# ---------------------------------------------------------------- the model
MIXERS = {"attention": attention_mixer, "mamba2": mamba2_mixer}


def run_order(c):
    n, loop = len(c["layers"]), c.get("loop") or {"start": 0, "stop": 0, "times": 1}
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def streams_step(x, t, p, n, inner):
    """One sublayer n (1 or 2) of the layer with prefix p: x is the list of streams, inner(h) what the sublayer computes."""
    mix, way_in, way_out = (t[f"{p}hc{n}.{k}"] for k in ("mix", "in", "out"))
    h, out = inner(sum(w * s for w, s in zip(way_in, x)))
    gate = sigmoid(h @ t[f"{p}rg{n}"].t() + t[f"{p}rg{n}.b"])
    y = out * gate
    return [sum(mix[s, d] * x[s] for s in range(len(x))) + way_out[d] * y for d in range(len(x))]


def forward(model, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) collects the sum of the streams after every layer run."""
    c, t = model["config"], model["tensors"]
    eps = c["norm"]["eps"]
    x = [embed(t, c, ids)] * c["streams"]
    for i in run_order(c):
        layer, p = c["layers"][i], f"l{i}."

        def sub(n, f):
            def inner(u):
                h = layer_norm(u, t[f"{p}norm{n}"], eps)
                return h, f(h + causal_conv(h, t[f"{p}canon{n}"]))
            return inner
        x = streams_step(x, t, p, 1, sub(1, lambda h: MIXERS[layer["type"]](h, t, p + "mix.", layer["mixer"], eps)))
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "moe"
            x = streams_step(x, t, p, 2, sub(2, lambda h: moe(h, t, p + "mlp.", layer["mlp"])))
        if layers_out is not None:
            layers_out.append(sum(x))
    return layer_norm(sum(x), t["final.norm"], eps) @ t["head"].t()


def generate(model, ids, n, stop=()):
    """Greedy ids by recomputing the whole sequence for every token."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(forward(model, ids)[-1].argmax()))
        ids.append(out[-1])
        if out[-1] in stop:
            break
    return out
