"""Plain, slow Budorax: one function per mechanism, written from the equations with a loop over tokens wherever a state or a mask is
involved.  Shares no code with the package; the tests compare the framework with it.

A model is a dict: ``config`` (the parsed config.json) and ``tensors`` (name -> tensor).  Everything is computed in the dtype
of :func:`cast` (float64 unless a test asks for something else)."""
import math

import torch


def cast(tensors, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in tensors.items()}


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def plain_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def tanh_norm(x, alpha, w, b):
    """Elementwise in place of a norm: no statistics of the row."""
    return torch.tanh(alpha * x) * w + b


def named_norm(x, t, name):
    return tanh_norm(x, t[name + ".alpha"], t[name], t[name + ".b"])


# ---------------------------------------------------------------- rotation
def rotate(x, pos, dims, base):
    """x [.., size] at position pos: neighbours (2i, 2i + 1) of the first ``dims`` entries turn by pos * base^(-2i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
    return y


def rotate_rows(x, dims, base, pos=None):
    return torch.stack([rotate(r, p, dims, base) for r, p in zip(x, range(len(x)) if pos is None else pos)])


# ---------------------------------------------------------------- attention
def same_chunk(i, j, size):
    """Whether the query at position i sees the key at position j when attention stays inside chunks of ``size`` positions."""
    return j <= i and i // size == j // size


def softmax_row(q, k, v, scale):
    """q [dim], k [S, dim], v [S, vdim] -> [vdim]."""
    s = k @ q * scale
    e = torch.exp(s - s.max())
    return (e / e.sum()) @ v


def two_maps_row(q, i, k, v, k_pos, scale, size, lam, diff, eps):
    """One query of one head: q [2, dim] at position i over k [S, 2, dim] and v [S, vdim].  Both maps weigh the same values; the
    second one's output is taken off, the rest normed."""
    see = [n for n, j in enumerate(k_pos) if same_chunk(i, j, size)]
    a = [softmax_row(q[m], k[see, m], v[see], scale) for m in range(2)]
    return rms(a[0] - lam * a[1], eps) * (1 - diff)


def two_maps_rows(q, k, v, scale, size, lam, diff, eps, q_pos=None, k_pos=None):
    """q [T, H, 2, dim], k [S, G, 2, dim], v [S, G, vdim] -> [T, H, vdim]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    q_pos = list(range(T)) if q_pos is None else list(q_pos)
    k_pos = list(range(k.shape[0])) if k_pos is None else list(k_pos)
    return torch.stack([torch.stack([two_maps_row(q[t, h], i, k[:, h // (H // G)], v[:, h // (H // G)], k_pos, scale, size, lam, diff, eps)
                                     for h in range(H)]) for t, i in enumerate(q_pos)])


def mix_factor(lq1, lk1, lq2, lk2, diff):
    return float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff)


def attention_mixer(h, t, p, m, eps):
    T, H, G, D, Dv, r = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q, k = (rotate_rows((h @ t[p + n].t()).view(T, heads, 2, D), r["dims"], r["base"]) for n, heads in (("q", H), ("k", G)))
    v = (h @ t[p + "v"].t()).view(T, G, Dv)
    lam = mix_factor(t[p + "lq1"], t[p + "lk1"], t[p + "lq2"], t[p + "lk2"], m["diff"])
    o = two_maps_rows(q, k, v, m["scale"], m["mask"]["size"], lam, m["diff"], eps)
    return o.reshape(T, H * Dv) @ t[p + "o"].t()


def latent_rows(q, k, v, scale, q_pos=None, k_pos=None):
    """q [T, H, size], k [S, H, size], v [S, H, vdim] -> [T, H, vdim]: every key up to the query's position."""
    T = q.shape[0]
    q_pos = list(range(T)) if q_pos is None else list(q_pos)
    k_pos = list(range(k.shape[0])) if k_pos is None else list(k_pos)
    out = []
    for t, i in enumerate(q_pos):
        see = [n for n, j in enumerate(k_pos) if j <= i]
        out.append(torch.stack([softmax_row(q[t, h], k[see, h], v[see, h], scale) for h in range(q.shape[1])]))
    return torch.stack(out)


def latent_mixer(h, t, p, m, eps):
    """Queries through a latent of their own; keys and values from one latent per token plus a rotated key part that all heads share."""
    T, H, D, R, Dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (plain_norm(h @ t[p + "dq"].t(), t[p + "dq.norm"], eps) @ t[p + "uq"].t()).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate_rows(q[..., D:], R, base)], -1)
    down = h @ t[p + "dkv"].t()
    c = plain_norm(down[:, :rank], t[p + "dkv.norm"], eps)
    shared = rotate_rows(down[:, rank:], R, base)
    k = torch.cat([(c @ t[p + "uk"].t()).view(T, H, D), shared[:, None, :].expand(T, H, R)], -1)
    v = (c @ t[p + "uv"].t()).view(T, H, Dv)
    o = latent_rows(q, k, v, m["scale"]) * sigmoid(h @ t[p + "g"].t())[:, :, None]
    return o.reshape(T, H * Dv) @ t[p + "o"].t()


# ---------------------------------------------------------------- gated delta rule
def causal_conv(x, w):
    """x [T, C], w [C, taps]: channel c of token i is the sum of w[c, taps - 1 - n] x[i - n, c], zeros before the first token."""
    T, C = x.shape
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    return torch.stack([sum(w[:, n] * full[i + n] for n in range(taps)) for i in range(T)])


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_step(S, q, k, v, g, beta):
    """One token of one head: S [dim, vdim], q / k [dim], v [vdim], one decay g -> (S, o).  The state decays, the part of v that it
    does not already return for k is written, and q reads it afterwards."""
    S = g * S
    u = beta * (v - S.t() @ k)
    S = S + torch.outer(k, u)
    return S, S.t() @ q


def head_decay(a, A_log, dt_bias):
    """a [.., H]: one decay per head."""
    return torch.exp(-torch.exp(A_log) * softplus(a + dt_bias))


def delta_mixer(h, t, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ t[p + n].t(), t[p + n + ".conv"])) for n in "qkv")
    q, k, v = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D)), v.view(T, H, Dv)
    beta = sigmoid(h @ t[p + "b"].t())
    g = head_decay(h @ t[p + "a"].t(), t[p + "A_log"], t[p + "dt_bias"])
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for n in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        c = n // (H // G)
        for i in range(T):
            S, out[i, n] = delta_step(S, q[i, c], k[i, c], v[i, n], g[i, n], beta[i, n])
    gate = silu(h @ t[p + "g"].t()).view(T, H, Dv)
    return (plain_norm(out, t[p + "norm"], eps) * gate).reshape(T, H * Dv) @ t[p + "o"].t()


# ---------------------------------------------------------------- mixture of experts
def route(z, correction, top, scale):
    """Router logits z [experts] -> (chosen experts, their weights): the correction has a say in the choice and none in the weights."""
    s = sigmoid(z)
    chosen = sorted(range(len(z)), key=lambda e: (-float(s[e] + correction[e]), e))[:top]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20) * scale


def expert(h, gate, up, down):
    return (silu(h @ gate.t()) * (h @ up.t())) @ down.t()


def experts(h, t, p, m):
    r, out = m["router"], torch.zeros_like(h)
    for i in range(h.shape[0]):
        chosen, w = route(t[p + "router"] @ h[i], t[p + "correction"], r["top"], r["scale"])
        for e, f in zip(chosen, w):
            out[i] += f * expert(h[i], *(t[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")))
    return out


# ---------------------------------------------------------------- the model
MIXERS = {"delta": delta_mixer, "attention": attention_mixer, "latent_attention": latent_mixer}


def run_order(c):
    """(layer, whether the embedding output is added ahead of it) of every layer run."""
    n, loop = len(c["layers"]), c.get("loop") or {"start": 0, "stop": 0, "times": 1}
    body = list(range(loop["start"], loop["stop"]))
    order = [(i, False) for i in range(loop["start"])]
    for k in range(loop["times"]):
        order += [(i, k > 0 and i == loop["start"]) for i in body]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(model, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) collects the residual stream after every layer run."""
    c, t = model["config"], model["tensors"]
    eps = c["norm"]["eps"]
    first = t["embed"][torch.tensor(ids)]
    x = first
    for i, again in run_order(c):
        layer, p = c["layers"][i], f"l{i}."
        if again:
            x = x + first
        x = x + named_norm(MIXERS[layer["type"]](named_norm(x, t, p + "norm1"), t, p + "mix.", layer["mixer"], eps), t, p + "norm1b")
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "moe"
            x = x + named_norm(experts(named_norm(x, t, p + "norm2"), t, p + "mlp.", layer["mlp"]), t, p + "norm2b")
        if layers_out is not None:
            layers_out.append(x)
    cap = c["logit_softcap"]
    return torch.tanh(named_norm(x, t, "final.norm") @ t["embed"].t() / cap) * cap


def generate(model, ids, n, stop=()):
    """Greedy ids by recomputing the whole sequence for every token."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(forward(model, ids)[-1].argmax()))
        ids.append(out[-1])
        if out[-1] in stop:
            break
    return out
