"""Plain, slow Gelutar: one function per mechanism, written from the equations with a loop over tokens wherever a state or a
window is involved.  Shares no code with the package; the tests compare the framework with it.

A model is a dict: ``config`` (the parsed config.json) and ``tensors`` (name -> tensor).  Everything is computed in the dtype
of :func:`cast` (float64 unless a test asks for something else)."""
import torch


def cast(tensors, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in tensors.items()}


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def plus_one_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def plain_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------- softmax attention: window, kept tokens, sink, gate
def visible(i, j, size, keep):
    """Whether the query at position i sees the key at position j."""
    return j <= i and (i - j < size or j < keep)


def attention_row(q, i, k, v, k_pos, scale, size, keep, sink):
    """q [H, dim] at position i over k [S, G, dim], v [S, G, vdim] at positions k_pos -> [H, vdim].  The sink of a head adds
    exp(sink) to the sum of its weights and nothing to its output."""
    H, G = q.shape[0], k.shape[1]
    see = [n for n, j in enumerate(k_pos) if visible(i, j, size, keep)]
    out = torch.zeros(H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = k[see, g] @ q[h] * scale
        top = torch.maximum(s.max(), sink[h]) if len(see) else sink[h]
        e = torch.exp(s - top)
        out[h] = (e / (e.sum() + torch.exp(sink[h] - top))) @ v[see, g]
    return out


def attention_rows(q, k, v, scale, size, keep, sink, q_pos=None, k_pos=None):
    T, S = q.shape[0], k.shape[0]
    q_pos = list(range(T)) if q_pos is None else list(q_pos)
    k_pos = list(range(S)) if k_pos is None else list(k_pos)
    return torch.stack([attention_row(q[t], i, k, v, k_pos, scale, size, keep, sink) for t, i in enumerate(q_pos)])


def window_mixer(h, t, p, m, eps):
    """h [T, width] -> [T, width]; tensors under the prefix p."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = plain_norm(h @ t[p + "q"].t(), t[p + "q.norm"], eps).view(T, H, D)          # over all heads together
    k = plain_norm(h @ t[p + "k"].t(), t[p + "k.norm"], eps).view(T, G, D)
    v = (h @ t[p + "v"].t()).view(T, G, Dv)
    a = attention_rows(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"], t[p + "sink"])
    a = a * sigmoid(h @ t[p + "g"].t())[:, :, None]
    return a.reshape(T, H * Dv) @ t[p + "o"].t()


# ---------------------------------------------------------------- gated delta rule
def causal_conv(x, w, before=None):
    """x [T, C], w [C, taps]: channel c of token i is the sum of w[c, taps - 1 - n] x[i - n, c]; ``before`` [taps - 1, C] stands
    in front of the first token (zeros by default)."""
    T, C = x.shape
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, C, dtype=x.dtype)
    full = torch.cat([before, x])
    return torch.stack([sum(w[:, n] * full[i + n] for n in range(taps)) for i in range(T)])


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_step(S, q, k, v, g, beta):
    """One token of one head: S [dim, vdim], q / k / g [dim], v [vdim] -> (S, o).  The state decays, the part of v that it does
    not already return for k is written, and q reads it afterwards."""
    S = g[:, None] * S
    u = beta * (v - S.t() @ k)
    S = S + torch.outer(k, u)
    return S, S.t() @ q


def delta_decay(a, A_log, dt_bias):
    """a [.., H, dim]: the decay of every head and key channel."""
    return torch.exp(-torch.exp(A_log)[:, None] * softplus(a + dt_bias))


def delta_mixer(h, t, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ t[p + n].t(), t[p + n + ".conv"])) for n in "qkv")
    q, k, v = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D)), v.view(T, H, Dv)
    beta = sigmoid(h @ t[p + "b"].t())
    g = delta_decay((h @ t[p + "a1"].t() @ t[p + "a2"].t()).view(T, H, D), t[p + "A_log"], t[p + "dt_bias"].view(H, D))
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for n in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        c = n // (H // G)
        for i in range(T):
            S, out[i, n] = delta_step(S, q[i, c], k[i, c], v[i, n], g[i, n], beta[i, n])
    gate = sigmoid(h @ t[p + "g1"].t() @ t[p + "g2"].t()).view(T, H, Dv)
    return (plain_norm(out, t[p + "norm"], eps) * gate).reshape(T, H * Dv) @ t[p + "o"].t()


def parallel_mixer(h, t, p, m, eps):
    """Both mixers on the same input; half the sum of their normalised outputs."""
    left = plain_norm(window_mixer(h, t, p + "left.", m["left"], eps), t[p + "left.out"], eps)
    right = plain_norm(delta_mixer(h, t, p + "right.", m["right"], eps), t[p + "right.out"], eps)
    return (left + right) / 2


# ---------------------------------------------------------------- linear attention with a fixed decay per head
def lightning_step(S, q, k, v, decay):
    S = decay * S + torch.outer(k, v)
    return S, S.t() @ q


def lightning_mixer(h, t, p, m, eps):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ t[p + n].t()).view(T, H, d) for n, d in (("q", D), ("k", D), ("v", Dv)))
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for n in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        for i in range(T):
            S, out[i, n] = lightning_step(S, q[i, n], k[i, n], v[i, n], m["decay"][n])
    y = plain_norm(out.reshape(T, H * Dv), t[p + "norm"], eps) * sigmoid(h @ t[p + "g"].t())
    return y @ t[p + "o"].t()


# ---------------------------------------------------------------- the model
def feed_forward(x, up, down):
    return torch.relu(x @ up.t()) ** 2 @ down.t()


MIXERS = {"parallel": parallel_mixer, "lightning": lightning_mixer}


def forward(model, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) collects the residual stream after every layer."""
    c, t = model["config"], model["tensors"]
    eps = c["norm"]["eps"]
    x = t["embed"][torch.tensor(ids)] * c["embedding"]["scale"]
    for i, layer in enumerate(c["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](plus_one_norm(x, t[p + "norm1"], eps), t, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            x = x + feed_forward(plus_one_norm(x, t[p + "norm2"], eps), t[p + "mlp.up"], t[p + "mlp.down"])
        if layers_out is not None:
            layers_out.append(x)
    return plus_one_norm(x, t["final.norm"], eps) @ t["head"].t() * c["logit_scale"]


def generate(model, ids, n, stop=()):
    """Greedy ids by recomputing the whole sequence for every token."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(forward(model, ids)[-1].argmax()))
        ids.append(out[-1])
        if out[-1] in stop:
            break
    return out
