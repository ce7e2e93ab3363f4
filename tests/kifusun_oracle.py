"""Plain, slow Kifusun: one function per mechanism, written from the equations with loops over tokens and heads where that
keeps them readable.  Shares no code with the package; the tests compare the framework with it.

A model is a dict: ``config`` (the parsed config.json) and ``tensors`` (name -> tensor).  Everything is computed in the dtype
of :func:`cast` (float64 unless a test asks for something else)."""
import math

import torch


def cast(tensors, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in tensors.items()}


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, g, eps):
    """RMS norm whose weight is one number."""
    return rms(x, eps) * g


def head_norm(x, w, eps):
    """x [T, heads, dim], w [dim]: RMS norm of every head's vector with one weight for all heads."""
    return rms(x, eps) * w


def distance_bucket(n, rows, dmax):
    """Row of the bias table for a key ``n`` tokens back: exact for near keys, logarithmic up to ``dmax``."""
    half = rows // 2
    if n < half:
        return n
    # floor of ln(n / half) / ln(dmax / half) * (rows - half); a value within 1e-12 of an integer counts as that integer
    v = math.log(n / half) / math.log(dmax / half) * (rows - half)
    return min(rows - 1, half + math.floor(v + 1e-12))


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def visible(i, j, window):
    return 0 <= i - j < window


def mix_heads(w, talk):
    """w [H, ...], talk [H, H]: row h of the result is the talk[h]-weighted sum over all heads."""
    return torch.einsum("hg,g...->h...", talk, w)


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def attention_weights(q, k, i, positions, scale, cap, window, rel, dmax, pb):
    """Unmixed weights [H, len(positions)] of the query q [H, dim] at position i over the keys k [n, G, dim]."""
    H, G = q.shape[0], k.shape[1]
    out = torch.zeros(H, len(positions), dtype=q.dtype)
    for n, j in enumerate(positions):
        if not visible(i, j, window):
            continue
        b = distance_bucket(i - j, rel.shape[0], dmax)
        for h in range(H):
            s = soft_cap((q[h] * k[n, h // (H // G)]).sum() * scale, cap) + rel[b, h] + pb[h]
            out[h, n] = torch.sigmoid(s)
    return out


def attention_rows(q, k, v, scale, cap, window, rel, dmax, pb, talk, q_pos=None, k_pos=None):
    """q [T, H, dim] at q_pos against k [S, G, dim], v [S, G, vdim] at k_pos -> [T, H, vdim], one query at a time; the same as
    :func:`attention_weights` followed by :func:`mix_heads`, with the keys of one query handled together."""
    T, H, S, G = q.shape[0], q.shape[1], k.shape[0], k.shape[1]
    q_pos = list(range(T)) if q_pos is None else list(q_pos)
    k_pos = list(range(S)) if k_pos is None else list(k_pos)
    kv = [h // (H // G) for h in range(H)]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t, i in enumerate(q_pos):
        see = [n for n, j in enumerate(k_pos) if visible(i, j, window)]
        if not see:
            continue
        bucket = [distance_bucket(i - k_pos[n], rel.shape[0], dmax) for n in see]
        kk, vv = k[see][:, kv], v[see][:, kv]                                   # [n, H, dim], [n, H, vdim]
        s = soft_cap(torch.einsum("hd,nhd->hn", q[t], kk) * scale, cap) + rel[bucket].t() + pb[:, None]
        w = mix_heads(torch.sigmoid(s), talk)
        out[t] = torch.einsum("hn,nhd->hd", w, vv)
    return out


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(x, gate, up, down):
    return (gelu_tanh(x @ gate.t()) * (x @ up.t())) @ down.t()


def forward(model, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out`` (a list) collects the residual stream after every layer."""
    c, t = model["config"], model["tensors"]
    eps = c["norm"]["eps"]
    x = t["embed"][torch.tensor(ids)] * c["embedding"]["scale"]
    T = len(ids)
    v_first = None
    for i, layer in enumerate(c["layers"]):
        assert layer["type"] == "attention"
        p, m = f"l{i}.", layer["mixer"]
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = (x @ t[p + "mix.q"].t() + t[p + "mix.q.b"]).view(T, H, D)
        k = (x @ t[p + "mix.k"].t() + t[p + "mix.k.b"]).view(T, G, D)
        v = (x @ t[p + "mix.v"].t() + t[p + "mix.v.b"]).view(T, G, Dv)
        q, k = head_norm(q, t[p + "mix.q.norm"], eps), head_norm(k, t[p + "mix.k.norm"], eps)
        if m["v_mix"]:
            if v_first is None:
                v_first = v
            else:
                v = mix_values(v, v_first, t[p + "mix.vmix"])
        a = attention_rows(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], t[p + "mix.rel"], m["bias_max"],
                           t[p + "mix.pb"], t[p + "mix.talk"])
        x = x + scalar_norm(a.reshape(T, H * Dv) @ t[p + "mix.o"].t(), t[p + "norm1"], eps)
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            x = x + scalar_norm(feed_forward(x, t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"]), t[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return scalar_norm(x, t["final.norm"], eps) @ t["head"].t()


def generate(model, ids, n, stop=()):
    """Greedy ids by recomputing the whole sequence for every token."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(forward(model, ids)[-1].argmax()))
        ids.append(out[-1])
        if out[-1] in stop:
            break
    return out
