"""Small random Gelutar models for the tests: a ``config.json`` object and tensors whose faults show.  Query and key norm weights
are large, so that single scores stand out; sinks reach the size of the scores; decays lie between slow and fast."""
import torch

from prometorch_b200.models.gelutar import GelutarConfig, GelutarWeights


def parallel(heads=3, kv=3, dim=20, vdim=28, scale=0.11, window=9, keep=2, d_heads=2, d_kv=2, d_dim=12, d_vdim=20, conv=4, ff=40):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window, "keep_first": keep}},
                      "right": {"heads": d_heads, "kv_heads": d_kv, "dim": d_dim, "vdim": d_vdim, "conv": conv}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def lightning(heads=3, dim=12, vdim=20, decay=None, ff=40):
    decay = decay if decay is not None else [0.5 ** (1 / (1 + 3 * h)) for h in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(layers, seed=0, vocab=61, width=48, scale=1.5, eps=1e-4, logit_scale=0.7, rank=6, a_log=0.5):
    """(config, tensors): tensors in bf16, so that every compute type starts from the same numbers."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, at=0.0, by=1.0):
        return (at + by * torch.randn(s, generator=g)).bfloat16()

    def m(*s, gain=1.0):
        return r(*s, by=gain * s[-1] ** -0.5)
    t = {"embed": r(vocab, width, by=0.8), "head": m(vocab, width, gain=1.4), "final.norm": r(width, by=0.2)}
    for i, e in enumerate(layers):
        p, x = f"l{i}.", e["mixer"]
        t[p + "norm1"] = r(width, by=0.2)
        if e["type"] == "parallel":
            a, b = x["left"], x["right"]
            q, l = p + "mix.left.", p + "mix.right."
            t.update({q + "q": m(a["heads"] * a["dim"], width), q + "k": m(a["kv_heads"] * a["dim"], width), q + "v": m(a["kv_heads"] * a["vdim"], width),
                      q + "q.norm": r(a["heads"] * a["dim"], at=1.6, by=0.3), q + "k.norm": r(a["kv_heads"] * a["dim"], at=1.6, by=0.3),
                      q + "sink": r(a["heads"], at=1.0, by=1.5), q + "g": m(a["heads"], width, gain=1.5), q + "o": m(width, a["heads"] * a["vdim"]),
                      q + "out": r(width, at=1.0, by=0.3)})
            qd, kd, hv = b["kv_heads"] * b["dim"], b["heads"] * b["dim"], b["heads"] * b["vdim"]
            for n, c in (("q", qd), ("k", qd), ("v", hv)):
                t[l + n], t[l + n + ".conv"] = m(c, width), r(c, b["conv"], at=0.3, by=0.5)
            t.update({l + "b": m(b["heads"], width, gain=1.5), l + "A_log": r(b["heads"], by=a_log), l + "norm": r(b["vdim"], at=1.0, by=0.3),
                      l + "a1": m(rank, width), l + "a2": m(kd, rank), l + "dt_bias": r(kd, at=-2.5, by=1.5), l + "g1": m(rank + 1, width),
                      l + "g2": m(hv, rank + 1, gain=1.5), l + "o": m(width, hv), l + "out": r(width, at=1.0, by=0.3)})
        else:
            hk, hv = x["heads"] * x["dim"], x["heads"] * x["vdim"]
            l = p + "mix."
            t.update({l + "q": m(hk, width), l + "k": m(hk, width), l + "v": m(hv, width), l + "g": m(hv, width), l + "o": m(width, hv),
                      l + "norm": r(hv, at=1.0, by=0.3)})
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            t.update({p + "norm2": r(width, by=0.2), p + "mlp.up": m(ff, width), p + "mlp.down": m(width, ff)})
    cfg = {"architecture": "Gelutar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "layers": layers}
    return cfg, t


def weights(cfg, tensors, max_positions=4096) -> GelutarWeights:
    c = GelutarConfig.from_dict(cfg)
    c.max_position_embeddings = max_positions
    return GelutarWeights.from_state_dict(c, tensors)


# every size differs from its neighbours: grouped heads on both sides, dim != vdim, no feed-forward, one tap, nothing kept
MIXED = [lightning(heads=5, dim=8, vdim=12, ff=24),
         parallel(heads=4, kv=2, dim=12, vdim=20, window=70, keep=5, d_heads=6, d_kv=3, d_dim=16, d_vdim=8, conv=5, ff=0),
         parallel(heads=3, kv=1, dim=28, vdim=12, window=9, keep=0, d_heads=2, d_kv=1, d_dim=40, d_vdim=24, conv=2, ff=33),
         lightning(heads=2, dim=20, vdim=36, ff=0),
         parallel(heads=2, kv=2, dim=16, vdim=16, window=1, keep=66, d_heads=3, d_kv=3, d_dim=8, d_vdim=20, conv=1, ff=16)]
EVEN = [parallel(heads=8, kv=4, dim=32, vdim=32, window=33, keep=4, d_heads=4, d_kv=2, d_dim=16, d_vdim=16, ff=64),
        lightning(heads=4, dim=16, vdim=16, ff=64)]
SINGLE = [parallel(heads=1, kv=1, dim=8, vdim=8, window=5, keep=1, d_heads=1, d_kv=1, d_dim=8, d_vdim=8, conv=2, ff=8, scale=0.3), lightning(heads=1, dim=8, vdim=8, decay=[0.9], ff=8)]
