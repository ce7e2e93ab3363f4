"""Small random Tifepel models for the tests: a ``config.json`` object and tensors whose faults show.  The biases by distance are large, so that
a bucket that is one off moves the logits; streams mix unevenly; decays lie between slow and fast; the router's corrections are spaced, so
that the choice of outputs (which the corrections make and the weights do not know) rests on no close call, whatever the compute type."""
import torch

from prometorch_b200.models.tifepel import TifepelConfig, TifepelWeights


def moe(ff=24, experts=5, top=2, identity=2, shared=20):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}, "shared": {"ff": shared} if shared else None}


def mamba(heads=6, groups=3, state=12, vdim=8, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def attention(heads=4, kv=2, dim=12, vdim=20, scale=0.4, bias_max=50, coef=0.3, every=16, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
                                           "q_temp": {"coef": coef, "every": every}}, "mlp": mlp}


def model(layers, seed=0, vocab=61, width=48, eps=1e-3, streams=3, taps=3, buckets=53, max_positions=1024, loop=None, rel_rows=10, muls=(31, 11), spaced=True):
    """(config, tensors): tensors in bf16, so that every compute type starts from the same numbers."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, at=0.0, by=1.0):
        return (at + by * torch.randn(s, generator=g)).bfloat16()

    def m(*s, gain=1.0):
        return r(*s, by=gain * s[-1] ** -0.5)
    t = {"embed": r(vocab, width), "bigram": r(buckets + 1, width), "pos": r(max_positions, width, by=0.7), "final.norm": r(width, at=1.0, by=0.2), "head": m(vocab, width)}
    for i, e in enumerate(layers):
        p, x = f"l{i}.", e["mixer"]
        q = p + "mix."
        H, Dv = x["heads"], x["vdim"]
        for n in ("1", "2") if e["mlp"] else ("1",):
            t.update({p + "norm" + n: r(width, at=1.0, by=0.2), p + "canon" + n: r(width, taps, by=0.3), p + "rg" + n: m(width, width, gain=1.5), f"{p}rg{n}.b": r(width, by=0.5),
                      f"{p}hc{n}.in": r(streams, at=1.0 / streams, by=0.15), f"{p}hc{n}.out": r(streams, at=0.7, by=0.3),
                      f"{p}hc{n}.mix": (0.9 * torch.eye(streams) + 0.15 * torch.randn(streams, streams, generator=g)).bfloat16()})
        if e["type"] == "mamba2":
            inner, GN = H * Dv, x["groups"] * x["state"]
            t.update({q + "in": m(2 * inner + 2 * GN + H, width), q + "conv": r(inner + 2 * GN, x["conv"], at=0.2, by=0.5), q + "conv.b": r(inner + 2 * GN, by=0.3),
                      q + "dt_bias": r(H, at=-2.0, by=1.0), q + "A_log": r(H, by=0.7), q + "D": r(H, at=1.0, by=0.5), q + "norm": r(inner, at=1.0, by=0.3)})
        else:
            G, D = x["kv_heads"], x["dim"]
            t.update({q + "q": m(H * D, width), q + "k": m(G * D, width), q + "v": m(G * Dv, width), q + "rel": r(rel_rows, H, by=1.5)})
        t[q + "o"] = m(width, H * Dv)
        if e["mlp"]:
            E, rt = e["mlp"]["router"]["experts"], e["mlp"]["router"]
            for name, ff in [(f"e{k}", e["mlp"]["expert"]["ff"]) for k in range(E)] + ([("shared", e["mlp"]["shared"]["ff"])] if e["mlp"]["shared"] else []):
                t.update({f"{p}mlp.{name}.gate": m(ff, width), f"{p}mlp.{name}.up": m(ff, width), f"{p}mlp.{name}.down": m(width, ff)})
            # scores lie in (0, 1): corrections a step of 1.1 apart decide the choice, smaller ones share in it
            O = E + rt["identity"]
            step = torch.randperm(O, generator=g).float() * (1.1 if spaced else 0.1)
            t.update({p + "mlp.router": m(O, width, gain=1.5), p + "mlp.correction": (step - step.mean()).bfloat16()})
    cfg = {"architecture": "Tifepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions, "streams": streams, "canon": {"taps": taps},
           "embedding": {"bigram": {"buckets": buckets, "mul_prev": muls[0], "mul_cur": muls[1]}}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg, t


def weights(cfg, tensors) -> TifepelWeights:
    return TifepelWeights.from_state_dict(TifepelConfig.from_dict(cfg), tensors)


# every size differs from its neighbours: grouped heads, dim != vdim, no feed-forward, no shared expert, no identities, one tap, odd widths
MIXED = [mamba(heads=6, groups=3, state=12, vdim=10, conv=5, norm_groups=4, mlp=moe(ff=20, experts=7, top=3, identity=3, shared=33)),
         attention(heads=6, kv=3, dim=12, vdim=20, scale=0.3, bias_max=37, coef=0.4, every=10, mlp=moe(ff=33, experts=4, top=1, identity=0, shared=8)),
         mamba(heads=2, groups=1, state=40, vdim=24, conv=1, norm_groups=1),
         attention(heads=3, kv=1, dim=20, vdim=9, scale=0.25, bias_max=200, coef=0.0, every=7, mlp=moe(ff=16, experts=3, top=4, identity=1, shared=0)),
         mamba(heads=4, groups=4, state=7, vdim=5, conv=2, norm_groups=5, mlp=moe(ff=9, experts=1, top=2, identity=6, shared=12))]
MIXED_LOOP = (1, 4, 2)
EVEN = [attention(heads=4, kv=2, dim=16, vdim=32, bias_max=64, mlp=moe(ff=32, experts=4, top=2, identity=4, shared=32)),
        mamba(heads=4, groups=2, state=16, vdim=16, conv=4, norm_groups=1, mlp=moe(ff=32, experts=4, top=2, identity=0, shared=64)),
        mamba(heads=2, groups=2, state=32, vdim=16, conv=3, norm_groups=2, mlp=moe(ff=16, experts=8, top=3, identity=2, shared=0))]
SINGLE = [mamba(heads=1, groups=1, state=8, vdim=8, conv=2, norm_groups=1, mlp=moe(ff=8, experts=1, top=1, identity=0, shared=8)),
          attention(heads=1, kv=1, dim=8, vdim=8, bias_max=9, coef=1.0, every=1)]
