"""Small random Budorax models for the tests: a ``config.json`` object and tensors whose faults show.  Queries and keys are large, so that
single scores stand out; decays lie between slow and fast; the experts' corrections are spaced, so that the choice of experts (which the
corrections make and the weights do not know) rests on no close call, whatever the compute type."""
import torch

from prometorch_b200.models.budorax import BudoraxConfig, BudoraxWeights


def moe(ff=24, experts=5, top=2, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def delta(heads=4, kv=2, dim=12, vdim=20, conv=4, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def attention(heads=4, kv=2, dim=12, vdim=20, scale=0.2, chunk=20, rot=8, base=1000.0, diff=0.3, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
                                           "rot": {"dims": rot, "base": base}, "diff": diff}, "mlp": mlp}


def latent(heads=3, dim=12, rot=8, vdim=20, q_rank=28, kv_rank=24, scale=0.2, base=5000.0, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"dims": rot, "base": base}}, "mlp": mlp}


def model(layers, seed=0, vocab=61, width=48, eps=1e-3, cap=20.0, loop=None, spaced=True):
    """(config, tensors): tensors in bf16, so that every compute type starts from the same numbers."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, at=0.0, by=1.0):
        return (at + by * torch.randn(s, generator=g)).bfloat16()

    def m(*s, gain=1.0):
        return r(*s, by=gain * s[-1] ** -0.5)
    t = {"embed": r(vocab, width)}

    def norm(name, alpha=0.7):
        t.update({name: r(width, at=1.0, by=0.2), name + ".b": r(width, by=0.2), name + ".alpha": r(at=alpha, by=0.1)})
    norm("final.norm", 0.4)
    for i, e in enumerate(layers):
        p, x = f"l{i}.", e["mixer"]
        q = p + "mix."
        H, D, Dv = x["heads"], x["dim"], x["vdim"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if e["type"] == "delta":
            qk, hv = x["kv_heads"] * D, H * Dv
            for n, c in (("q", qk), ("k", qk), ("v", hv)):
                t[q + n], t[q + n + ".conv"] = m(c, width), r(c, x["conv"], at=0.3, by=0.5)
            t.update({q + "b": m(H, width, gain=1.5), q + "a": m(H, width, gain=1.5), q + "A_log": r(H, by=0.5), q + "dt_bias": r(H, at=-2.5, by=1.5),
                      q + "norm": r(Dv, at=1.0, by=0.3), q + "g": m(hv, width, gain=1.5)})
        elif e["type"] == "attention":
            t.update({q + "q": m(2 * H * D, width, gain=1.7), q + "k": m(2 * x["kv_heads"] * D, width, gain=1.7), q + "v": m(x["kv_heads"] * Dv, width)})
            t.update({q + n: r(D, by=0.2) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            R, kr, qr = x["rot_dim"], x["kv_rank"], x["q_rank"]
            t.update({q + "dq": m(qr, width), q + "dq.norm": r(qr, at=1.5, by=0.3), q + "uq": m(H * (D + R), qr, gain=1.5), q + "dkv": m(kr + R, width, gain=1.5),
                      q + "dkv.norm": r(kr, at=1.5, by=0.3), q + "uk": m(H * D, kr, gain=1.5), q + "uv": m(H * Dv, kr), q + "g": m(H, width, gain=1.5)})
        t[q + "o"] = m(width, H * Dv)
        if e["mlp"]:
            ff, E = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"]
            norm(p + "norm2")
            norm(p + "norm2b")
            for k in range(E):
                t.update({f"{p}mlp.e{k}.gate": m(ff, width, gain=1.5), f"{p}mlp.e{k}.up": m(ff, width, gain=1.5), f"{p}mlp.e{k}.down": m(width, ff)})
            # scores lie in (0, 1): corrections a step of 1.1 apart decide the choice, smaller ones share in it
            step = torch.randperm(E, generator=g).float() * (1.1 if spaced else 0.15)
            t.update({p + "mlp.router": m(E, width, gain=1.5), p + "mlp.correction": (step - step.mean()).bfloat16()})
    cfg = {"architecture": "Budorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg, t


def weights(cfg, tensors, max_positions=2048) -> BudoraxWeights:
    c = BudoraxConfig.from_dict(cfg)
    c.max_position_embeddings = max_positions
    return BudoraxWeights.from_state_dict(c, tensors)


# every size differs from its neighbours: grouped heads, dim != vdim, partial rotation, no feed-forward, one tap, odd expert widths
MIXED = [attention(heads=6, kv=3, dim=12, vdim=20, chunk=37, rot=8, diff=0.4, mlp=moe(ff=20, experts=7, top=3, scale=0.8)),
         latent(heads=5, dim=20, rot=12, vdim=28, q_rank=20, kv_rank=36, mlp=moe(ff=33, experts=4, top=1, scale=2.5)),
         delta(heads=6, kv=3, dim=16, vdim=8, conv=5),
         attention(heads=3, kv=1, dim=10, vdim=36, chunk=70, rot=0, base=7.0, diff=0.2),
         delta(heads=2, kv=1, dim=40, vdim=24, conv=1, mlp=moe(ff=16, experts=3, top=3, scale=1.0)),
         latent(heads=1, dim=8, rot=2, vdim=8, q_rank=9, kv_rank=7, base=30.0)]
MIXED_LOOP = (1, 4, 2)
EVEN = [delta(heads=4, kv=4, dim=16, vdim=16, conv=4, mlp=moe(ff=32, experts=4, top=2)),
        attention(heads=4, kv=2, dim=16, vdim=32, chunk=24, rot=16, mlp=moe(ff=32, experts=4, top=2)),
        latent(heads=4, dim=16, rot=16, vdim=16, q_rank=32, kv_rank=32, mlp=moe(ff=32, experts=4, top=2))]
SINGLE = [attention(heads=1, kv=1, dim=8, vdim=8, chunk=5, rot=2, mlp=moe(ff=8, experts=1, top=1)), delta(heads=1, kv=1, dim=8, vdim=8, conv=2)]
