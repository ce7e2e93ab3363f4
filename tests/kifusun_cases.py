"""Small random Kifusun models for the tests: a ``config.json`` object and tensors whose faults show.  The keys' and queries' norm
weights are large, so single scores stand out, and the biases differ from head to head."""
import torch

from prometorch_b200.models.kifusun import KifusunConfig, KifusunWeights


def layer(heads=3, kv=3, dim=20, vdim=28, window=9, ff=40, v_mix=True, scale=0.3, cap=4.0, dmax=50):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "mask": {"size": window},
                      "bias_max": dmax, "v_mix": v_mix},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(layers, seed=0, vocab=61, width=48, scale=3.0, eps=1e-4, rows=10):
    """(config, tensors): tensors in bf16, so that every compute type starts from the same numbers."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, at=0.0, by=1.0):
        return (at + by * torch.randn(s, generator=g)).bfloat16()
    t = {"embed": r(vocab, width, by=0.5), "head": r(vocab, width, by=width ** -0.5), "final.norm": r(at=0.9, by=0.1)}
    for i, e in enumerate(layers):
        m, p = e["mixer"], f"l{i}."
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, n in (("q", H * D), ("k", G * D), ("v", G * Dv)):
            t[f"{p}mix.{name}"], t[f"{p}mix.{name}.b"] = r(n, width, by=width ** -0.5), r(n, by=0.3)
        t.update({p + "mix.q.norm": r(D, at=1.5, by=0.3), p + "mix.k.norm": r(D, at=1.5, by=0.3), p + "mix.rel": r(rows, H, by=1.0),
                  p + "mix.vmix": r(at=0.45, by=0.05), p + "mix.talk": r(H, H, at=0.0, by=0.5) + torch.eye(H).bfloat16(), p + "mix.pb": r(H, at=-1.0),
                  p + "mix.o": r(width, H * Dv, by=(H * Dv) ** -0.5), p + "norm1": r(at=1.1, by=0.1)})
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            t.update({p + "mlp.gate": r(ff, width, by=width ** -0.5), p + "mlp.up": r(ff, width, by=width ** -0.5),
                      p + "mlp.down": r(width, ff, by=ff ** -0.5), p + "norm2": r(at=0.8, by=0.1)})
    cfg = {"architecture": "Kifusun", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    return cfg, t


def weights(cfg, tensors, max_positions=4096) -> KifusunWeights:
    c = KifusunConfig.from_dict(cfg)
    c.max_position_embeddings = max_positions
    return KifusunWeights.from_state_dict(c, tensors)


MIXED = [layer(heads=4, kv=1, dim=24, vdim=16, window=70, ff=40, v_mix=False, dmax=40, scale=0.25, cap=6.0),
         layer(heads=3, kv=3, dim=20, vdim=28, window=9, ff=0, v_mix=True),
         layer(heads=6, kv=3, dim=16, vdim=28, window=130, ff=33, v_mix=True, dmax=100, scale=0.2),
         layer(heads=2, kv=2, dim=40, vdim=12, window=1, ff=16, v_mix=False),
         layer(heads=6, kv=3, dim=16, vdim=28, window=64, ff=24, v_mix=True, cap=2.5)]
EVEN = [layer(heads=8, kv=4, dim=32, vdim=32, window=33, ff=64, v_mix=True, dmax=32, scale=0.2) for _ in range(2)]
SINGLE = [layer(heads=1, kv=1, dim=8, vdim=8, window=5, ff=8, v_mix=True, scale=1.0, cap=30.0)]
