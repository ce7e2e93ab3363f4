"""Gelutar for the batching engine: configuration, weights and the two passes.

A pre-norm decoder with an fp32 residual stream and one-plus norm weights, whose layers each bring their own mixer and sizes:

* ``parallel``: window attention (``ops/window_attention.py``: norm over the whole q and k projections, kept first tokens, a sink,
  a gate per head) and the gated delta rule (``ops/recurrence.py``: short convolutions, unit q and k, a decay per head and key
  channel, gated output norm) on the same input; half the sum of their normalised outputs joins the stream;
* ``lightning``: linear attention with a fixed decay per head, SiLU on q, k and v, a gated norm over all heads.

The feed-forward is ``down relu(up x)^2``; a layer may have none.  All projections of a mixer's input are one matrix product.

A model directory holds ``config.json`` (``"architecture": "Gelutar"``) and ``model.safetensors`` with the names of
:meth:`GelutarWeights.state_dict`."""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops import recurrence as R
from ..ops import residual as S
from ..ops import window_attention as A
from .paged import PagedModel, PromptBatch, RowPack, register_model


@dataclass
class WindowHalf:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int


@dataclass
class DeltaHalf:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                          # taps


@dataclass
class ParallelMixer:
    left: WindowHalf
    right: DeltaHalf


@dataclass
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: List[float]


@dataclass
class GelutarLayer:
    mixer: Union[ParallelMixer, LightningMixer]
    ff: int = 0                        # feed-forward width; 0: the layer has none

    def __post_init__(self):
        m = self.mixer
        for half in ((m.left, m.right) if isinstance(m, ParallelMixer) else (m,)):
            kv = getattr(half, "kv_heads", half.heads)
            if half.heads < 1 or kv < 1 or half.heads % kv:
                raise ValueError(f"{half.heads} heads over {kv} key/value heads")
            if min(half.dim, half.vdim) < 1:
                raise ValueError(f"head sizes {half.dim} / {half.vdim} must be positive")
        if isinstance(m, ParallelMixer):
            if m.left.window < 1 or m.left.keep_first < 0 or m.right.conv < 1:
                raise ValueError(f"window {m.left.window}, kept tokens {m.left.keep_first}, taps {m.right.conv}")
        elif len(m.decay) != m.heads:
            raise ValueError(f"{len(m.decay)} decays for {m.heads} heads")


@dataclass
class GelutarConfig:
    vocab_size: int
    hidden_size: int
    embed_scale: float
    eps: float
    logit_scale: float = 1.0
    layers: List[GelutarLayer] = field(default_factory=list)
    max_position_embeddings: int = 131072      # nothing in the design bounds a position; this sizes the page table
    bos_token_id: Optional[int] = None
    eos_token_id: int = -1

    @classmethod
    def from_dict(cls, d: dict) -> "GelutarConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, ff = e["mixer"], e.get("mlp")
            if ff is not None and ff["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {ff['kind']!r} is not part of Gelutar")
            if e["type"] == "parallel":
                a, b = m["left"], m["right"]
                mixer = ParallelMixer(WindowHalf(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                                                 int(a["mask"]["size"]), int(a["mask"]["keep_first"])),
                                      DeltaHalf(int(b["heads"]), int(b["kv_heads"]), int(b["dim"]), int(b["vdim"]), int(b["conv"])))
            elif e["type"] == "lightning":
                mixer = LightningMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), [float(x) for x in m["decay"]])
            else:
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of Gelutar")
            layers.append(GelutarLayer(mixer, int(ff["ff"]) if ff is not None else 0))
        return cls(int(d["vocab"]), int(d["width"]), float(d["embedding"]["scale"]), float(d["norm"]["eps"]), float(d["logit_scale"]), layers)

    @classmethod
    def from_json(cls, path: str) -> "GelutarConfig":
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for e in self.layers:
            m = e.mixer
            if isinstance(m, ParallelMixer):
                a, b = m.left, m.right
                mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                                  "mask": {"size": a.window, "keep_first": a.keep_first}},
                         "right": {"heads": b.heads, "kv_heads": b.kv_heads, "dim": b.dim, "vdim": b.vdim, "conv": b.conv}}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            layers.append({"type": "parallel" if isinstance(m, ParallelMixer) else "lightning", "mixer": mixer,
                           "mlp": {"kind": "dense", "ff": e.ff} if e.ff else None})
        return {"architecture": "Gelutar", "vocab": self.vocab_size, "width": self.hidden_size, "embedding": {"scale": self.embed_scale},
                "norm": {"eps": self.eps}, "logit_scale": self.logit_scale, "layers": layers}


MERGE_GATES = 128                      # rows up to which the two low-rank gates are one product of their own
_LEFT = ("left.q", "left.k", "left.v")
_CONV = ("right.q", "right.k", "right.v")


def _shapes(m, W: int, ff: int, rank_a: int, rank_g: int) -> Dict[str, Tuple[int, ...]]:
    """Tensor shapes of one layer (names without the layer's prefix)."""
    if isinstance(m, ParallelMixer):
        a, b = m.left, m.right
        qd, kd, hv = b.kv_heads * b.dim, b.heads * b.dim, b.heads * b.vdim
        mix = {"left.q": (a.heads * a.dim, W), "left.k": (a.kv_heads * a.dim, W), "left.v": (a.kv_heads * a.vdim, W), "left.q.norm": (a.heads * a.dim,),
               "left.k.norm": (a.kv_heads * a.dim,), "left.sink": (a.heads,), "left.g": (a.heads, W), "left.o": (W, a.heads * a.vdim),
               "right.q": (qd, W), "right.q.conv": (qd, b.conv), "right.k": (qd, W), "right.k.conv": (qd, b.conv), "right.v": (hv, W),
               "right.v.conv": (hv, b.conv), "right.b": (b.heads, W), "right.A_log": (b.heads,), "right.norm": (b.vdim,), "right.a1": (rank_a, W),
               "right.a2": (kd, rank_a), "right.dt_bias": (kd,), "right.g1": (rank_g, W), "right.g2": (hv, rank_g), "right.o": (W, hv),
               "left.out": (W,), "right.out": (W,)}
    else:
        hk, hv = m.heads * m.dim, m.heads * m.vdim
        mix = {"q": (hk, W), "k": (hk, W), "v": (hv, W), "g": (hv, W), "o": (W, hv), "norm": (hv,)}
    t = {"norm1": (W,), **{"mix." + k: v for k, v in mix.items()}}
    if ff:
        t.update({"norm2": (W,), "mlp.up": (ff, W), "mlp.down": (W, ff)})
    return t


class GelutarWeights:
    """Weights by the names of the checkpoint, layer by layer (prefix dropped); :class:`PagedGelutar` packs what its passes read."""

    def __init__(self, cfg: GelutarConfig):
        self.cfg = cfg
        self.embed: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.final_norm: Optional[torch.Tensor] = None
        self.layers: List[Dict[str, torch.Tensor]] = []

    @classmethod
    def from_state_dict(cls, cfg: GelutarConfig, sd: Dict[str, torch.Tensor]) -> "GelutarWeights":
        w, V, W = cls(cfg), cfg.vocab_size, cfg.hidden_size

        def take(name, shape):
            if tuple(sd[name].shape) != shape:
                raise ValueError(f"{name} has shape {tuple(sd[name].shape)}, the configuration asks for {shape}")
            return sd[name]
        w.embed, w.head, w.final_norm = take("embed", (V, W)), take("head", (V, W)), take("final.norm", (W,))
        for i, e in enumerate(cfg.layers):
            p = f"l{i}."
            ranks = [sd[p + f"mix.right.{n}"].shape[0] for n in ("a1", "g1")] if isinstance(e.mixer, ParallelMixer) else [0, 0]
            w.layers.append({k: take(p + k, s) for k, s in _shapes(e.mixer, W, e.ff, *ranks).items()})
        return w

    def state_dict(self) -> Dict[str, torch.Tensor]:
        sd = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        sd.update({f"l{i}.{k}": t for i, L in enumerate(self.layers) for k, t in L.items()})
        return sd

    @classmethod
    def random(cls, cfg: GelutarConfig, seed: int = 0, dtype=torch.float32, device="cpu", rank: int = 64) -> "GelutarWeights":
        """Random weights of the right scales (benchmarks and tests), drawn on ``device``; ``rank``: of the two low-rank gates."""
        g = torch.Generator(device=device).manual_seed(seed)

        def r(*s, scale=1.0, at=0.0):
            return (at + torch.randn(*s, generator=g, device=device) * scale).to(dtype)
        W, w = cfg.hidden_size, cls(cfg)
        w.embed, w.head = r(cfg.vocab_size, W, scale=1.0 / cfg.embed_scale), r(cfg.vocab_size, W, scale=W ** -0.5)
        w.final_norm = r(W, scale=0.1)
        plain = ("q.norm", "k.norm", "mix.norm", "right.norm", ".out")               # weights around one; the others lie around zero
        for e in cfg.layers:
            L = {}
            for name, shape in _shapes(e.mixer, W, e.ff, rank, rank).items():
                if len(shape) == 2:
                    L[name] = r(*shape, scale=shape[1] ** -0.5)
                elif name.endswith(plain):
                    L[name] = r(*shape, scale=0.1, at=1.0)
                elif name.endswith("dt_bias"):
                    L[name] = r(*shape, scale=0.5, at=-4.0)
                else:
                    L[name] = r(*shape, scale=0.1)
            w.layers.append(L)
        return w

    def num_parameters(self) -> int:
        return sum(t.numel() for t in self.state_dict().values())

    def to(self, device, dtype) -> "GelutarWeights":
        """Matrices in ``dtype``; vectors and convolution taps, which enter fp32 arithmetic, in fp32."""
        w = GelutarWeights(self.cfg)
        mv = lambda t, exact=False: t.to(device=device, dtype=torch.float32 if exact or t.dim() == 1 else dtype).contiguous()
        w.embed, w.head, w.final_norm = mv(self.embed), mv(self.head), mv(self.final_norm)
        w.layers = [{k: mv(v, k.endswith(".conv")) for k, v in L.items()} for L in self.layers]
        return w


class PagedGelutar(PagedModel):
    architecture = "gelutar"
    continues_prompts = True
    rewinds = False                    # a recurrent state cannot give a token back

    def __init__(self, weights: GelutarWeights, device, dtype):
        super().__init__(weights, device, dtype)
        c, w = self.cfg, self.weights
        self.final_norm = 1 + w.final_norm
        self.logit_norm = self.final_norm * c.logit_scale
        self.head = RowPack.pad(w.head)
        self.prep: List[dict] = []
        for e, L in zip(c.layers, w.layers):
            d = dict(norm1=1 + L["norm1"], ff=e.ff)
            m = e.mixer
            if isinstance(m, ParallelMixer):
                a, b = m.left, m.right
                d["pack"] = RowPack({**{n: L["mix." + n].shape[0] for n in _LEFT}, "conv": sum(L["mix." + n].shape[0] for n in _CONV),
                                     "left.g": a.heads, "right.b": b.heads, "low": RowPack.up(L["mix.right.a1"].shape[0]) + L["mix.right.g1"].shape[0]})
                low = torch.cat([RowPack.pad(L["mix.right.a1"]), L["mix.right.g1"]])
                d["w_in"] = d["pack"].pack({**{n: L["mix." + n] for n in _LEFT + ("left.g", "right.b")}, "low": low,
                                            "conv": torch.cat([L["mix." + n] for n in _CONV])})
                d["conv"] = torch.cat([L[f"mix.{n}.conv"] for n in _CONV]).t().contiguous()          # [taps, channels]
                # few rows: both low-rank gates as one product, block-diagonal second matrices over the packed first ones; many rows: the
                # output gate's alone, the decays' is formed where it is used
                ra, rg = RowPack.up(L["mix.right.a1"].shape[0]), L["mix.right.g1"].shape[0]
                a2, g2 = L["mix.right.a2"], L["mix.right.g2"]
                gates = a2.new_zeros(RowPack.up(a2.shape[0]) + g2.shape[0], RowPack.up(ra + rg))
                gates[:a2.shape[0], :a2.shape[1]] = a2
                gates[RowPack.up(a2.shape[0]):, ra:ra + rg] = g2
                d["gates"], d["gate_cols"] = RowPack.pad(gates), RowPack.up(a2.shape[0])
                d["a2"], d["g2"], d["rank_a"] = gates[:d["gate_cols"], :ra].contiguous(), RowPack.pad(gates[d["gate_cols"]:, ra:]), ra
                d["attn"] = A.WindowAttention(a.heads, a.kv_heads, a.dim, a.vdim, min(a.window, A.UNBOUNDED), min(a.keep_first, A.UNBOUNDED), a.scale, L["mix.left.sink"])
                d["delta"] = R.DeltaRule(b.heads, b.kv_heads, b.dim, b.vdim, L["mix.right.A_log"].exp(), L["mix.right.dt_bias"])
                for n in ("left.q.norm", "left.k.norm", "right.norm", "left.out", "right.out"):
                    d[n] = L["mix." + n]
                d["left.o"], d["right.o"] = L["mix.left.o"], L["mix.right.o"]
            else:
                d["pack"] = RowPack({n: L["mix." + n].shape[0] for n in "qkvg"})
                d["w_in"] = d["pack"].pack({n: L["mix." + n] for n in "qkvg"})
                d["light"] = R.DecayAttention(m.heads, m.dim, m.vdim, torch.tensor(m.decay, dtype=torch.float32, device=device))
                d["norm"], d["o"] = L["mix.norm"], L["mix.o"]
            if e.ff:
                d["norm2"] = 1 + L["norm2"]
                d["up"] = RowPack.pad(L["mlp.up"])
                d["down"] = RowPack.pad(L["mlp.down"].t()).t().contiguous() if e.ff % 8 else L["mlp.down"]
            self.prep.append(d)
        self.attns = [d["attn"] for d in self.prep if "attn" in d]
        # the packed copies are what runs: keep the unpacked matrices out of device memory
        w.layers = [{k: t for k, t in L.items() if t.dim() == 1} for L in w.layers]
        count = weights.num_parameters()
        w.num_parameters = lambda: count

    # ---- what the cache holds
    def kv_shapes(self):
        return [(d["attn"].kv_heads, d["attn"].dim_stored, d["attn"].vdim_stored) if "attn" in d else (0, 0, 0) for d in self.prep]

    def state_shapes(self):
        out = []
        for e in self.cfg.layers:
            m = e.mixer
            if isinstance(m, ParallelMixer):
                b = m.right
                out.append({"S": ((b.heads, b.dim, b.vdim), torch.float32),
                            "conv": ((b.conv - 1, 2 * b.kv_heads * b.dim + b.heads * b.vdim), self.dtype)})
            else:
                out.append({"S": ((m.heads, m.dim, m.vdim), torch.float32)})
        return out

    def cache_window(self):
        return max((a.window for a in self.attns), default=1)

    def kept_tokens(self):
        return max((a.keep for a in self.attns), default=0)

    def pick_splits(self, rows: int, max_len: int) -> int:
        return max((A.pick_splits(rows, a.kv_heads, a.most_keys(max_len)) for a in self.attns), default=1)

    # ---- the passes
    def _parallel(self, d, h, l, kv, page_table, pos, req, seqs, attend) -> list:
        from ..ops.gemm import linear
        a, pk, eps = d["attn"], d["pack"], self.cfg.eps
        p = linear(h, d["w_in"])
        q = A.proj_norm_write(p, tuple(pk.at[n] for n in _LEFT), a, d["left.q.norm"], d["left.k.norm"], eps, pos, req, page_table, kv.k[l], kv.v[l])
        c = R.short_conv(pk.cols(p, "conv"), d["conv"], kv.state[l]["conv"], pos, req, seqs)
        r, at, low = d["delta"], d["gate_cols"], pk.cols(p, "low", padded=True)
        if p.shape[0] > MERGE_GATES:
            decay, gate = (low[:, :d["rank_a"]], d["a2"]), linear(low[:, d["rank_a"]:], d["g2"])
        else:
            gates = S.linear_f32(low, d["gates"])
            decay, gate = gates[:, :r.heads * r.dim], gates[:, at:]
        o = R.delta_rule(c, r, pk.cols(p, "right.b"), decay, kv.state[l]["S"], pos, req, seqs)
        o = R.group_norm_gate(o, d["right.norm"], gate[:, :r.heads * r.vdim], eps, self.dtype)
        y = attend(l, a, q, pk.cols(p, "left.g"))
        return [S.linear_branch(y, d["left.o"], 0.5, d["left.out"]), S.linear_branch(o, d["right.o"], 0.5, d["right.out"])]

    def _lightning(self, d, h, l, kv, pos, req, seqs) -> list:
        from ..ops.gemm import linear
        pk = d["pack"]
        p = linear(h, d["w_in"])
        o = R.decay_attention(p, d["light"], tuple(pk.at[n] for n in "qkv"), kv.state[l]["S"], pos, req, seqs)
        y = R.group_norm_gate(o, d["norm"], pk.cols(p, "g"), self.cfg.eps, self.dtype)
        return [S.linear_branch(y, d["o"])]

    def _layers(self, ids, kv, page_table, pos, req, seqs, attend, last: Optional[torch.Tensor]):
        """``attend(layer, attention, q, gate)``: the attention over the pages once this pass's keys and values are in them.  Returns
        the fp32 stream and, with ``last`` (a norm weight), its norm."""
        from ..ops.gemm import linear_relu2
        eps = self.cfg.eps
        x, _ = S.embed_residual(ids, self.weights.embed, self.cfg.embed_scale, copy=False)
        steps = [(d, w) for d in self.prep for w in ("norm1", "norm2") if w in d]
        h = S.row_norm((x, x), 1.0, eps, w=steps[0][0]["norm1"], dtype=self.dtype) if steps else None
        l = -1
        for i, (d, which) in enumerate(steps):
            after = steps[i + 1][0][steps[i + 1][1]] if i + 1 < len(steps) else last
            if which == "norm1":
                l += 1
                b = self._parallel(d, h, l, kv, page_table, pos, req, seqs, attend) if "attn" in d else self._lightning(d, h, l, kv, pos, req, seqs)
            else:
                b = [S.linear_branch(linear_relu2(h, d["up"]), d["down"])]
            h = S.residual_norm(x, b, eps, after, self.dtype)
        if last is not None and not steps:
            h = S.row_norm((x, x), 1.0, eps, w=last, dtype=self.dtype)
        return x, h

    def prompt_pass(self, kv, page_table, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        top = max(at + n for at, n in zip(batch.starts, batch.lens()))
        seqs = R.Sequences.of(batch.offs, batch.starts, batch.rows, self.device)
        tiles = A.PromptTiles.of(batch.offs, batch.starts, batch.rows, self.device) if batch.offs[-1] >= A.TILES_FROM else None

        def attend(l, a, q, gate):
            if tiles is not None and A.tiles_supported(q, a):
                return A.window_attention_tiles(q, a, tiles, page_table, kv.k[l], kv.v[l], gate)
            ns = A.pick_splits(q.shape[0], a.kv_heads, a.most_keys(top))
            return A.window_attention(q, a, batch.pos, batch.req, page_table, kv.k[l], kv.v[l], ns, top, gate)
        x, _ = self._layers(batch.ids, kv, page_table, batch.pos, batch.req, seqs, attend, None)
        if hidden:
            return S.row_norm((x, x), 1.0, self.cfg.eps, w=self.final_norm, dtype=self.dtype)
        h = S.row_norm((x, x), 1.0, self.cfg.eps, w=self.logit_norm, index=batch.want, dtype=self.dtype)
        return S.linear_f32(h, self.head)[:, :self.cfg.vocab_size]

    def decode_pass(self, kv, page_table, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        ids, pos, req = meta[:, 0], meta[:, 1], meta[:, 2]

        def attend(l, a, q, gate):
            # no row sees more keys than the splits were chosen for; a layer that sees fewer needs no more than its own
            cover = min(a.window + a.keep, nsplit * A.KEYS_PER_CTA)
            return A.window_attention(q, a, pos, req, page_table, kv.k[l], kv.v[l], min(nsplit, max(1, -(-cover // 16))), cover, gate)
        _, h = self._layers(ids, kv, page_table, pos, req, None, attend, self.logit_norm)
        return S.linear_f32(h, self.head)[:, :self.cfg.vocab_size]


register_model(GelutarConfig, GelutarWeights, PagedGelutar, "gelutar")
