"""Kifusun for the batching engine: configuration, weights and the two passes.

The residual stream is fp32 and a sublayer reads it as it is; an RMS norm with a single number as its weight sits on each
sublayer's output, before the sum.  Attention is gated (``ops/gated_attention.py``): q and k are normalised per head, there is no
rotation, a score is soft-capped, gets a learned bias by distance and a number per head, and its sigmoid, mixed across the heads,
weighs the values inside a sliding window.  Layers marked ``v_mix`` blend their values with those of the first such layer.  The
feed-forward is gated with the tanh form of GELU.  Every layer brings its own sizes.

A model directory holds ``config.json`` (``"architecture": "Kifusun"``) and ``model.safetensors`` with the names of
:meth:`KifusunWeights.state_dict`."""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import gated_attention as A
from ..ops import residual as S
from .paged import PagedModel, PromptBatch, register_model


@dataclass
class AttentionLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    window: int
    bias_max: float
    v_mix: bool = False
    ff: int = 0                        # feed-forward width; 0: the layer has none

    def __post_init__(self):
        if self.heads < 1 or self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads over {self.kv_heads} key/value heads")
        if min(self.dim, self.vdim, self.window) < 1:
            raise ValueError(f"head sizes {self.dim} / {self.vdim} and window {self.window} must be positive")


@dataclass
class KifusunConfig:
    vocab_size: int
    hidden_size: int
    embed_scale: float
    eps: float
    layers: List[AttentionLayer] = field(default_factory=list)
    max_position_embeddings: int = 131072      # nothing in the design bounds a position; this sizes the page table
    bos_token_id: Optional[int] = None
    eos_token_id: int = -1

    @classmethod
    def from_dict(cls, d: dict) -> "KifusunConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "attention":
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of Kifusun")
            m, ff = e["mixer"], e.get("mlp")
            if ff is not None and ff["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {ff['kind']!r} is not part of Kifusun")
            layers.append(AttentionLayer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                         float(m["softcap"]), int(m["mask"]["size"]), float(m["bias_max"]), bool(m.get("v_mix", False)),
                                         int(ff["ff"]) if ff is not None else 0))
        return cls(int(d["vocab"]), int(d["width"]), float(d["embedding"]["scale"]), float(d["norm"]["eps"]), layers)

    @classmethod
    def from_json(cls, path: str) -> "KifusunConfig":
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        def num(v):
            return int(v) if float(v).is_integer() else v
        layers = [{"type": "attention",
                   "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "softcap": m.softcap,
                             "mask": {"size": m.window}, "bias_max": num(m.bias_max), "v_mix": m.v_mix},
                   "mlp": {"kind": "dense", "ff": m.ff} if m.ff else None} for m in self.layers]
        return {"architecture": "Kifusun", "vocab": self.vocab_size, "width": self.hidden_size, "embedding": {"scale": self.embed_scale},
                "norm": {"eps": self.eps}, "layers": layers}


class KifusunWeights:
    """Weights in the layout the passes run: q/k/v packed into one matrix, gate/up packed into one, single numbers as floats."""

    def __init__(self, cfg: KifusunConfig):
        self.cfg = cfg
        self.embed: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.final_norm = 1.0
        self.layers: List[Dict[str, torch.Tensor]] = []      # wqkv, bqkv, q_norm, k_norm, rel, talk, head_bias, wo[, w_gate_up, w_down]
        self.numbers: List[Dict[str, float]] = []            # norm1, norm2, vmix

    @classmethod
    def from_state_dict(cls, cfg: KifusunConfig, sd: Dict[str, torch.Tensor]) -> "KifusunWeights":
        w = cls(cfg)
        w.embed, w.head, w.final_norm = sd["embed"], sd["head"], float(sd["final.norm"])
        if tuple(w.embed.shape) != (cfg.vocab_size, cfg.hidden_size) or tuple(w.head.shape) != (cfg.vocab_size, cfg.hidden_size):
            raise ValueError(f"embed {tuple(w.embed.shape)} / head {tuple(w.head.shape)} for vocab {cfg.vocab_size}, width {cfg.hidden_size}")
        for i, m in enumerate(cfg.layers):
            p = f"l{i}."
            x = p + "mix."
            L = dict(wqkv=torch.cat([sd[x + "q"], sd[x + "k"], sd[x + "v"]]), bqkv=torch.cat([sd[x + "q.b"], sd[x + "k.b"], sd[x + "v.b"]]),
                     q_norm=sd[x + "q.norm"], k_norm=sd[x + "k.norm"], rel=sd[x + "rel"], talk=sd[x + "talk"], head_bias=sd[x + "pb"], wo=sd[x + "o"])
            n = dict(norm1=float(sd[p + "norm1"]), norm2=0.0, vmix=float(sd[x + "vmix"]) if x + "vmix" in sd else 0.0)
            if m.ff:
                L["w_gate_up"] = torch.cat([sd[p + "mlp.gate"], sd[p + "mlp.up"]])
                L["w_down"] = sd[p + "mlp.down"]
                n["norm2"] = float(sd[p + "norm2"])
            qkv = m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)
            want = dict(wqkv=(qkv, cfg.hidden_size), bqkv=(qkv,), q_norm=(m.dim,), k_norm=(m.dim,), talk=(m.heads, m.heads), head_bias=(m.heads,),
                        wo=(cfg.hidden_size, m.heads * m.vdim), w_gate_up=(2 * m.ff, cfg.hidden_size), w_down=(cfg.hidden_size, m.ff))
            for k, t in L.items():
                if k in want and tuple(t.shape) != want[k]:
                    raise ValueError(f"layer {i}: {k} has shape {tuple(t.shape)}, the configuration asks for {want[k]}")
            w.layers.append(L)
            w.numbers.append(n)
        return w

    def state_dict(self) -> Dict[str, torch.Tensor]:
        one = lambda v: torch.tensor(v, dtype=self.embed.dtype)
        sd = {"embed": self.embed, "head": self.head, "final.norm": one(self.final_norm)}
        for i, (m, L, n) in enumerate(zip(self.cfg.layers, self.layers, self.numbers)):
            p, sizes = f"l{i}.", [m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim]
            for name, t, b in zip("qkv", L["wqkv"].split(sizes), L["bqkv"].split(sizes)):
                sd[f"{p}mix.{name}"], sd[f"{p}mix.{name}.b"] = t, b
            sd.update({p + "norm1": one(n["norm1"]), p + "mix.vmix": one(n["vmix"]), p + "mix.q.norm": L["q_norm"], p + "mix.k.norm": L["k_norm"],
                       p + "mix.rel": L["rel"], p + "mix.talk": L["talk"], p + "mix.pb": L["head_bias"], p + "mix.o": L["wo"]})
            if m.ff:
                gate, up = L["w_gate_up"].split([m.ff, m.ff])
                sd.update({p + "norm2": one(n["norm2"]), p + "mlp.gate": gate, p + "mlp.up": up, p + "mlp.down": L["w_down"]})
        return sd

    @classmethod
    def random(cls, cfg: KifusunConfig, seed: int = 0, dtype=torch.float32, device="cpu", bias_rows: int = 32) -> "KifusunWeights":
        """Random weights of the right scales (benchmarks and tests), drawn on ``device``."""
        g = torch.Generator(device=device).manual_seed(seed)

        def r(*s, scale=1.0, at=0.0):
            return (at + torch.randn(*s, generator=g, device=device) * scale).to(dtype)
        W = cfg.hidden_size
        w = cls(cfg)
        w.embed, w.head = r(cfg.vocab_size, W, scale=1.0 / cfg.embed_scale), r(cfg.vocab_size, W, scale=W ** -0.5)
        for m in cfg.layers:
            qkv = m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)
            L = dict(wqkv=r(qkv, W, scale=W ** -0.5), bqkv=r(qkv, scale=0.1), q_norm=r(m.dim, scale=0.1, at=1.0), k_norm=r(m.dim, scale=0.1, at=1.0),
                     rel=r(bias_rows, m.heads, scale=0.3), talk=r(m.heads, m.heads, scale=0.2 * m.heads ** -0.5), head_bias=r(m.heads, scale=0.3, at=-2.0),
                     wo=r(W, m.heads * m.vdim, scale=(m.heads * m.vdim) ** -0.5))
            L["talk"] += torch.eye(m.heads, dtype=dtype, device=device)
            if m.ff:
                L.update(w_gate_up=r(2 * m.ff, W, scale=W ** -0.5), w_down=r(W, m.ff, scale=m.ff ** -0.5))
            w.layers.append(L)
            w.numbers.append(dict(norm1=1.0, norm2=0.75, vmix=0.375))
        return w

    def num_parameters(self) -> int:
        return sum(t.numel() for L in self.layers for t in L.values()) + self.embed.numel() + self.head.numel()

    _exact = ("bqkv", "q_norm", "k_norm", "rel", "talk", "head_bias")        # enter fp32 arithmetic

    def to(self, device, dtype) -> "KifusunWeights":
        w = KifusunWeights(self.cfg)
        mv = lambda t, k="": t.to(device=device, dtype=torch.float32 if k in self._exact else dtype).contiguous()
        w.embed, w.head, w.final_norm = mv(self.embed), mv(self.head), self.final_norm
        w.layers = [{k: mv(v, k) for k, v in L.items()} for L in self.layers]
        w.numbers = [dict(n) for n in self.numbers]
        return w


def _pad_rows(t: torch.Tensor) -> torch.Tensor:
    pad = -t.shape[0] % 8
    return torch.cat([t, t.new_zeros((pad,) + tuple(t.shape[1:]))]) if pad else t


class PagedKifusun(PagedModel):
    architecture = "kifusun"
    continues_prompts = True

    def __init__(self, weights: KifusunWeights, device, dtype):
        super().__init__(weights, device, dtype)
        self.attn = [A.GatedAttention(m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.scale, m.softcap,
                                      A.distance_bias(L["rel"], m.bias_max, m.window, L["head_bias"]), L["talk"])
                     for m, L in zip(self.cfg.layers, self.weights.layers)]
        # the projection kernel takes rows in groups of eight: odd sizes get rows (and the columns that read them) of zeros
        self.head = _pad_rows(self.weights.head)
        fp32_bias = dtype == torch.bfloat16 and self.cfg.hidden_size % 8 == 0 and torch.device(device).type == "cuda"
        for m, L in zip(self.cfg.layers, self.weights.layers):
            L["wqkv"], L["bqkv"] = _pad_rows(L["wqkv"]), _pad_rows(L["bqkv"]).to(torch.float32 if fp32_bias else dtype)
            if m.ff % 8:
                L["w_gate_up"] = torch.cat([_pad_rows(t) for t in L["w_gate_up"].split([m.ff, m.ff])])
                L["w_down"] = _pad_rows(L["w_down"].t()).t().contiguous()

    def kv_shapes(self):
        return [(a.kv_heads, a.dim_stored, a.vdim_stored) for a in self.attn]

    def cache_window(self):
        return max(a.window for a in self.attn)

    def pick_splits(self, rows: int, max_len: int) -> int:
        return A.pick_splits(rows, self.cache_window(), max_len)

    def _layers(self, stream: S.Stream, kv, page_table, pos, req, attend) -> S.Stream:
        """``attend(layer, q)``: the attention over the pages once this pass's keys and values are in them."""
        from ..ops.gemm import linear, linear_swiglu
        eps, v_first = self.cfg.eps, None
        for l, (m, L, n, a) in enumerate(zip(self.cfg.layers, self.weights.layers, self.weights.numbers, self.attn)):
            qkv = linear(stream[1], L["wqkv"], L["bqkv"])
            q = A.head_norm_write(qkv, a, L["q_norm"], L["k_norm"], eps, pos, req, page_table, kv.k[l], kv.v[l],
                                  v_first if m.v_mix else None, n["vmix"])
            if m.v_mix and v_first is None:
                v_first = qkv[:, (m.heads + m.kv_heads) * m.dim:][:, :m.kv_heads * m.vdim]
            stream = S.linear_post_norm_add(attend(l, q), L["wo"], stream, n["norm1"], eps)
            if m.ff:
                stream = S.linear_post_norm_add(linear_swiglu(stream[1], L["w_gate_up"], gelu=True), L["w_down"], stream, n["norm2"], eps)
        return stream

    def _logits(self, stream: S.Stream, index=None) -> torch.Tensor:
        h = S.row_norm(stream, self.weights.final_norm, self.cfg.eps, index=index)
        return S.linear_f32(h, self.head)[:, :self.cfg.vocab_size]

    def prompt_pass(self, kv, page_table, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        top = max(at + n for at, n in zip(batch.starts, batch.lens()))
        tiles = A.PromptTiles.of(batch.offs, batch.starts, batch.rows, self.device) if batch.offs[-1] >= A.TILES_FROM else None

        def attend(l, q):
            a = self.attn[l]
            if tiles is not None and A.tiles_supported(q, a):
                return A.gated_attention_tiles(q, a, tiles, page_table, kv.k[l], kv.v[l])
            return A.gated_attention(q, a, batch.pos, batch.req, page_table, kv.k[l], kv.v[l], A.pick_splits(q.shape[0], a.window, top), top)
        stream = self._layers(S.embed_residual(batch.ids, self.weights.embed, self.cfg.embed_scale), kv, page_table, batch.pos, batch.req, attend)
        if hidden:
            return S.row_norm(stream, self.weights.final_norm, self.cfg.eps)
        return self._logits(stream, batch.want)

    def decode_pass(self, kv, page_table, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        ids, pos, req = meta[:, 0], meta[:, 1], meta[:, 2]

        def attend(l, q):
            # no row sees more keys than the splits were chosen for; a layer with a shorter window needs no more than its own
            a = self.attn[l]
            cover = min(a.window, nsplit * A.KEYS_PER_CTA)
            return A.gated_attention(q, a, pos, req, page_table, kv.k[l], kv.v[l], min(nsplit, max(1, -(-cover // 16))), cover)
        return self._logits(self._layers(S.embed_residual(ids, self.weights.embed, self.cfg.embed_scale), kv, page_table, pos, req, attend))


register_model(KifusunConfig, KifusunWeights, PagedKifusun, "kifusun")
