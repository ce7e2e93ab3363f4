"""Tifepel for the batching engine: configuration, weights and the two passes.

A pre-norm decoder (layer norm without bias) over several fp32 residual streams (``ops/streams.py``): every sublayer reads a weighed sum of
them, passes its input through a causal convolution over time, and its output is gated element by element before it joins the streams.
The streams start from a token, a pair and a position table.  Every layer brings its own mixer and sizes:

* ``mamba2``: a state-space recurrence (``ops/recurrence.py``) behind a short convolution, the gate ahead of a grouped norm;
* ``attention``: softmax attention over all earlier tokens (``ops/window_attention.py``) with q and k normed per head, a factor on q that
  grows with the position, and a learned bias by distance.

The feed-forward is a mixture of experts (``ops/experts.py``) with a softmax router, identity outputs and a shared expert; a layer may have
none.  A run of layers may be passed several times with the same weights; every pass has pages and states of its own.

A model directory holds ``config.json`` (``"architecture": "Tifepel"``) and ``model.safetensors`` with the names of
:meth:`TifepelWeights.state_dict`."""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops import experts as X
from ..ops import recurrence as R
from ..ops import residual as S
from ..ops import streams as H
from ..ops import window_attention as A
from ..ops.gated_attention import distance_bias, head_norm_write
from .paged import PagedModel, PromptBatch, RowPack, register_model


@dataclass
class Mamba2Mixer:
    heads: int
    groups: int
    state: int                         # rows of a head's state
    vdim: int
    conv: int                          # taps
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass
class BiasedMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float                    # distance at which the last bucket of the bias begins to repeat
    temp_coef: float = 0.0
    temp_every: float = 1.0


@dataclass
class SharedExpertsFF:
    ff: int
    experts: int
    top: int
    identity: int = 0                  # router outputs that return the input itself
    shared: int = 0                    # width of the expert that runs for every token; 0: none


@dataclass
class TifepelLayer:
    mixer: Union[Mamba2Mixer, BiasedMixer]
    experts: Optional[SharedExpertsFF] = None

    def __post_init__(self):
        m, x = self.mixer, self.experts
        part = m.groups if isinstance(m, Mamba2Mixer) else m.kv_heads
        if m.heads < 1 or part < 1 or m.heads % part:
            raise ValueError(f"{m.heads} heads over {part} groups")
        if min(m.vdim, m.state if isinstance(m, Mamba2Mixer) else m.dim) < 1:
            raise ValueError("head sizes must be positive")
        if isinstance(m, Mamba2Mixer) and (m.conv < 1 or m.norm_groups < 1 or m.inner % m.norm_groups):
            raise ValueError(f"a convolution of {m.conv} taps, {m.inner} columns in {m.norm_groups} groups")
        if isinstance(m, BiasedMixer) and m.temp_every <= 0:
            raise ValueError(f"a temperature that changes every {m.temp_every} positions")
        if x is not None and not (x.experts >= 1 and x.identity >= 0 and 1 <= x.top <= x.experts + x.identity):
            raise ValueError(f"{x.top} of {x.experts} + {x.identity} experts")

    @property
    def kind(self) -> str:
        return "mamba2" if isinstance(self.mixer, Mamba2Mixer) else "attention"


@dataclass
class TifepelConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    max_position_embeddings: int       # rows of the position table
    streams: int
    taps: int                          # of the convolution on every sublayer's input
    buckets: int                       # of the pair table
    mul_prev: int
    mul_cur: int
    layers: List[TifepelLayer] = field(default_factory=list)
    loop: Optional[Tuple[int, int, int]] = None      # layers start .. stop - 1 run `times` times in a row
    bos_token_id: Optional[int] = None
    eos_token_id: int = -1

    def __post_init__(self):
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start <= stop <= len(self.layers) or times < 1:
                raise ValueError(f"a loop over layers {start} .. {stop} of {len(self.layers)}, {times} times")
        if not 1 <= self.streams <= H.MAX_STREAMS or self.taps < 1 or self.buckets < 1:
            raise ValueError(f"{self.streams} streams (at most {H.MAX_STREAMS}), {self.taps} taps, {self.buckets} buckets")

    def runs(self) -> List[int]:
        """The layer of every layer run."""
        n = len(self.layers)
        start, stop, times = self.loop or (0, 0, 1)
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    @classmethod
    def from_dict(cls, d: dict) -> "TifepelConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, ff = e["mixer"], e.get("mlp")
            ints = lambda *names: [int(m[n]) for n in names]
            if e["type"] == "mamba2":
                mixer = Mamba2Mixer(*ints("heads", "groups", "state", "vdim", "conv", "norm_groups"))
            elif e["type"] == "attention":
                t = m.get("q_temp") or {"coef": 0.0, "every": 1}
                mixer = BiasedMixer(*ints("heads", "kv_heads", "dim", "vdim"), float(m["scale"]), float(m["bias_max"]), float(t["coef"]), float(t["every"]))
            else:
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of Tifepel")
            experts = None
            if ff is not None:
                if ff["kind"] != "moe":
                    raise ValueError(f"layer {i}: feed-forward {ff['kind']!r} is not part of Tifepel")
                r, shared = ff["router"], ff.get("shared")
                experts = SharedExpertsFF(int(ff["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(r.get("identity") or 0), int(shared["ff"]) if shared else 0)
            layers.append(TifepelLayer(mixer, experts))
        lp, b = d.get("loop"), d["embedding"]["bigram"]
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), int(d["max_positions"]), int(d["streams"]), int(d["canon"]["taps"]),
                   int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]), layers, (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None)

    @classmethod
    def from_json(cls, path: str) -> "TifepelConfig":
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for e in self.layers:
            m, x = e.mixer, e.experts
            if isinstance(m, Mamba2Mixer):
                mixer = {"heads": m.heads, "groups": m.groups, "state": m.state, "vdim": m.vdim, "conv": m.conv, "norm_groups": m.norm_groups}
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "bias_max": m.bias_max,
                         "q_temp": {"coef": m.temp_coef, "every": m.temp_every}}
            mlp = None
            if x:
                mlp = {"kind": "moe", "expert": {"ff": x.ff}, "router": {"experts": x.experts, "top": x.top, "identity": x.identity},
                       "shared": {"ff": x.shared} if x.shared else None}
            layers.append({"type": e.kind, "mixer": mixer, "mlp": mlp})
        d = {"architecture": "Tifepel", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps}, "max_positions": self.max_position_embeddings,
             "streams": self.streams, "canon": {"taps": self.taps}, "embedding": {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}},
             "layers": layers}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d


def _shapes(e: TifepelLayer, c: TifepelConfig, rel_rows: int) -> Dict[str, Tuple[int, ...]]:
    """Tensor shapes of one layer (names without the layer's prefix); ``rel_rows``: buckets of an attention layer's bias."""
    m, x, W = e.mixer, e.experts, c.hidden_size
    if isinstance(m, Mamba2Mixer):
        mix = {"in": (m.inner + m.channels + m.heads, W), "conv": (m.channels, m.conv), "conv.b": (m.channels,), "dt_bias": (m.heads,), "A_log": (m.heads,),
               "D": (m.heads,), "norm": (m.inner,)}
    else:
        mix = {"q": (m.heads * m.dim, W), "k": (m.kv_heads * m.dim, W), "v": (m.kv_heads * m.vdim, W), "rel": (rel_rows, m.heads)}
    t = {"mix." + k: s for k, s in mix.items()}
    t["mix.o"] = (W, m.heads * m.vdim)
    for n in ("1", "2") if x else ("1",):
        t.update({"norm" + n: (W,), "canon" + n: (W, c.taps), "rg" + n: (W, W), f"rg{n}.b": (W,), f"hc{n}.in": (c.streams,), f"hc{n}.out": (c.streams,),
                  f"hc{n}.mix": (c.streams, c.streams)})
    if x:
        for name, ff in [(f"e{i}", x.ff) for i in range(x.experts)] + ([("shared", x.shared)] if x.shared else []):
            t.update({f"mlp.{name}.gate": (ff, W), f"mlp.{name}.up": (ff, W), f"mlp.{name}.down": (W, ff)})
        t.update({"mlp.router": (x.experts + x.identity, W), "mlp.correction": (x.experts + x.identity,)})
    return t


_OUTER = ("embed", "bigram", "pos", "final.norm", "head")
_EXACT = (".conv", ".rel", "canon1", "canon2", ".mix")           # matrices that enter fp32 arithmetic


class TifepelWeights:
    """Weights by the names of the checkpoint, layer by layer (prefix dropped); :class:`PagedTifepel` packs what its passes read."""

    def __init__(self, cfg: TifepelConfig):
        self.cfg = cfg
        self.outer: Dict[str, torch.Tensor] = {}
        self.layers: List[Dict[str, torch.Tensor]] = []

    @staticmethod
    def _outer_shapes(c: TifepelConfig) -> Dict[str, Tuple[int, ...]]:
        W = c.hidden_size
        return dict(zip(_OUTER, ((c.vocab_size, W), (c.buckets + 1, W), (c.max_position_embeddings, W), (W,), (c.vocab_size, W))))

    @classmethod
    def from_state_dict(cls, cfg: TifepelConfig, sd: Dict[str, torch.Tensor]) -> "TifepelWeights":
        w = cls(cfg)

        def take(name, shape):
            if tuple(sd[name].shape) != shape:
                raise ValueError(f"{name} has shape {tuple(sd[name].shape)}, the configuration asks for {shape}")
            return sd[name]
        w.outer = {k: take(k, s) for k, s in cls._outer_shapes(cfg).items()}
        for i, e in enumerate(cfg.layers):
            rel = sd.get(f"l{i}.mix.rel")
            w.layers.append({k: take(f"l{i}.{k}", s) for k, s in _shapes(e, cfg, rel.shape[0] if rel is not None else 0).items()})
        return w

    def state_dict(self) -> Dict[str, torch.Tensor]:
        return {**self.outer, **{f"l{i}.{k}": t for i, L in enumerate(self.layers) for k, t in L.items()}}

    @classmethod
    def random(cls, cfg: TifepelConfig, seed: int = 0, dtype=torch.float32, device="cpu", rel_rows: int = 32) -> "TifepelWeights":
        """Random weights of the right scales (benchmarks and tests), drawn on ``device``."""
        g = torch.Generator(device=device).manual_seed(seed)

        def r(*s, scale=1.0, at=0.0):
            return (at + torch.randn(s, generator=g, device=device) * scale).to(dtype)

        def one(name, s):
            if name.startswith("hc"):
                if len(s) == 2:
                    return (torch.eye(s[0], device=device) + 0.1 * torch.randn(s, generator=g, device=device)).to(dtype)
                return r(*s, scale=0.1, at=1.0 / s[0] if name.endswith("in") else 1.0)
            if name.startswith("canon") or name.endswith(".conv"):
                return r(*s, scale=0.3)
            if len(s) == 2:
                return r(*s, scale=0.3 if name.endswith(".rel") else s[1] ** -0.5)
            if "norm" in name or name.endswith(".D"):
                return r(*s, scale=0.1, at=1.0)
            return r(*s, scale=0.5, at=-4.0) if name.endswith("dt_bias") else r(*s, scale=0.1)
        w = cls(cfg)
        w.outer = {k: one(k, s) if k in ("final.norm", "head") else r(*s) for k, s in cls._outer_shapes(cfg).items()}
        w.layers = [{k: one(k, s) for k, s in _shapes(e, cfg, rel_rows).items()} for e in cfg.layers]
        return w

    def num_parameters(self) -> int:
        return sum(t.numel() for t in self.state_dict().values())

    def to(self, device, dtype) -> "TifepelWeights":
        """Matrices in ``dtype``; vectors, numbers, convolution taps, biases by distance and connections, which enter fp32 arithmetic, in fp32."""
        w = TifepelWeights(self.cfg)
        mv = lambda k, t: t.to(device=device, dtype=torch.float32 if t.dim() < 2 or k.endswith(_EXACT) else dtype).contiguous()
        w.outer = {k: mv(k, t) for k, t in self.outer.items()}
        w.layers = [{k: mv(k, t) for k, t in L.items()} for L in self.layers]
        return w


class PagedTifepel(PagedModel):
    architecture = "tifepel"
    continues_prompts = True
    rewinds = False                    # convolutions and recurrent states cannot give a token back

    def __init__(self, weights: TifepelWeights, device, dtype):
        super().__init__(weights, device, dtype)
        c, w = self.cfg, self.weights
        o = w.outer
        self.embedding = H.PairEmbedding(o["embed"], o["bigram"], o["pos"], c.mul_prev, c.mul_cur)
        self.final, self.head = o["final.norm"], RowPack.pad(o["head"])
        gains: Dict[tuple, torch.Tensor] = {}

        def gain(coef, every):
            """The factor on q by position (fp32; the logarithm is taken in double precision)."""
            if coef and (coef, every) not in gains:
                p = torch.arange(1, c.max_position_embeddings + 1, dtype=torch.float64)
                gains[coef, every] = (1 + coef * torch.log1p(torch.floor(p / every))).float().to(device)
            return gains.get((coef, every))
        self.prep: List[dict] = []
        for e, L in zip(c.layers, w.layers):
            m, x = e.mixer, e.experts
            mix = {k[4:]: t for k, t in L.items() if k.startswith("mix.")}
            d = dict(kind=e.kind, o=mix["o"])
            for n in ("1", "2") if x else ("1",):
                d["link" + n] = H.Connection(L[f"hc{n}.in"], L[f"hc{n}.mix"], L[f"hc{n}.out"], L["norm" + n], L["canon" + n].t().contiguous(), L[f"rg{n}.b"])
                d["gate" + n] = RowPack.pad(L["rg" + n])
            if isinstance(m, Mamba2Mixer):
                z, xbc, dt = mix["in"].split([m.inner, m.channels, m.heads])
                d["pack"] = RowPack({"z": m.inner, "xbc": m.channels, "dt": m.heads})
                d["w_in"] = d["pack"].pack({"z": z, "xbc": xbc, "dt": dt})
                d["conv"], d["conv.b"] = mix["conv"].t().contiguous(), mix["conv.b"]             # [taps, channels]
                d["ssm"] = R.StateSpace(m.heads, m.groups, m.state, m.vdim, mix["A_log"].exp(), mix["dt_bias"], mix["D"])
                d["cols"] = (m.inner + m.groups * m.state, m.inner, 0)                           # of C, B and x behind the convolution
                d["norm"], d["norm_groups"] = mix["norm"], m.norm_groups
            else:
                d["pack"] = RowPack({n: mix[n].shape[0] for n in "qkv"})
                d["w_in"] = d["pack"].pack({n: mix[n] for n in "qkv"})
                d["attn"] = A.WindowAttention(m.heads, m.kv_heads, m.dim, m.vdim, A.UNBOUNDED, 0, m.scale, 
                                              rel=distance_bias(mix["rel"], m.bias_max, c.max_position_embeddings))
                d["gain"] = gain(m.temp_coef, m.temp_every)
            if x:
                parts = lambda n: [L[f"mlp.e{i}.{n}"] for i in range(x.experts)]
                shared = tuple(L["mlp.shared." + n] for n in ("gate", "up", "down")) if x.shared else None
                join = x.shared <= X.SHARED_PARTS * x.ff
                d["experts"] = X.Experts.of(parts("gate"), parts("up"), parts("down"), L["mlp.router"], L["mlp.correction"], x.top, 1.0, softmax=True,
                                            shared=shared if join else None)
                if shared and not join:
                    d["shared"] = X.SharedExpert.of(*shared)
                for k in [k for k in L if k.startswith("mlp.e")]:
                    L[k] = L[k][:0]                        # the packed copy is what runs
            self.prep.append(d)
        self.runs = [self.prep[i] for i in c.runs()]
        count = weights.num_parameters()
        w.layers = [{k: t for k, t in L.items() if t.dim() < 2} for L in w.layers]
        w.num_parameters = lambda: count

    # ---- what the cache holds: every layer run has entries of its own, and one more entry holds what the embedding carries along
    def kv_shapes(self):
        return [(d["attn"].kv_heads, d["attn"].dim_stored, d["attn"].vdim_stored) if "attn" in d else (0, 0, 0) for d in self.runs]

    def state_shapes(self):
        c, out = self.cfg, []
        for d in self.runs:
            s = {n: ((c.taps - 1, c.hidden_size), self.dtype) for n in ("canon1", "canon2") if "link" + n[-1] in d}
            r = d.get("ssm")
            if r:
                s.update({"S": ((r.heads, r.dim, r.vdim), torch.float32), "conv": ((d["conv"].shape[0] - 1, d["conv"].shape[1]), self.dtype)})
            out.append(s)
        return out + [{"token": ((1,), torch.int32)}]

    def cache_window(self):
        return None if any("attn" in d for d in self.runs) else 1

    def pick_splits(self, rows: int, max_len: int) -> int:
        """Keys that the splits of every attention layer have to cover, in units of 32: a power of two, so that it changes rarely."""
        units = 1
        while units * 32 < max_len:
            units *= 2
        return units

    # ---- the passes
    def _mamba2(self, d, h, l, kv, pos, req, seqs):
        from ..ops.gemm import linear
        pk = d["pack"]
        p = linear(h, d["w_in"])
        x = R.short_conv(pk.cols(p, "xbc"), d["conv"], kv.state[l]["conv"], pos, req, seqs, bias=d["conv.b"])
        y = R.state_space(x, d["ssm"], d["cols"], pk.cols(p, "dt"), kv.state[l]["S"], pos, req, seqs)
        return R.group_norm_gate(y, d["norm"], pk.cols(p, "z"), self.cfg.eps, self.dtype, act="silu", groups=d["norm_groups"], gate_first=True)

    def _attention(self, d, h, l, kv, page_table, pos, req, attend):
        from ..ops.gemm import linear
        a, at = d["attn"], d["pack"].at
        q = head_norm_write(linear(h, d["w_in"]), a, None, None, self.cfg.eps, pos, req, page_table, kv.k[l], kv.v[l], cols=(at["k"], at["v"]), gain=d["gain"])
        return attend(a, q, kv.k[l], kv.v[l])

    def _layers(self, ids, kv, page_table, pos, req, seqs, attend):
        """``attend``: the attention over the pages once this pass's keys are in them.  Returns the streams ``[n, S, W]``."""
        c = self.cfg
        x = H.pair_embed(ids, self.embedding, c.streams, kv.state[-1]["token"], pos, req, seqs)
        before = None
        for l, d in enumerate(self.runs):
            for n in ("1", "2") if "link2" in d else ("1",):
                link = d["link" + n]
                h, hc = H.step(x, before, link, c.eps, self.dtype, kv.state[l]["canon" + n], pos, req, seqs)
                gate = S.linear_branch(h, d["gate" + n])
                if n == "2":
                    before = H.Output(link, gate, X.run_shared(hc, d["shared"]) if "shared" in d else None, X.run(hc, d["experts"]))
                    continue
                o = self._mamba2(d, hc, l, kv, pos, req, seqs) if d["kind"] == "mamba2" else self._attention(d, hc, l, kv, page_table, pos, req, attend)
                before = H.Output(link, gate, S.linear_branch(o, d["o"]))
        if before is not None:
            H.step(x, before, None, c.eps, self.dtype, None, pos, req, seqs)
        return x

    def _logits(self, h):
        return S.linear_f32(h, self.head)[:, :self.cfg.vocab_size]

    def prompt_pass(self, kv, page_table, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        top = max(at + n for at, n in zip(batch.starts, batch.lens()))
        seqs = R.Sequences.of(batch.offs, batch.starts, batch.rows, self.device)
        tiles = A.PromptTiles.of(batch.offs, batch.starts, batch.rows, self.device) if batch.offs[-1] >= A.TILES_FROM else None

        def attend(a, q, k, v):
            if tiles is not None and A.tiles_supported(q, a):
                return A.window_attention_tiles(q, a, tiles, page_table, k, v)
            return A.window_attention(q, a, batch.pos, batch.req, page_table, k, v, A.pick_splits(q.shape[0], a.kv_heads, a.most_keys(top)), top)
        x = self._layers(batch.ids, kv, page_table, batch.pos, batch.req, seqs, attend)
        h = H.rows(x, self.final, self.cfg.eps, None if hidden else batch.want, self.dtype)
        return h if hidden else self._logits(h)

    def decode_pass(self, kv, page_table, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        ids, pos, req = meta[:, 0], meta[:, 1], meta[:, 2]
        cover = nsplit * 32

        def attend(a, q, k, v):
            keys = a.most_keys(cover)
            return A.window_attention(q, a, pos, req, page_table, k, v, A.pick_splits(q.shape[0], a.kv_heads, keys), cover)
        x = self._layers(ids, kv, page_table, pos, req, None, attend)
        return self._logits(H.rows(x, self.final, self.cfg.eps, None, self.dtype))


register_model(TifepelConfig, TifepelWeights, PagedTifepel, "tifepel")
