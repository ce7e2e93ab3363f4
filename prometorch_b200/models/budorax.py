"""Budorax for the batching engine: configuration, weights and the two passes.

A decoder whose norms are elementwise (``ops/tanh_norm.py``), one ahead of every sublayer and one on its output, around an fp32
residual stream.  Every layer brings its own mixer and sizes:

* ``delta``: the gated delta rule (``ops/recurrence.py``) with one decay per head, short convolutions, a gated output norm;
* ``attention``: differential attention (``ops/window_attention.py``), two softmax maps over the same values, inside chunks of
  positions, with interleaved rotary positions;
* ``latent_attention``: keys and values from one cached latent per token (``ops/latent_attention.py``), a gate per head.

The feed-forward is a mixture of experts (``ops/experts.py``); a layer may have none.  A run of layers may be passed several times
with the same weights; every pass has pages and states of its own and starts by adding the embedding output to the stream.  The
output projection is the embedding table, its logits are soft-capped.

A model directory holds ``config.json`` (``"architecture": "Budorax"``) and ``model.safetensors`` with the names of
:meth:`BudoraxWeights.state_dict`."""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops import experts as X
from ..ops import latent_attention as M
from ..ops import recurrence as R
from ..ops import residual as S
from ..ops import tanh_norm as T
from ..ops import window_attention as A
from ..ops.rotary import Rotary
from .paged import PagedModel, PromptBatch, RowPack, register_model


@dataclass
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                          # taps


@dataclass
class ChunkMixer:
    heads: int
    kv_heads: int
    dim: int                           # of each of the two maps
    vdim: int
    scale: float
    chunk: int
    rot_dims: int
    rot_base: float
    diff: float


@dataclass
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass
class ExpertFF:
    ff: int
    experts: int
    top: int
    scale: float


_KINDS = {"delta": DeltaMixer, "attention": ChunkMixer, "latent_attention": LatentMixer}


@dataclass
class BudoraxLayer:
    mixer: Union[DeltaMixer, ChunkMixer, LatentMixer]
    experts: Optional[ExpertFF] = None

    def __post_init__(self):
        m, x = self.mixer, self.experts
        kv = getattr(m, "kv_heads", m.heads)
        if m.heads < 1 or kv < 1 or m.heads % kv:
            raise ValueError(f"{m.heads} heads over {kv} key/value heads")
        if min(m.dim, m.vdim) < 1:
            raise ValueError(f"head sizes {m.dim} / {m.vdim} must be positive")
        if isinstance(m, DeltaMixer) and m.conv < 1:
            raise ValueError(f"a convolution of {m.conv} taps")
        if isinstance(m, ChunkMixer) and (m.chunk < 1 or m.rot_dims < 0 or m.rot_dims % 2 or m.rot_dims > m.dim):
            raise ValueError(f"chunks of {m.chunk}, {m.rot_dims} rotated of {m.dim} dimensions")
        if isinstance(m, LatentMixer) and (min(m.q_rank, m.kv_rank) < 1 or m.rot_dim < 0 or m.rot_dim % 2):
            raise ValueError(f"ranks {m.q_rank} / {m.kv_rank}, {m.rot_dim} rotated dimensions")
        if x is not None and not 1 <= x.top <= x.experts:
            raise ValueError(f"{x.top} of {x.experts} experts")

    @property
    def kind(self) -> str:
        return next(n for n, c in _KINDS.items() if isinstance(self.mixer, c))


@dataclass
class BudoraxConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: List[BudoraxLayer] = field(default_factory=list)
    loop: Optional[Tuple[int, int, int]] = None      # layers start .. stop - 1 run `times` times in a row
    softcap: Optional[float] = None
    max_position_embeddings: int = 131072      # nothing in the design bounds a position; this sizes the page table and the angles
    bos_token_id: Optional[int] = None
    eos_token_id: int = -1

    def __post_init__(self):
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start <= stop <= len(self.layers) or times < 1:
                raise ValueError(f"a loop over layers {start} .. {stop} of {len(self.layers)}, {times} times")

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, whether the embedding output joins the stream ahead of it) of every layer run."""
        start, stop, times = self.loop or (0, 0, 1)
        body = [(i, False) for i in range(start, stop)]
        again = [(start, True)] + body[1:] if body else []
        return [(i, False) for i in range(start)] + body + again * (times - 1) + [(i, False) for i in range(stop, len(self.layers))]

    @classmethod
    def from_dict(cls, d: dict) -> "BudoraxConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, ff = e["mixer"], e.get("mlp")
            ints = lambda *names: [int(m[n]) for n in names]
            if e["type"] == "delta":
                mixer = DeltaMixer(*ints("heads", "kv_heads", "dim", "vdim", "conv"))
            elif e["type"] == "attention":
                mixer = ChunkMixer(*ints("heads", "kv_heads", "dim", "vdim"), float(m["scale"]), int(m["mask"]["size"]), int(m["rot"]["dims"]),
                                   float(m["rot"]["base"]), float(m["diff"]))
            elif e["type"] == "latent_attention":
                mixer = LatentMixer(*ints("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), float(m["scale"]), float(m["rot"]["base"]))
                if int(m["rot"].get("dims", mixer.rot_dim)) != mixer.rot_dim:
                    raise ValueError(f"layer {i}: {m['rot']['dims']} rotated dimensions in a rotated part of {mixer.rot_dim}")
            else:
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of Budorax")
            experts = None
            if ff is not None:
                if ff["kind"] != "moe":
                    raise ValueError(f"layer {i}: feed-forward {ff['kind']!r} is not part of Budorax")
                r = ff["router"]
                experts = ExpertFF(int(ff["expert"]["ff"]), int(r["experts"]), int(r["top"]), float(r["scale"]))
            layers.append(BudoraxLayer(mixer, experts))
        lp, cap = d.get("loop"), d.get("logit_softcap")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers,
                   (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None, float(cap) if cap else None)

    @classmethod
    def from_json(cls, path: str) -> "BudoraxConfig":
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for e in self.layers:
            m, x = e.mixer, e.experts
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, DeltaMixer):
                mixer.update(kv_heads=m.kv_heads, conv=m.conv)
            elif isinstance(m, ChunkMixer):
                mixer.update(kv_heads=m.kv_heads, scale=m.scale, mask={"size": m.chunk}, rot={"dims": m.rot_dims, "base": m.rot_base}, diff=m.diff)
            else:
                mixer.update(rot_dim=m.rot_dim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale, rot={"dims": m.rot_dim, "base": m.rot_base})
            mlp = {"kind": "moe", "expert": {"ff": x.ff}, "router": {"experts": x.experts, "top": x.top, "scale": x.scale}} if x else None
            layers.append({"type": e.kind, "mixer": mixer, "mlp": mlp})
        d = {"architecture": "Budorax", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps}, "logit_softcap": self.softcap,
             "layers": layers}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d


_CONV = ("q", "k", "v")


def _norm_shapes(name: str, W: int) -> Dict[str, Tuple[int, ...]]:
    return {name: (W,), name + ".b": (W,), name + ".alpha": ()}


def _shapes(e: BudoraxLayer, W: int) -> Dict[str, Tuple[int, ...]]:
    """Tensor shapes of one layer (names without the layer's prefix)."""
    m, x = e.mixer, e.experts
    H, D, Dv = m.heads, m.dim, m.vdim
    if isinstance(m, DeltaMixer):
        qk, hv = m.kv_heads * D, H * Dv
        mix = {"q": (qk, W), "q.conv": (qk, m.conv), "k": (qk, W), "k.conv": (qk, m.conv), "v": (hv, W), "v.conv": (hv, m.conv), "b": (H, W),
               "A_log": (H,), "norm": (Dv,), "a": (H, W), "dt_bias": (H,), "g": (hv, W)}
    elif isinstance(m, ChunkMixer):
        mix = {"q": (2 * H * D, W), "k": (2 * m.kv_heads * D, W), "v": (m.kv_heads * Dv, W), "lq1": (D,), "lk1": (D,), "lq2": (D,), "lk2": (D,)}
    else:
        mix = {"dq": (m.q_rank, W), "dq.norm": (m.q_rank,), "uq": (H * (D + m.rot_dim), m.q_rank), "dkv": (m.kv_rank + m.rot_dim, W),
               "dkv.norm": (m.kv_rank,), "uk": (H * D, m.kv_rank), "uv": (H * Dv, m.kv_rank), "g": (H, W)}
    t = {"mix." + k: s for k, s in mix.items()}
    t["mix.o"] = (W, H * Dv)
    for n in ("norm1", "norm1b") + (("norm2", "norm2b") if x else ()):
        t.update(_norm_shapes(n, W))
    if x:
        for i in range(x.experts):
            t.update({f"mlp.e{i}.gate": (x.ff, W), f"mlp.e{i}.up": (x.ff, W), f"mlp.e{i}.down": (W, x.ff)})
        t.update({"mlp.router": (x.experts, W), "mlp.correction": (x.experts,)})
    return t


class BudoraxWeights:
    """Weights by the names of the checkpoint, layer by layer (prefix dropped); :class:`PagedBudorax` packs what its passes read."""

    def __init__(self, cfg: BudoraxConfig):
        self.cfg = cfg
        self.embed: Optional[torch.Tensor] = None
        self.final: Dict[str, torch.Tensor] = {}
        self.layers: List[Dict[str, torch.Tensor]] = []

    @classmethod
    def from_state_dict(cls, cfg: BudoraxConfig, sd: Dict[str, torch.Tensor]) -> "BudoraxWeights":
        w, W = cls(cfg), cfg.hidden_size

        def take(name, shape):
            if tuple(sd[name].shape) != shape:
                raise ValueError(f"{name} has shape {tuple(sd[name].shape)}, the configuration asks for {shape}")
            return sd[name]
        w.embed = take("embed", (cfg.vocab_size, W))
        w.final = {k: take("final." + k, s) for k, s in _norm_shapes("norm", W).items()}
        for i, e in enumerate(cfg.layers):
            w.layers.append({k: take(f"l{i}.{k}", s) for k, s in _shapes(e, W).items()})
        return w

    def state_dict(self) -> Dict[str, torch.Tensor]:
        sd = {"embed": self.embed, **{"final." + k: t for k, t in self.final.items()}}
        sd.update({f"l{i}.{k}": t for i, L in enumerate(self.layers) for k, t in L.items()})
        return sd

    @classmethod
    def random(cls, cfg: BudoraxConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> "BudoraxWeights":
        """Random weights of the right scales (benchmarks and tests), drawn on ``device``."""
        g = torch.Generator(device=device).manual_seed(seed)

        def r(*s, scale=1.0, at=0.0):
            return (at + torch.randn(s, generator=g, device=device) * scale).to(dtype)

        def one(name, s):
            if name.endswith(".alpha"):
                return r(scale=0.1, at=0.7)
            if len(s) == 2:
                return r(*s, scale=s[1] ** -0.5)
            if ".norm" in name or name.startswith("norm"):
                return r(*s, scale=0.1, at=0.0 if name.endswith(".b") else 1.0)
            return r(*s, scale=0.5, at=-4.0) if name.endswith("dt_bias") else r(*s, scale=0.1)
        w, W = cls(cfg), cfg.hidden_size
        w.embed = r(cfg.vocab_size, W)
        w.final = {k: one(k, s) for k, s in _norm_shapes("norm", W).items()}
        w.layers = [{k: one(k, s) for k, s in _shapes(e, W).items()} for e in cfg.layers]
        return w

    def num_parameters(self) -> int:
        return sum(t.numel() for t in self.state_dict().values())

    def to(self, device, dtype) -> "BudoraxWeights":
        """Matrices in ``dtype``; vectors, numbers and convolution taps, which enter fp32 arithmetic, in fp32."""
        w = BudoraxWeights(self.cfg)
        mv = lambda t, exact=False: t.to(device=device, dtype=torch.float32 if exact or t.dim() < 2 else dtype).contiguous()
        w.embed, w.final = mv(self.embed), {k: mv(t) for k, t in self.final.items()}
        w.layers = [{k: mv(t, k.endswith(".conv")) for k, t in L.items()} for L in self.layers]
        return w


class PagedBudorax(PagedModel):
    architecture = "budorax"
    continues_prompts = True

    def __init__(self, weights: BudoraxWeights, device, dtype):
        super().__init__(weights, device, dtype)
        c, w = self.cfg, self.weights
        norm = lambda L, name: T.TanhNorm(float(L[name + ".alpha"]), L[name], L[name + ".b"])
        self.final = norm(w.final, "norm")
        self.head = RowPack.pad(w.embed)
        rotary: Dict[tuple, Rotary] = {}

        def rot(dims, base):
            if (dims, base) not in rotary:
                rotary[dims, base] = Rotary(dims, base, c.max_position_embeddings, device)
            return rotary[dims, base]
        self.prep: List[dict] = []
        for e, L in zip(c.layers, w.layers):
            m, x = e.mixer, e.experts
            mix = {k[4:]: t for k, t in L.items() if k.startswith("mix.")}
            d = dict(kind=e.kind, norm1=norm(L, "norm1"), norm1b=norm(L, "norm1b"), o=mix["o"])
            if isinstance(m, DeltaMixer):
                d["pack"] = RowPack({"conv": sum(mix[n].shape[0] for n in _CONV), "b": m.heads, "a": m.heads, "g": m.heads * m.vdim})
                d["w_in"] = d["pack"].pack({"conv": torch.cat([mix[n] for n in _CONV]), "b": mix["b"], "a": mix["a"], "g": mix["g"]})
                d["conv"] = torch.cat([mix[n + ".conv"] for n in _CONV]).t().contiguous()            # [taps, channels]
                d["delta"] = R.DeltaRule(m.heads, m.kv_heads, m.dim, m.vdim, mix["A_log"].exp(), mix["dt_bias"], head_decay=True)
                d["norm"] = mix["norm"]
            elif isinstance(m, ChunkMixer):
                d["pack"] = RowPack({n: mix[n].shape[0] for n in "qkv"})
                d["w_in"] = d["pack"].pack({n: mix[n] for n in "qkv"})
                lam = torch.exp((mix["lq1"] * mix["lk1"]).sum()) - torch.exp((mix["lq2"] * mix["lk2"]).sum()) + m.diff
                d["attn"] = A.WindowAttention(m.heads, m.kv_heads, m.dim, m.vdim, min(m.chunk, A.UNBOUNDED), 0, m.scale, chunked=True, maps=2,
                                              mix=float(lam), mix_gain=1 - m.diff, mix_eps=c.eps)
                d["rot"] = rot(m.rot_dims, m.rot_base)
            else:
                d["pack"] = RowPack({"dq": m.q_rank, "dkv": m.kv_rank + m.rot_dim, "g": m.heads})
                d["w_in"] = d["pack"].pack({n: mix[n] for n in ("dq", "dkv", "g")})
                d["uq"] = RowPack.pad(mix["uq"])
                d["latent"] = M.LatentAttention.of(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, mix["uk"], mix["uv"], rot(m.rot_dim, m.rot_base))
                d["q_norm"], d["kv_norm"] = mix["dq.norm"], mix["dkv.norm"]
            if x:
                d["norm2"], d["norm2b"] = norm(L, "norm2"), norm(L, "norm2b")
                parts = lambda n: [L[f"mlp.e{i}.{n}"] for i in range(x.experts)]
                d["experts"] = X.Experts.of(parts("gate"), parts("up"), parts("down"), L["mlp.router"], L["mlp.correction"], x.top, x.scale)
                for k in [k for k in L if k.startswith("mlp.e")]:
                    L[k] = L[k][:0]                        # the packed copy is what runs
            self.prep.append(d)
        self.runs = [(self.prep[i], again) for i, again in c.runs()]
        self.rewinds = not any(d["kind"] == "delta" for d, _ in self.runs)      # a recurrent state cannot give a token back
        count = weights.num_parameters()
        w.layers = [{k: t for k, t in L.items() if t.dim() < 2} for L in w.layers]
        w.num_parameters = lambda: count

    # ---- what the cache holds: every layer run has entries of its own
    def kv_shapes(self):
        out = []
        for d, _ in self.runs:
            a = d.get("attn")
            out.append((a.kv_heads, a.key_stored, a.vdim_stored) if a else (1, d["latent"].row, 0) if "latent" in d else (0, 0, 0))
        return out

    def state_shapes(self):
        out = []
        for d, _ in self.runs:
            r = d.get("delta")
            out.append({"S": ((r.heads, r.dim, r.vdim), torch.float32), "conv": ((d["conv"].shape[0] - 1, d["conv"].shape[1]), self.dtype)} if r else {})
        return out

    def cache_window(self):
        if any("latent" in d for d, _ in self.runs):
            return None
        return max((d["attn"].window for d, _ in self.runs if "attn" in d), default=1)

    def pick_splits(self, rows: int, max_len: int) -> int:
        """Keys that the splits of every layer have to cover, in units of 32: a power of two, so that it changes rarely."""
        units = 1
        while units * 32 < max_len:
            units *= 2
        return units

    # ---- the passes
    def _delta(self, d, h, l, kv, pos, req, seqs):
        from ..ops.gemm import linear
        pk = d["pack"]
        p = linear(h, d["w_in"])
        c = R.short_conv(pk.cols(p, "conv"), d["conv"], kv.state[l]["conv"], pos, req, seqs)
        o = R.delta_rule(c, d["delta"], pk.cols(p, "b"), pk.cols(p, "a"), kv.state[l]["S"], pos, req, seqs)
        return R.group_norm_gate(o, d["norm"], pk.cols(p, "g"), self.cfg.eps, self.dtype, act="silu")

    def _attention(self, d, h, l, kv, page_table, pos, req, attend):
        from ..ops.gemm import linear
        a, at = d["attn"], d["pack"].at
        q = A.rope_write(linear(h, d["w_in"]), (at["q"], at["k"], at["v"]), a, d["rot"], pos, req, page_table, kv.k[l], kv.v[l])
        return attend(a, q, kv.k[l], kv.v[l])

    def _latent(self, d, h, l, kv, page_table, pos, req, attend):
        from ..ops.gemm import linear
        a, pk = d["latent"], d["pack"]
        p = linear(h, d["w_in"])
        c = M.latent_write(p, (pk.at["dq"], pk.at["dkv"]), a, d["q_norm"], d["kv_norm"], self.cfg.eps, pos, req, page_table, kv.k[l])
        return attend(a, linear(c, d["uq"]), kv.k[l], pk.cols(p, "g"))

    def _layers(self, ids, kv, page_table, pos, req, seqs, attend, attend_latent, last: Optional[T.TanhNorm]):
        """``attend`` / ``attend_latent``: the attentions over the pages once this pass's keys are in them.  Returns the fp32 stream
        and, with ``last``, its norm."""
        embed = self.weights.embed
        x, _ = S.embed_residual(ids, embed, copy=False)
        steps = [(l, d, again and w == "norm1", w) for l, (d, again) in enumerate(self.runs) for w in ("norm1", "norm2") if w in d]
        first = steps[0][1][steps[0][3]] if steps else last
        h = T.rows(x, first, dtype=self.dtype) if first is not None else None
        for i, (l, d, _, which) in enumerate(steps):
            _, nd, again, nw = steps[i + 1] if i + 1 < len(steps) else (0, {"last": last}, False, "last")
            if which == "norm2":
                y = X.run(h, d["experts"])
            else:
                if d["kind"] == "delta":
                    o = self._delta(d, h, l, kv, pos, req, seqs)
                elif d["kind"] == "attention":
                    o = self._attention(d, h, l, kv, page_table, pos, req, attend)
                else:
                    o = self._latent(d, h, l, kv, page_table, pos, req, attend_latent)
                y = S.linear_branch(o, d["o"])
            h = T.residual(x, y, d[which + "b"], nd[nw], dtype=self.dtype, again=(ids, embed) if again else None)
        return x, h

    def _logits(self, h):
        z = S.linear_f32(h, self.head)[:, :self.cfg.vocab_size]
        return T.softcap(z, self.cfg.softcap) if self.cfg.softcap else z

    def prompt_pass(self, kv, page_table, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        top = max(at + n for at, n in zip(batch.starts, batch.lens()))
        seqs = R.Sequences.of(batch.offs, batch.starts, batch.rows, self.device)
        tiles = A.PromptTiles.of(batch.offs, batch.starts, batch.rows, self.device) if batch.offs[-1] >= A.TILES_FROM else None
        context: List[M.PromptContext] = []

        def attend(a, q, k, v):
            if tiles is not None and A.tiles_supported(q, a):
                return A.window_attention_tiles(q, a, tiles, page_table, k, v)
            ns = A.pick_splits(q.shape[0], a.kv_heads, a.most_keys(top))
            return A.window_attention(q, a, batch.pos, batch.req, page_table, k, v, ns, top)

        def attend_latent(a, q, pages, gate):
            if M.tiles_pay(q, a, batch.offs[-1]):
                if not context:
                    context.append(M.PromptContext.of(batch.offs, batch.starts, batch.rows, self.device))
                return M.latent_attention_tiles(q, a, context[0], batch.pos, page_table, pages, gate)
            return M.latent_attention(q, a, batch.pos, batch.req, page_table, pages, top, gate)
        x, _ = self._layers(batch.ids, kv, page_table, batch.pos, batch.req, seqs, attend, attend_latent, None)
        if hidden:
            return T.rows(x, self.final, dtype=self.dtype)
        return self._logits(T.rows(x, self.final, index=batch.want, dtype=self.dtype))

    def decode_pass(self, kv, page_table, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        ids, pos, req = meta[:, 0], meta[:, 1], meta[:, 2]
        cover = nsplit * 32

        def attend(a, q, k, v):
            keys = a.most_keys(cover)
            return A.window_attention(q, a, pos, req, page_table, k, v, A.pick_splits(q.shape[0], a.kv_heads, keys), cover)

        def attend_latent(a, q, pages, gate):
            return M.latent_attention(q, a, pos, req, page_table, pages, cover, gate)
        _, h = self._layers(ids, kv, page_table, pos, req, None, attend, attend_latent, self.final)
        return self._logits(h)


register_model(BudoraxConfig, BudoraxWeights, PagedBudorax, "budorax")
