"""Llama for the batching engine: configuration and weights of a Hugging Face directory, prompt and decode pass over the paged
cache (rotary + page write, FlashAttention over the prompt, page-table attention, fused residual + RMSNorm)."""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

from ..ops import paged as P
from .paged import PagedModel, PromptBatch, register_model


@dataclass
class LlamaConfig:
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 32
    max_position_embeddings: int = 4096
    rms_norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    bos_token_id: int = 1
    eos_token_id: int = 2
    tie_word_embeddings: bool = False

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_attention_heads

    @classmethod
    def from_json(cls, path: str) -> "LlamaConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))

    @classmethod
    def from_dict(cls, d: dict) -> "LlamaConfig":
        c = cls()
        for k in cls.__dataclass_fields__:
            if k in d and d[k] is not None:
                v = d[k]
                if k == "eos_token_id" and isinstance(v, list):
                    v = v[0]
                setattr(c, k, type(getattr(c, k))(v))
        if "num_key_value_heads" not in d:
            c.num_key_value_heads = c.num_attention_heads
        return c


class LlamaWeights:
    """Weights in the layout the engine runs: q/k/v packed into one matrix, gate/up packed into one."""

    def __init__(self, cfg: LlamaConfig):
        self.cfg = cfg
        self.tok_emb: Optional[torch.Tensor] = None
        self.layers: List[Dict[str, torch.Tensor]] = []
        self.final_norm: Optional[torch.Tensor] = None
        self.lm_head: Optional[torch.Tensor] = None

    @classmethod
    def random(cls, cfg: LlamaConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> "LlamaWeights":
        """Random weights of the right scales (benchmarks and tests); drawn on ``device`` so a large model never sits in
        host memory."""
        g = torch.Generator(device=device).manual_seed(seed)
        D, I, H, Hk, Dh = cfg.hidden_size, cfg.intermediate_size, cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim

        def r(*s, scale):
            return (torch.randn(*s, generator=g, device=device) * scale).to(dtype)

        def norm_w():
            return (1 + 0.1 * torch.randn(D, generator=g, device=device)).to(dtype)
        w = cls(cfg)
        w.tok_emb = r(cfg.vocab_size, D, scale=1.0)
        for _ in range(cfg.num_hidden_layers):
            w.layers.append(dict(attn_norm=norm_w(), wqkv=r((H + 2 * Hk) * Dh, D, scale=D ** -0.5), wo=r(D, H * Dh, scale=(H * Dh) ** -0.5),
                                 ffn_norm=norm_w(), w_gate_up=r(2 * I, D, scale=D ** -0.5), w_down=r(D, I, scale=I ** -0.5)))
        w.final_norm = norm_w()
        w.lm_head = r(cfg.vocab_size, D, scale=D ** -0.5)
        return w

    @classmethod
    def from_state_dict(cls, cfg: LlamaConfig, sd: Dict[str, torch.Tensor]) -> "LlamaWeights":
        """Hugging Face names: ``model.layers.N.self_attn.{q,k,v,o}_proj.weight`` and so on."""
        w = cls(cfg)
        if "embed_tokens.weight" in sd and "model.embed_tokens.weight" not in sd:          # a bare LlamaModel checkpoint
            sd = {("model." + k if not k.startswith("lm_head") else k): v for k, v in sd.items()}
        w.tok_emb = sd["model.embed_tokens.weight"]
        for l in range(cfg.num_hidden_layers):
            p = f"model.layers.{l}."
            w.layers.append(dict(
                attn_norm=sd[p + "input_layernorm.weight"],
                wqkv=torch.cat([sd[p + "self_attn.q_proj.weight"], sd[p + "self_attn.k_proj.weight"], sd[p + "self_attn.v_proj.weight"]]),
                wo=sd[p + "self_attn.o_proj.weight"], ffn_norm=sd[p + "post_attention_layernorm.weight"],
                w_gate_up=torch.cat([sd[p + "mlp.gate_proj.weight"], sd[p + "mlp.up_proj.weight"]]), w_down=sd[p + "mlp.down_proj.weight"]))
        w.final_norm = sd["model.norm.weight"]
        w.lm_head = sd.get("lm_head.weight", w.tok_emb)
        return w

    def state_dict(self) -> Dict[str, torch.Tensor]:
        c = self.cfg
        H, Hk, Dh, I = c.num_attention_heads, c.num_key_value_heads, c.head_dim, c.intermediate_size
        sd = {"model.embed_tokens.weight": self.tok_emb, "model.norm.weight": self.final_norm, "lm_head.weight": self.lm_head}
        for l, L in enumerate(self.layers):
            p = f"model.layers.{l}."
            q, k, v = L["wqkv"].split([H * Dh, Hk * Dh, Hk * Dh])
            g, u = L["w_gate_up"].split([I, I])
            sd.update({p + "input_layernorm.weight": L["attn_norm"], p + "self_attn.q_proj.weight": q, p + "self_attn.k_proj.weight": k,
                       p + "self_attn.v_proj.weight": v, p + "self_attn.o_proj.weight": L["wo"],
                       p + "post_attention_layernorm.weight": L["ffn_norm"], p + "mlp.gate_proj.weight": g,
                       p + "mlp.up_proj.weight": u, p + "mlp.down_proj.weight": L["w_down"]})
        return sd

    def num_parameters(self) -> int:
        return sum(t.numel() for L in self.layers for t in L.values()) + self.tok_emb.numel()

    def to(self, device, dtype) -> "LlamaWeights":
        w = LlamaWeights(self.cfg)
        mv = lambda t: t.to(device=device, dtype=dtype).contiguous()
        w.tok_emb, w.final_norm, w.lm_head = mv(self.tok_emb), mv(self.final_norm), mv(self.lm_head)
        w.layers = [{k: mv(v) for k, v in L.items()} for L in self.layers]
        return w


class PagedLlama(PagedModel):
    architecture = "llama"

    def __init__(self, weights: LlamaWeights, device, dtype):
        super().__init__(weights, device, dtype)
        c = self.cfg
        self.cos, self.sin = P.rope_tables(c.max_position_embeddings, c.head_dim, c.rope_theta, device)

    def kv_shapes(self):
        c = self.cfg
        return [(c.num_key_value_heads, c.head_dim, c.head_dim)] * c.num_hidden_layers

    def pick_splits(self, rows: int, max_len: int) -> int:
        return P.pick_splits(rows, self.cfg.num_key_value_heads, max_len)

    def _linear(self, x, w):
        if x.is_cuda:
            from ..ops.gemm import linear
            return linear(x, w)
        return F.linear(x, w)

    def _norm(self, x, w):
        from ..ops.fused_ops import rms_norm
        return rms_norm(x, w, self.cfg.rms_norm_eps)

    def _mlp(self, x, L):
        from ..ops.fused_ops import swiglu
        return self._linear(swiglu(self._linear(x, L["w_gate_up"])), L["w_down"])

    def prompt_pass(self, kv, page_table, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        """Attention runs per request over the prompt's own keys (requests of equal length share a call)."""
        from ..ops.attention import flash_attention
        if any(batch.starts):
            raise ValueError("the Llama prompt pass starts at position 0")
        c, w = self.cfg, self.weights
        H, Hk, Dh = c.num_attention_heads, c.num_key_value_heads, c.head_dim
        groups: Dict[int, List[int]] = {}
        for i, n in enumerate(batch.lens()):
            groups.setdefault(n, []).append(i)
        consecutive = all(g == list(range(g[0], g[0] + len(g))) for g in groups.values())
        x = w.tok_emb[batch.ids.long()]
        for l, L in enumerate(w.layers):
            qkv = self._linear(self._norm(x, L["attn_norm"]), L["wqkv"]).contiguous()
            k = P.paged_rope_write(qkv, H, Hk, Dh, batch.pos, batch.req, page_table, self.cos, self.sin, kv.k[l], kv.v[l], want_k=True)
            a = torch.empty(qkv.shape[0], H * Dh, dtype=qkv.dtype, device=x.device)
            for n, members in groups.items():
                runs = [members] if consecutive else [[i] for i in members]      # equal lengths side by side: one call
                for run in runs:
                    lo, hi, nb = batch.offs[run[0]], batch.offs[run[-1] + 1], len(run)
                    q = qkv[lo:hi, :H * Dh].reshape(nb, n, H, Dh)
                    v = qkv[lo:hi, (H + Hk) * Dh:].reshape(nb, n, Hk, Dh)
                    a[lo:hi] = flash_attention(q, k[lo:hi].view(nb, n, Hk, Dh), v, causal=True).reshape(nb * n, H * Dh)
            x = x + self._linear(a, L["wo"])
            x = x + self._mlp(self._norm(x, L["ffn_norm"]), L)
        if hidden:                                             # the embedding path: every position after the final norm
            return self._norm(x, w.final_norm)
        return self._linear(self._norm(x[batch.want], w.final_norm), w.lm_head).float()

    def decode_pass(self, kv, page_table, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        from ..ops.gemm import linear_add_rms_norm, linear_swiglu
        c, w = self.cfg, self.weights
        H, Hk, Dh = c.num_attention_heads, c.num_key_value_heads, c.head_dim
        B = meta.shape[0]
        ids, pos, rows, lens = meta[:, 0].long(), meta[:, 1].contiguous(), meta[:, 2].long(), meta[:, 3].contiguous()
        table = page_table[rows]                          # [B, pt_stride] rows in batch order
        req = torch.arange(B, dtype=torch.int32, device=meta.device)
        x = w.tok_emb[ids]
        h = self._norm(x, w.layers[0]["attn_norm"])
        for l, L in enumerate(w.layers):
            q = P.qkv_rope_write(h, L["wqkv"], H, Hk, Dh, pos, req, table, self.cos, self.sin, kv.k[l], kv.v[l])
            a = P.paged_attention_decode(q, H, Hk, Dh, lens, table, kv.k[l], kv.v[l], nsplit=nsplit)
            h, x = linear_add_rms_norm(a, L["wo"], x, L["ffn_norm"], c.rms_norm_eps)
            nxt = w.layers[l + 1]["attn_norm"] if l + 1 < len(w.layers) else w.final_norm
            h, x = linear_add_rms_norm(linear_swiglu(h, L["w_gate_up"]), L["w_down"], x, nxt, c.rms_norm_eps)
        return self._linear(h, w.lm_head).float()


register_model(LlamaConfig, LlamaWeights, PagedLlama, "llama", "LlamaForCausalLM", "LlamaModel")
