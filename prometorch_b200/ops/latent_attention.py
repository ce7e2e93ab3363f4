"""Latent attention over the paged cache: a token keeps one RMS-normed latent c and one rotated key part that all heads share; a
head's unrotated key is ``W_uk c``, its value ``W_uv c`` (csrc/latent_attn.cu, csrc/window_attn_sm100.cu).

A cache row is ``[c, rotated part]``, each padded to a multiple of 16.  Two ways through it:

* few query rows (:func:`latent_attention`): ``W_uk`` is folded into the query, so that every head reads the cached rows as they are,
  both as keys and as values, and ``W_uv`` is applied to the weighted latent;
* prompts (:func:`latent_attention_tiles`): keys and values of the whole context are formed once per pass and go through the
  tensor-core tiles.

CUDA tensors run the kernels, CPU tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .. import _native as N
from . import window_attention as A
from .paged import PAGE, _status
from .rotary import Rotary


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_latent_write.argtypes = [vp, ll, ci, ci, ci, ci, ci, vp, vp, cf, vp, vp, ci, vp, vp, ci, ci, vp, ci, vp, ci, vp, ci, ci, ci, vp, ci, vp]
    L.ptb_head_linear.argtypes = [vp, ll, ci, vp, ci, ci, ci, vp, ll, ci, ci, vp, ll, ci, ci, vp, vp, ci, vp, ci, vp, ci, vp]
    for n in ("ptb_latent_write", "ptb_head_linear"):
        getattr(L, n).restype = ci


@dataclass
class LatentAttention:
    heads: int
    dim: int                           # unrotated query / key size per head
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    absorb: torch.Tensor               # [H, rank, dim]: W_uk, transposed per head
    expand: torch.Tensor               # [H, vdim, stored rank]: W_uv
    prompt: torch.Tensor               # [H stored dim + H stored vdim, stored rank]: W_uk, then W_uv, heads padded to 16 rows
    rotary: Rotary

    @classmethod
    def of(cls, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float, uk: torch.Tensor, uv: torch.Tensor, rotary: Rotary) -> "LatentAttention":
        k, v = uk.view(heads, dim, rank), uv.view(heads, vdim, rank)
        more = A.stored(rank) - rank
        pad = lambda t, size: torch.nn.functional.pad(t, (0, more, 0, A.stored(size) - size)).reshape(-1, rank + more)
        return cls(heads, dim, rot_dim, vdim, rank, scale, k.transpose(1, 2).contiguous(), torch.nn.functional.pad(v, (0, more)).contiguous(),
                   torch.cat([pad(k, dim), pad(v, vdim)]).contiguous(), rotary)

    @property
    def rank_stored(self) -> int:
        return A.stored(self.rank)

    @property
    def row(self) -> int:
        """Elements of a cache row."""
        return A.stored(self.rank) + A.stored(self.rot_dim)


def latent_write(p: torch.Tensor, cols: Tuple[int, int], a: LatentAttention, q_weight: torch.Tensor, kv_weight: torch.Tensor, eps: float, pos: torch.Tensor,
                 req: torch.Tensor, page_table: torch.Tensor, pages: torch.Tensor) -> torch.Tensor:
    """``p [n, *]``: a packed projection with the queries' latent and the keys' (latent, then the shared key part) at the columns
    ``cols``.  Returns the queries' latent after its RMS norm ``[n, q rank]``; the normed key latent and the rotated part go to the page
    slot of ``(req[i], pos[i])``."""
    n, qr = p.shape[0], q_weight.shape[0]
    out = torch.empty(n, qr, dtype=p.dtype, device=p.device)
    if p.is_cuda:
        assert p.stride(1) == 1 and pos.dtype == req.dtype == page_table.dtype == torch.int32 and p.dtype in (torch.bfloat16, torch.float32)
        N.check(N.lib().ptb_latent_write(p.data_ptr(), p.stride(0), *cols, qr, a.rank, a.rot_dim, q_weight.data_ptr(), kv_weight.data_ptr(), float(eps),
                                         N.ptr(a.rotary.cos), N.ptr(a.rotary.sin), a.rotary.positions, out.data_ptr(), pages.data_ptr(), a.rank_stored, a.row,
                                         pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0), page_table.data_ptr(), page_table.stride(0), pages.shape[0], n,
                                         _status(p.device).data_ptr(), int(p.dtype == torch.bfloat16), torch.cuda.current_stream(p.device).cuda_stream), "latent_write")
        return out
    x = p.float()
    norm = lambda t, w: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
    out.copy_(norm(x[:, cols[0]:cols[0] + qr], q_weight))
    c = norm(x[:, cols[1]:cols[1] + a.rank], kv_weight)
    rot = a.rotary.apply(x[:, cols[1] + a.rank:cols[1] + a.rank + a.rot_dim][:, None], pos)[:, 0]
    wide = lambda t: torch.nn.functional.pad(t, (0, A.stored(t.shape[1]) - t.shape[1]))
    at = pos.long()
    pages[page_table[req.long(), at // PAGE].long(), 0, at % PAGE] = torch.cat([wide(c), wide(rot)], -1).to(pages.dtype)
    return out


def _st(t):
    return torch.cuda.current_stream(t.device).cuda_stream


def fold_queries(q: torch.Tensor, a: LatentAttention, pos: torch.Tensor) -> torch.Tensor:
    """``q [n, >= H (dim + rot_dim)]`` as projected -> ``[n, H, row]``: ``W_uk^T q`` beside the rotated part, padded like a cache row."""
    n, H, D, r = q.shape[0], a.heads, a.dim, a.rot_dim
    out = torch.empty(n, H, a.row, dtype=q.dtype, device=q.device)
    N.check(N.lib().ptb_head_linear(q.data_ptr(), q.stride(0), D + r, a.absorb.data_ptr(), H, a.rank, D, out.data_ptr(), H * a.row, a.row, n, 0, 0, a.rank_stored, r,
                                    N.ptr(a.rotary.cos), N.ptr(a.rotary.sin), a.rotary.positions, pos.data_ptr(), pos.stride(0), _status(q.device).data_ptr(),
                                    int(q.dtype == torch.bfloat16), _st(q)), "head_linear")
    return out


def unfold_values(o: torch.Tensor, a: LatentAttention, gate: Optional[torch.Tensor]) -> torch.Tensor:
    """``o [n, H, stored rank]`` weighted latents -> ``[n, H vdim]``: ``W_uv`` per head, times the sigmoid of ``gate [n, H]``."""
    n, H = o.shape[0], a.heads
    out = torch.empty(n, H * a.vdim, dtype=o.dtype, device=o.device)
    N.check(N.lib().ptb_head_linear(o.data_ptr(), o.stride(0), a.rank_stored, a.expand.data_ptr(), H, a.vdim, a.rank_stored, out.data_ptr(), H * a.vdim, a.vdim, n,
                                    N.ptr(gate), gate.stride(0) if gate is not None else 0, 0, 0, 0, 0, 0, 0, 0, _status(o.device).data_ptr(),
                                    int(o.dtype == torch.bfloat16), _st(o)), "head_linear")
    return out


HEADS_PER_CTA = 32                     # of the row kernels


def latent_attention(q: torch.Tensor, a: LatentAttention, pos: torch.Tensor, req: torch.Tensor, page_table: torch.Tensor, pages: torch.Tensor,
                     max_len: int, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rows ``q [n, >= H (dim + rot_dim)]`` (as projected) at ``pos`` against the cached rows of their sequences, their own included;
    ``max_len``: no row's position is at or past it.  Returns ``[n, H vdim]``."""
    if not q.is_cuda:
        return latent_attention_reference(q, a, pos, req, page_table, pages, gate)
    n, H = q.shape[0], a.heads
    qs = fold_queries(q, a, pos)
    o = torch.empty(n, H, a.rank_stored, dtype=q.dtype, device=q.device)
    args = A.WindowArgs(k_pages=pages.data_ptr(), v_pages=pages.data_ptr(), page_table=page_table.data_ptr(), pt_stride=page_table.stride(0), n_pages=pages.shape[0],
                        H=H, G=1, D=a.row, Dp=a.row, Dv=a.rank_stored, Dvp=a.rank_stored, v_ld=a.row, maps=1, window=A.UNBOUNDED, keep=0, chunked=0,
                        scale=float(a.scale), bf16=int(q.dtype == torch.bfloat16), status=_status(q.device).data_ptr(), max_keys=max(1, max_len))
    A.run_rows(args, qs, o, pos, req, A.pick_splits(n, -(-H // HEADS_PER_CTA), max_len))
    return unfold_values(o, a, gate)


@dataclass
class PromptContext:
    """Where the context of every sequence of a prompt pass lies in the flat keys and values of that pass."""
    tiles: A.PromptTiles
    rows: int

    @classmethod
    def of(cls, offs: List[int], starts: List[int], rows: List[int], device) -> "PromptContext":
        raise NotImplementedError


def tiles_pay(q: torch.Tensor, a: LatentAttention, rows: int, max_len: int) -> bool:
    return False


def latent_attention_tiles(q, a, context, pos, page_table, pages, gate):
    raise NotImplementedError


def latent_attention_reference(q, a: LatentAttention, pos, req, page_table, pages, gate=None) -> torch.Tensor:
    """The same in plain fp32 math, sequence by sequence (CPU path)."""
    n, H, D, r = q.shape[0], a.heads, a.dim, a.rot_dim
    x = q[:, :H * (D + r)].float().reshape(n, H, D + r)
    x = torch.cat([torch.einsum("nhd,hrd->nhr", x[..., :D], a.absorb.float()), a.rotary.apply(x[..., D:], pos)], -1)
    out = torch.zeros(n, H, a.vdim)
    for s in torch.unique(req).tolist():
        rows = (req == s).nonzero()[:, 0]
        p = pos[rows].long()
        j = torch.arange(int(p.max()) + 1)
        k = pages[page_table[s, j // PAGE].long(), 0, j % PAGE].float()
        k = torch.cat([k[:, :a.rank], k[:, a.rank_stored:a.rank_stored + r]], -1)
        w = (torch.einsum("nhd,jd->hnj", x[rows], k) * a.scale).masked_fill(j[None, :] > p[:, None], float("-inf"))
        o = torch.einsum("hnj,jr->nhr", torch.softmax(w, -1), k[:, :a.rank])
        out[rows] = torch.einsum("nhr,hvr->nhv", o, a.expand[..., :a.rank].float())
    if gate is not None:
        out *= torch.sigmoid(gate.float())[..., None]
    return out.reshape(n, H * a.vdim).to(q.dtype)
