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
    L.ptb_latent_gather.argtypes = [vp, ci, ci, vp, ci, ci, vp, ci, vp, ci, vp, vp]
    L.ptb_latent_q.argtypes = [vp, ll, vp, ci, ci, ci, ci, ci, vp, vp, ci, ci, vp, ci, vp, vp]
    L.ptb_latent_attn_rows.argtypes = [C.POINTER(A.WindowArgs), vp]
    for n in ("ptb_latent_write", "ptb_head_linear", "ptb_latent_gather", "ptb_latent_q", "ptb_latent_attn_rows"):
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


def _runs_mma(q: torch.Tensor, a: LatentAttention) -> bool:
    """Whether the kernel of csrc/latent_attn.cu takes these rows: latents up to 512 and their shared part fit its registers and rings."""
    return q.dtype == torch.bfloat16 and a.rank_stored <= 512 and a.row <= 640


def pick_splits(rows: int, heads: int, keys: int, sms: int = 148) -> int:
    """CTAs that share a row's keys in the tensor-core kernel, which walks any number of pages: as many as fill the machine once."""
    return max(1, min(-(-keys // PAGE), sms // max(1, rows * -(-heads // HEADS_PER_CTA))))


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
    if _runs_mma(q, a):
        A.run_rows(args, qs, o, pos, req, pick_splits(n, H, max_len), kernel=N.lib().ptb_latent_attn_rows)
    else:
        splits = A.pick_splits(n, -(-H // HEADS_PER_CTA), max_len)
        if q.dtype == torch.bfloat16 and a.rank_stored > 512:                # a CTA's values have to fit its shared memory
            splits = max(splits, -(-max_len // 32))
        A.run_rows(args, qs, o, pos, req, splits)
    return unfold_values(o, a, gate)


@dataclass
class PromptContext:
    """The context of the sequences of a prompt pass, cached tokens included, laid out one after the other: the pages it comes from
    (``[pieces, 4]`` int32: first row, row of the page table, page of the sequence, rows) and the query tiles with the first row of their
    sequence's context."""
    rows: int
    pieces: torch.Tensor
    tiles: torch.Tensor

    @classmethod
    def of(cls, offs: List[int], starts: List[int], rows: List[int], device) -> "PromptContext":
        pieces, tiles, base = [], [], 0
        for lo, hi, at, r in zip(offs, offs[1:], starts, rows):
            total = at + hi - lo
            pieces += [(base + j, r, j // PAGE, min(PAGE, total - j)) for j in range(0, total, PAGE)]
            tiles += [(lo + i, at + i, min(A.QUERY_TILE, hi - lo - i), base) for i in range(0, hi - lo, A.QUERY_TILE)]
            base += total
        tiles.sort(key=lambda t: -t[1])
        up = lambda t: torch.tensor(t, dtype=torch.int32).to(device)
        return cls(base, up(pieces), up(tiles))


TILES_FROM = 32                        # rows of a prompt pass from which keys and values are formed


def tiles_supported(a: LatentAttention) -> bool:
    return A.stored(a.dim) <= 128 and A.stored(a.rot_dim) <= 64 and A.stored(a.vdim) <= 128


def tiles_pay(q: torch.Tensor, a: LatentAttention, rows: int) -> bool:
    return q.is_cuda and q.dtype == torch.bfloat16 and rows >= TILES_FROM and tiles_supported(a)


def latent_attention_tiles(q: torch.Tensor, a: LatentAttention, context: PromptContext, pos: torch.Tensor, page_table: torch.Tensor, pages: torch.Tensor,
                           gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """A prompt pass's rows ``q [n, >= H (dim + rot_dim)]`` (as projected) against the whole context of their sequences, on tcgen05."""
    from .gemm import linear
    n, H, status = q.shape[0], a.heads, _status(q.device).data_ptr()
    flat = torch.empty(context.rows, a.row, dtype=q.dtype, device=q.device)
    N.check(N.lib().ptb_latent_gather(pages.data_ptr(), pages.shape[0], a.row, page_table.data_ptr(), page_table.stride(0), page_table.shape[0], context.pieces.data_ptr(),
                                      context.pieces.shape[0], flat.data_ptr(), context.rows, status, _st(q)), "latent_gather")
    kv = linear(flat[:, :a.rank_stored], a.prompt)
    Dp, Dvp, Rp = A.stored(a.dim), A.stored(a.vdim), A.stored(a.rot_dim)
    Do = -(-Dp // 64) * 64
    qs = torch.empty(n, H, Do + Rp, dtype=q.dtype, device=q.device)
    N.check(N.lib().ptb_latent_q(q.data_ptr(), q.stride(0), qs.data_ptr(), n, H, a.dim, Do, Rp, N.ptr(a.rotary.cos), N.ptr(a.rotary.sin), a.rot_dim, a.rotary.positions,
                                 pos.data_ptr(), pos.stride(0), status, _st(q)), "latent_q")
    out = torch.empty(n, H * a.vdim, dtype=q.dtype, device=q.device)
    args = A.WindowArgs(q=qs.data_ptr(), out=out.data_ptr(), k_pages=kv.data_ptr(), v_pages=kv[:, H * Dp:].data_ptr(), k_rot=flat[:, a.rank_stored:].data_ptr(),
                        k_ld=kv.stride(0), v_row=kv.stride(0), rot_ld=a.row, gate=N.ptr(gate), gate_ld=gate.stride(0) if gate is not None else 0,
                        tiles=context.tiles.data_ptr(), n_tiles=context.tiles.shape[0], n=n, H=H, G=H, D=a.dim, Dp=Dp, Dv=a.vdim, Dvp=Dvp, v_ld=Dvp, maps=1,
                        window=A.UNBOUNDED, scale=float(a.scale), bf16=1, flat_rows=context.rows, rot_dim=a.rot_dim, status=status)
    N.check(N.lib().ptb_window_attn_tiles(C.byref(args), _st(q)), "window_attn_tiles")
    return out


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
