"""Softmax attention over the paged cache inside a sliding window or inside chunks of positions (csrc/window_attn.cu,
csrc/window_attn_sm100.cu), with what designs add to it: the first tokens of a sequence stay visible, a learned sink joins every head's
denominator, a gate scales every head's output, two maps weigh the same values and their difference is normed, a learned bias joins every
score by the key's distance.

:class:`WindowAttention` holds what a layer fixes; :func:`proj_norm_write` normalises the whole q and k projections of new tokens
and fills the pages, :func:`rope_write` rotates them instead (``ops/gated_attention.py`` norms them per head);
:func:`window_attention` runs query rows at given positions against the
pages, :func:`window_attention_tiles` the many rows of a prompt.  CUDA tensors run the kernels, CPU tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .. import _native as N
from .paged import PAGE, _status
from .rotary import Rotary

KEYS_PER_CTA = 128                     # WA_KEYS of csrc/window_attn.cuh
UNBOUNDED = 1 << 30                    # a window that never ends


class WindowArgs(C.Structure):
    """``PtbWindowAttn`` of csrc/ptb200_types.h."""
    _fields_ = [(n, C.c_void_p) for n in ("q", "out", "k_pages", "v_pages", "page_table", "pos", "req", "sink", "gate")] + \
        [("gate_ld", C.c_longlong), ("work", C.c_void_p), ("status", C.c_void_p), ("tiles", C.c_void_p), ("rel", C.c_void_p), ("k_rot", C.c_void_p)] + \
        [(n, C.c_longlong) for n in ("k_ld", "v_row", "rot_ld")] + \
        [(n, C.c_int) for n in ("n", "H", "G", "D", "Dp", "Dv", "Dvp", "v_ld", "maps", "pos_stride", "req_stride", "pt_stride", "n_pages", "window", "keep", "chunked",
                                "max_keys", "nsplit", "bf16", "rel_n", "n_tiles", "flat_rows", "rot_dim")] + \
        [(n, C.c_float) for n in ("scale", "mix", "mix_gain", "mix_eps")]


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_proj_norm_write.argtypes = [vp, ll, ci, ci, ci, vp, vp, vp, vp, vp, vp, ci, vp, ci, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, cf, vp, ci, vp]
    L.ptb_proj_norm_write.restype = ci
    L.ptb_window_rows_work_floats.argtypes = [ci, ci, ci, ci]
    L.ptb_window_rows_work_floats.restype = ll
    L.ptb_window_attn_rows.argtypes = [C.POINTER(WindowArgs), vp]
    L.ptb_window_attn_rows.restype = ci
    L.ptb_window_attn_tiles.argtypes = [C.POINTER(WindowArgs), vp]
    L.ptb_window_attn_tiles.restype = ci
    L.ptb_rope_write.argtypes = [vp, ll, ci, ci, ci, vp, vp, vp, vp, vp, ci, ci, vp, ci, vp, ci, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, ci, vp, ci, vp]
    L.ptb_rope_write.restype = ci


def stored(size: int) -> int:
    """Size of a head's vector as the cache stores it: the kernels address 16-element groups."""
    return (size + 15) // 16 * 16


@dataclass
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int                           # query / key size per head
    vdim: int                          # value size per head
    window: int                        # a query sees itself and the window - 1 tokens before it (chunked: what its own chunk has before it)
    keep: int                          # ... and the first `keep` tokens of its sequence
    scale: float
    sink: Optional[torch.Tensor] = None      # [heads] fp32: exp(sink) joins the denominator
    chunked: bool = False              # chunks of `window` positions, counted from the sequence's first
    maps: int = 1                      # 2: q and k of a head are [map 1, map 2]; the output is rms-normed (map 1 - mix map 2) times mix_gain
    mix: float = 0.0
    mix_gain: float = 1.0
    mix_eps: float = 0.0
    rel: Optional[torch.Tensor] = None       # [heads, distances] fp32: added to a scaled score, the last one for all beyond (ops/gated_attention.py makes it)

    @property
    def dim_stored(self) -> int:
        return stored(self.dim)

    @property
    def key_stored(self) -> int:
        """Elements of a token's key row in the pages: its maps side by side."""
        return self.maps * self.dim_stored

    @property
    def vdim_stored(self) -> int:
        return stored(self.vdim)

    def most_keys(self, max_len: int) -> int:
        """The most keys a row at a position below ``max_len`` sees."""
        return max(1, min(max_len, self.window + self.keep))


def proj_norm_write(p: torch.Tensor, cols: Tuple[int, int, int], a: WindowAttention, q_weight: torch.Tensor, k_weight: torch.Tensor, eps: float,
                    pos: torch.Tensor, req: torch.Tensor, page_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor) -> torch.Tensor:
    """``p [n, *]``: a packed projection whose q, k and v rows start at the columns ``cols``.  q ``[n, H, stored dim]`` after an RMS
    norm over all its heads together (fp32 weight ``[H dim]``); k, normed the same way, and v go to the page slot of
    ``(req[i], pos[i])``.  ``pos`` / ``req``: int32 vectors of any stride."""
    n, H, G, D, Dv, Dp, Dvp = p.shape[0], a.heads, a.kv_heads, a.dim, a.vdim, a.dim_stored, a.vdim_stored
    q = torch.empty(n, H, Dp, dtype=p.dtype, device=p.device)
    if p.is_cuda:
        if p.dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"proj_norm_write takes bf16 or fp32, got {p.dtype}")
        assert p.stride(1) == 1 and pos.dtype == req.dtype == page_table.dtype == torch.int32
        st = torch.cuda.current_stream(p.device).cuda_stream
        N.check(N.lib().ptb_proj_norm_write(p.data_ptr(), p.stride(0), *cols, q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), q_weight.data_ptr(),
                                            k_weight.data_ptr(), pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0), page_table.data_ptr(),
                                            page_table.stride(0), k_pages.shape[0], n, H, G, D, Dp, Dv, Dvp, float(eps), _status(p.device).data_ptr(),
                                            int(p.dtype == torch.bfloat16), st), "proj_norm_write")
        return q
    x = p.float()

    def norm(at, heads, w):
        t = x[:, at:at + heads * D]
        return (t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w).reshape(n, heads, D)
    q.zero_()
    q[..., :D] = norm(cols[0], H, q_weight).to(q.dtype)
    at = pos.long()
    pages = page_table[req.long(), at // PAGE].long()
    k_pages[pages, :, at % PAGE] = torch.nn.functional.pad(norm(cols[1], G, k_weight), (0, Dp - D)).to(k_pages.dtype)
    v_pages[pages, :, at % PAGE] = torch.nn.functional.pad(x[:, cols[2]:cols[2] + G * Dv].reshape(n, G, Dv), (0, Dvp - Dv)).to(v_pages.dtype)
    return q


def rope_write(p: torch.Tensor, cols: Tuple[int, int, int], a: WindowAttention, rot: Rotary, pos: torch.Tensor, req: torch.Tensor,
               page_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor) -> torch.Tensor:
    """``p [n, *]``: a packed projection whose q, k and v rows start at the columns ``cols``.  Rotated q ``[n, H maps, stored dim]``; k,
    rotated likewise, and v go to the page slot of ``(req[i], pos[i])``."""
    n, G, D, Dv, Dp, Dvp = p.shape[0], a.kv_heads, a.dim, a.vdim, a.dim_stored, a.vdim_stored
    Hm, Gm = a.heads * a.maps, G * a.maps
    q = torch.empty(n, Hm, Dp, dtype=p.dtype, device=p.device)
    if p.is_cuda:
        if p.dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"rope_write takes bf16 or fp32, got {p.dtype}")
        assert p.stride(1) == 1 and pos.dtype == req.dtype == page_table.dtype == torch.int32
        N.check(N.lib().ptb_rope_write(p.data_ptr(), p.stride(0), *cols, q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), N.ptr(rot.cos), N.ptr(rot.sin), rot.dims,
                                       rot.positions, pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0), page_table.data_ptr(), page_table.stride(0),
                                       k_pages.shape[0], n, a.heads, G, a.maps, D, Dp, Dv, Dvp, _status(p.device).data_ptr(), int(p.dtype == torch.bfloat16),
                                       torch.cuda.current_stream(p.device).cuda_stream), "rope_write")
        return q
    x = p.float()
    turn = lambda at, heads: torch.nn.functional.pad(rot.apply(x[:, at:at + heads * D].reshape(n, heads, D), pos), (0, Dp - D))
    q.copy_(turn(cols[0], Hm))
    at = pos.long()
    pages = page_table[req.long(), at // PAGE].long()
    k_pages[pages, :, at % PAGE] = turn(cols[1], Gm).reshape(n, G, a.maps * Dp).to(k_pages.dtype)
    v_pages[pages, :, at % PAGE] = torch.nn.functional.pad(x[:, cols[2]:cols[2] + G * Dv].reshape(n, G, Dv), (0, Dvp - Dv)).to(v_pages.dtype)
    return q


def pick_splits(rows: int, kv_heads: int, keys: int, sms: int = 148) -> int:
    """CTAs that share a row's keys: as many as bring the grid to about four per SM while a CTA keeps 32 keys, and at least as many
    as the kernel's limit of keys per CTA asks for.  The number of keys is rounded up to a power of two so that the choice (part of
    a CUDA graph's key) changes rarely as a context grows."""
    bucket = 32
    while bucket < keys:
        bucket *= 2
    need = (bucket + KEYS_PER_CTA - 1) // KEYS_PER_CTA
    return int(max(need, min(bucket // 32, -(-4 * sms // max(1, rows * kv_heads)))))


def _args(q: torch.Tensor, a: WindowAttention, page_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, gate) -> WindowArgs:
    return WindowArgs(k_pages=k_pages.data_ptr(), v_pages=v_pages.data_ptr(), page_table=page_table.data_ptr(), pt_stride=page_table.stride(0),
                      n_pages=k_pages.shape[0], sink=N.ptr(a.sink), gate=N.ptr(gate), gate_ld=gate.stride(0) if gate is not None else 0, H=a.heads, G=a.kv_heads,
                      D=a.dim, Dp=a.dim_stored, Dv=a.vdim, Dvp=a.vdim_stored, v_ld=a.vdim_stored, maps=a.maps, window=a.window, keep=a.keep,
                      chunked=int(a.chunked), scale=float(a.scale), mix=float(a.mix), mix_gain=float(a.mix_gain), mix_eps=float(a.mix_eps),
                      bf16=int(q.dtype == torch.bfloat16), status=_status(q.device).data_ptr(), rel=N.ptr(a.rel), rel_n=a.rel.shape[1] if a.rel is not None else 0)


def run_rows(args: WindowArgs, q: torch.Tensor, out: torch.Tensor, pos: torch.Tensor, req: torch.Tensor, nsplit: int, gate=None,
             kernel=None) -> torch.Tensor:
    """The row kernels over all rows of ``q``, in launches whose workspace stays bounded; ``kernel``: another entry point than the usual."""
    n = q.shape[0]
    st = torch.cuda.current_stream(q.device).cuda_stream
    merged = nsplit > 1 or args.maps > 1
    per_row = int(N.lib().ptb_window_rows_work_floats(1, args.H * args.maps, args.Dvp, nsplit)) if merged else 0
    step = min(n, 65535) if not merged else max(1, min(n, 65535, (256 << 20) // max(1, 4 * per_row)))
    work = torch.empty(step * per_row, dtype=torch.float32, device=q.device) if merged else None
    args.nsplit, args.work, args.pos_stride, args.req_stride = nsplit, N.ptr(work), pos.stride(0), req.stride(0)
    for lo in range(0, n, step):
        args.n = min(step, n - lo)
        args.q, args.out, args.pos, args.req = q[lo:].data_ptr(), out[lo:].data_ptr(), pos[lo:].data_ptr(), req[lo:].data_ptr()
        if gate is not None:
            args.gate = gate[lo:].data_ptr()
        N.check((kernel or N.lib().ptb_window_attn_rows)(C.byref(args), st), "attention rows")
    return out


def window_attention(q: torch.Tensor, a: WindowAttention, pos: torch.Tensor, req: torch.Tensor, page_table: torch.Tensor, k_pages: torch.Tensor,
                     v_pages: torch.Tensor, nsplit: int, max_len: int, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rows ``q [n, H maps, stored dim]`` at ``pos`` of the sequences in page-table rows ``req``, against their cached tokens (their own
    included).  ``max_len``: no row's position is at or past it.  ``gate [n, H]`` (any row pitch): its sigmoid scales the heads.
    Returns ``[n, H vdim]``."""
    if not q.is_cuda:
        return window_attention_reference(q, a, pos, req, page_table, k_pages, v_pages, gate)
    out = torch.empty(q.shape[0], a.heads * a.vdim, dtype=q.dtype, device=q.device)
    args = _args(q, a, page_table, k_pages, v_pages, gate)
    args.max_keys = a.most_keys(max_len)
    return run_rows(args, q, out, pos, req, nsplit, gate)


QUERY_TILE = 128                       # queries per tile of csrc/window_attn_sm100.cu
TILE_DISTANCES = 8192                  # entries of a head's distance bias that its tiles hold (MAX_REL there)
TILES_FROM = 16                        # rows of a prompt pass from which the tile kernel is the better choice


@dataclass
class PromptTiles:
    """The query tiles of a prompt pass: on the device ``[tiles, 4]`` int32 (first row, its position, rows, page-table row), tiles
    with many keys first."""
    host: List[Tuple[int, int, int, int]]
    device: torch.Tensor

    @classmethod
    def of(cls, offs: List[int], starts: List[int], rows: List[int], device) -> "PromptTiles":
        host = [(lo + i, at + i, min(QUERY_TILE, hi - lo - i), r) for lo, hi, at, r in zip(offs, offs[1:], starts, rows)
                for i in range(0, hi - lo, QUERY_TILE)]
        host.sort(key=lambda t: -t[1])
        return cls(host, torch.tensor(host, dtype=torch.int32).to(device))


def tiles_supported(q: torch.Tensor, a: WindowAttention) -> bool:
    return q.is_cuda and q.dtype == torch.bfloat16 and a.dim_stored <= 128 and a.vdim_stored <= 128 and \
        (a.rel is None or (a.maps == 1 and a.rel.shape[1] <= TILE_DISTANCES))


def window_attention_tiles(q: torch.Tensor, a: WindowAttention, tiles: PromptTiles, page_table: torch.Tensor, k_pages: torch.Tensor,
                           v_pages: torch.Tensor, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """A prompt pass's rows against the pages, both products on tcgen05 (sizes: :func:`tiles_supported`)."""
    out = torch.empty(q.shape[0], a.heads * a.vdim, dtype=q.dtype, device=q.device)
    args = _args(q, a, page_table, k_pages, v_pages, gate)
    args.q, args.out, args.n, args.tiles, args.n_tiles = q.data_ptr(), out.data_ptr(), q.shape[0], tiles.device.data_ptr(), len(tiles.host)
    N.check(N.lib().ptb_window_attn_tiles(C.byref(args), torch.cuda.current_stream(q.device).cuda_stream), "window_attn_tiles")
    return out


def window_attention_reference(q, a: WindowAttention, pos, req, page_table, k_pages, v_pages, gate=None) -> torch.Tensor:
    """The same in plain fp32 math, sequence by sequence (CPU path).  Pages between the kept tokens and the first window are gone."""
    n, H, G, D, Dv = q.shape[0], a.heads, a.kv_heads, a.dim, a.vdim
    out = torch.zeros(n, H * Dv, dtype=q.dtype, device=q.device)
    R = H // G
    qs = q.reshape(n, H, a.maps, a.dim_stored)[..., :D].float()
    for r in torch.unique(req).tolist():
        rows = (req == r).nonzero()[:, 0]
        p = pos[rows].long()
        low = p - p % a.window if a.chunked else (p - a.window + 1).clamp_min(0)           # first position inside the window
        top, first = int(p.max()) + 1, int(low.min())
        j = torch.cat([torch.arange(0, min(a.keep, first)), torch.arange(first, top)]).to(q.device)
        pages = page_table[r, j // PAGE].long()
        k = k_pages[pages, :, j % PAGE].float().reshape(len(j), G, a.maps, a.dim_stored)[..., :D]
        v = v_pages[pages, :, j % PAGE].float()[..., :Dv].transpose(0, 1).repeat_interleave(R, 0)          # [H, keys, Dv]
        see = (j[None, :] <= p[:, None]) & ((j[None, :] >= low[:, None]) | (j[None, :] < a.keep))
        o = []
        for m in range(a.maps):
            km = k[:, :, m].transpose(0, 1).repeat_interleave(R, 0)                                        # [H, keys, D]
            s = torch.einsum("nhd,hjd->hnj", qs[rows, :, m], km) * a.scale
            if a.rel is not None:
                s = s + a.rel[:, (p[:, None] - j[None, :]).clamp(0, a.rel.shape[1] - 1)]
            s = s.masked_fill(~see, float("-inf"))
            if a.sink is not None:
                s = torch.cat([s, a.sink.float()[:, None, None].expand(H, len(rows), 1)], -1)
            o.append(torch.einsum("hnj,hjd->nhd", torch.softmax(s, -1)[..., :len(j)], v))
        y = o[0]
        if a.maps == 2:
            y = y - a.mix * o[1]
            y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + a.mix_eps) * a.mix_gain
        if gate is not None:
            y = y * torch.sigmoid(gate[rows].float())[..., None]
        out[rows] = y.reshape(len(rows), H * Dv).to(q.dtype)
    return out
