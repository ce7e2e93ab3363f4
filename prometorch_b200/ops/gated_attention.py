"""Gated attention over the paged cache (csrc/gated_attn.cuh): weights are a sigmoid of the soft-capped, distance-biased score,
not normalised over the keys, optionally mixed across heads, inside a sliding window.

:class:`GatedAttention` holds what a layer fixes; :func:`head_norm_write` normalises q and k of new tokens, mixes values and fills
the pages; :func:`gated_attention` runs query rows at given positions against the pages.  CUDA tensors run the kernels, CPU
tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .. import _native as N
from .paged import PAGE, _status

KEYS_PER_CTA = 128                     # GA_KEYS of csrc/gated_attn.cuh


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_head_norm_write.argtypes = [vp, ll, ci, ci, vp, vp, vp, vp, vp, vp, ci, vp, ll, cf, vp, ci, vp, ci, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, cf, vp, ci, vp]
    L.ptb_head_norm_write.restype = ci
    L.ptb_gated_rows_work_floats.argtypes = [ci, ci, ci, ci]
    L.ptb_gated_rows_work_floats.restype = ll
    L.ptb_gated_attn_rows.argtypes = [vp, vp, ci, ci, ci, ci, ci, ci, vp, ci, vp, ci, vp, ci, ci, vp, vp, vp, ci, vp, ci, cf, cf, ci, vp, ci, vp, ci, vp]
    L.ptb_gated_attn_rows.restype = ci
    L.ptb_gated_tiles_supported.argtypes = [ci, ci, ci, ci]
    L.ptb_gated_tiles_supported.restype = ci
    L.ptb_gated_attn_tiles.argtypes = [vp, vp, ci, vp, ci, ci, ci, ci, ci, ci, vp, ci, ci, vp, vp, vp, ci, vp, ci, cf, cf, vp, ci, ci, ci, vp, vp]
    L.ptb_gated_attn_tiles.restype = ci


def stored(size: int) -> int:
    """Size of a head's vector as the cache stores it: the kernels address 16-element groups."""
    return (size + 15) // 16 * 16


def distance_buckets(rows: int, dmax: float, count: int) -> torch.Tensor:
    """Row of a bias table with ``rows`` rows for the distances 0 .. count - 1: the distance itself below half = rows // 2, then
    half + floor(ln(n / half) / ln(dmax / half) * (rows - half)), at most rows - 1.  The floor is decided in exact integer
    arithmetic when dmax is one (n / half >= (dmax / half)^(k / (rows - half)) without logarithms), so a distance that falls on
    a bucket's edge does not depend on how a logarithm is rounded."""
    import math
    half = rows // 2
    if half < 1 or (count > half and dmax <= half):
        raise ValueError(f"distance buckets: {rows} rows up to distance {dmax}")
    m, out, k = rows - half, [], 0
    exact = float(dmax).is_integer()
    for n in range(count):
        if n < half:
            out.append(n)
            continue
        if exact:
            D = int(dmax)
            while k + 1 <= m and D ** (k + 1) * half ** m <= n ** m * half ** (k + 1):     # (D/h)^(k+1) <= (n/h)^m
                k += 1
        else:
            k = math.floor(math.log(n / half) / math.log(dmax / half) * m)
        out.append(min(rows - 1, half + k))
        if out[-1] == rows - 1:
            out += [rows - 1] * (count - len(out))
            break
    return torch.tensor(out, dtype=torch.long)


def distance_bias(rel: torch.Tensor, dmax: float, window: int, head_bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``[H, nb]`` fp32: what is added to a score at distance n (the last column stands for every larger distance), from a table
    ``rel [rows, H]`` of learned biases and an optional number per head."""
    rows = rel.shape[0]
    b = distance_buckets(rows, dmax, window)
    last = (b == rows - 1).nonzero()
    nb = int(last[0]) + 1 if len(last) else window
    t = rel.float()[b[:nb].to(rel.device)].t()
    if head_bias is not None:
        t = t + head_bias.float()[:, None]
    return t.contiguous()


@dataclass
class GatedAttention:
    heads: int
    kv_heads: int
    dim: int                           # query / key size per head
    vdim: int                          # value size per head
    window: int                        # a query sees itself and the window - 1 tokens before it
    scale: float
    softcap: float                     # 0: none
    bias: torch.Tensor                 # [heads, nb] fp32, see distance_bias
    talk: Optional[torch.Tensor]       # [heads, heads] fp32 (to, from), or None

    @property
    def dim_stored(self) -> int:
        return stored(self.dim)

    @property
    def vdim_stored(self) -> int:
        return stored(self.vdim)


def head_norm_write(qkv: torch.Tensor, a, q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor], eps: float, pos: torch.Tensor, req: torch.Tensor,
                    page_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, v_first: Optional[torch.Tensor] = None, lam: float = 0.0,
                    cols: Optional[Tuple[int, int]] = None, gain: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``a``: anything with the sizes of a :class:`GatedAttention`.  ``qkv [n, *]``: q heads, then k and v heads (at the columns ``cols``, by default one
    after the other) -> q ``[n, H, stored dim]`` after the heads' norm (a weight may be None), times ``gain[pos]`` (fp32 ``[positions]``); keys (normalised) and values
    ``(1 - lam) v + lam v_first`` go to the page slot of ``(req[i], pos[i])``.  ``pos`` / ``req``: int32 vectors of any stride."""
    n, H, G, D, Dv, Dp, Dvp = qkv.shape[0], a.heads, a.kv_heads, a.dim, a.vdim, a.dim_stored, a.vdim_stored
    kc, vc = cols or (H * D, (H + G) * D)
    q = torch.empty(n, H, Dp, dtype=qkv.dtype, device=qkv.device)
    if qkv.is_cuda:
        if qkv.dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"head_norm_write takes bf16 or fp32, got {qkv.dtype}")
        assert qkv.stride(1) == 1 and (v_first is None or v_first.stride(1) == 1) and pos.dtype == req.dtype == page_table.dtype == torch.int32
        st = torch.cuda.current_stream(qkv.device).cuda_stream
        N.check(N.lib().ptb_head_norm_write(qkv.data_ptr(), qkv.stride(0), kc, vc, q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), N.ptr(q_weight),
                                            N.ptr(k_weight), N.ptr(gain), gain.shape[0] if gain is not None else 0, N.ptr(v_first), v_first.stride(0) if v_first is not None else 0, float(lam),
                                            pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0), page_table.data_ptr(),
                                            page_table.stride(0), k_pages.shape[0], n, H, G, D, Dp, Dv, Dvp, float(eps),
                                            _status(qkv.device).data_ptr(), int(qkv.dtype == torch.bfloat16), st), "head_norm_write")
        return q
    x = qkv.float()
    qs, ks, v = x[:, :H * D].reshape(n, H, D), x[:, kc:kc + G * D].reshape(n, G, D), x[:, vc:vc + G * Dv].reshape(n, G, Dv)

    def norm(t, w):
        t = t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)
        return t if w is None else t * w
    if v_first is not None:
        v = (1 - lam) * v + lam * v_first.float().reshape(n, G, Dv)
    q.zero_()
    p = pos.long()
    qn = norm(qs, q_weight)
    q[..., :D] = (qn if gain is None else qn * gain[p][:, None, None]).to(q.dtype)
    pages = page_table[req.long(), p // PAGE].long()
    k_pages[pages, :, p % PAGE] = torch.nn.functional.pad(norm(ks, k_weight), (0, Dp - D)).to(k_pages.dtype)
    v_pages[pages, :, p % PAGE] = torch.nn.functional.pad(v, (0, Dvp - Dv)).to(v_pages.dtype)
    return q


def pick_splits(rows: int, window: int, max_len: int, sms: int = 148) -> int:
    """CTAs that share a row's keys: as many as bring the grid to about two per SM while a CTA keeps 16 keys, and at least as
    many as the kernel's limit of keys per CTA asks for.  The visible length is rounded up to a power of two so that the choice
    (part of a CUDA graph's key) changes rarely as a context grows."""
    keys = 16
    while keys < min(window, max_len):
        keys *= 2
    keys = min(keys, max(window, 1))
    need = (keys + KEYS_PER_CTA - 1) // KEYS_PER_CTA
    return int(max(need, min((keys + 15) // 16, -(-2 * sms // max(1, rows)))))


def gated_attention(q: torch.Tensor, a: GatedAttention, pos: torch.Tensor, req: torch.Tensor, page_table: torch.Tensor, k_pages: torch.Tensor,
                    v_pages: torch.Tensor, nsplit: int, max_len: int) -> torch.Tensor:
    """Rows ``q [n, H, stored dim]`` at ``pos`` of the sequences in page-table rows ``req``, against their cached tokens (their own
    included).  ``max_len``: no row's position is at or past it.  Returns ``[n, H vdim]``."""
    n, H, G = q.shape[0], a.heads, a.kv_heads
    if not q.is_cuda:
        return gated_attention_reference(q, a, pos, req, page_table, k_pages, v_pages)
    out = torch.empty(n, H * a.vdim, dtype=q.dtype, device=q.device)
    st = torch.cuda.current_stream(q.device).cuda_stream
    per_row = int(N.lib().ptb_gated_rows_work_floats(1, H, a.vdim_stored, nsplit))
    step = n if nsplit == 1 else max(1, min(n, (256 << 20) // max(1, 4 * per_row)))       # bound the workspace
    step = min(step, 65535)
    work = torch.empty(step * per_row, dtype=torch.float32, device=q.device) if nsplit > 1 else None
    for lo in range(0, n, step):
        m = min(step, n - lo)
        N.check(N.lib().ptb_gated_attn_rows(q[lo:].data_ptr(), out[lo:].data_ptr(), m, H, G, a.dim_stored, a.vdim, a.vdim_stored, pos[lo:].data_ptr(),
                                            pos.stride(0), req[lo:].data_ptr(), req.stride(0), page_table.data_ptr(), page_table.stride(0),
                                            k_pages.shape[0], k_pages.data_ptr(), v_pages.data_ptr(), a.bias.data_ptr(), a.bias.shape[1],
                                            N.ptr(a.talk), a.window, float(a.scale), float(a.softcap), int(max_len), N.ptr(work), nsplit,
                                            _status(q.device).data_ptr(), int(q.dtype == torch.bfloat16), st), "gated_attn_rows")
    return out


QUERY_TILE = 32                        # queries per tile of csrc/gated_prefill.cu
TILES_FROM = 64                        # rows of a prompt pass from which the tile kernels are the better choice
STEPS_PER_CTA = 9                      # 32-key steps of one CTA: short enough to balance bands of different lengths
WEIGHTS_BYTES = 320 << 20              # scratch of the tile kernels per launch


@dataclass
class PromptTiles:
    """The query tiles of a prompt pass: on the device ``[tiles, 4]`` int32 (first row, its position, rows, page-table row)."""
    host: List[Tuple[int, int, int, int]]
    device: torch.Tensor
    n: int

    @classmethod
    def of(cls, offs: List[int], starts: List[int], rows: List[int], device) -> "PromptTiles":
        host = [(lo + i, at + i, min(QUERY_TILE, hi - lo - i), r) for lo, hi, at, r in zip(offs, offs[1:], starts, rows)
                for i in range(0, hi - lo, QUERY_TILE)]
        return cls(host, torch.tensor(host, dtype=torch.int32).to(device), offs[-1])

    def width(self, window: int) -> int:
        """Columns of the weights' band: whole 64-key blocks from the first one a tile sees to its last query."""
        return max((at + n - max(0, at - window + 1) // PAGE * PAGE + PAGE - 1) // PAGE * PAGE for _, at, n, _ in self.host)


def tiles_supported(q: torch.Tensor, a: GatedAttention) -> bool:
    return q.is_cuda and q.dtype == torch.bfloat16 and bool(N.lib().ptb_gated_tiles_supported(a.heads, a.kv_heads, a.dim_stored, a.vdim_stored))


def gated_attention_tiles(q: torch.Tensor, a: GatedAttention, tiles: PromptTiles, page_table: torch.Tensor, k_pages: torch.Tensor,
                          v_pages: torch.Tensor, tensor_cores: bool = True) -> torch.Tensor:
    """A prompt pass's rows against the pages, on the tensor cores (sizes: :func:`tiles_supported`).  ``tensor_cores``: the
    scores and the head mixing on tcgen05 where its kernel takes the sizes, else on mma.sync."""
    H, n, nt = a.heads, q.shape[0], len(tiles.host)
    out = torch.empty(n, H * a.vdim, dtype=q.dtype, device=q.device)
    KW = tiles.width(a.window)
    step = max(1, min(nt, WEIGHTS_BYTES // (2 * H * QUERY_TILE * KW), 65535))
    step = -(-nt // -(-nt // step))                                    # equal shares
    weights = torch.empty(step * H * QUERY_TILE * KW, dtype=torch.bfloat16, device=q.device)
    st = torch.cuda.current_stream(q.device).cuda_stream
    for lo in range(0, nt, step):
        m = min(step, nt - lo)
        N.check(N.lib().ptb_gated_attn_tiles(q.data_ptr(), out.data_ptr(), n, tiles.device[lo:].data_ptr(), m, H, a.kv_heads, a.dim_stored, a.vdim,
                                             a.vdim_stored, page_table.data_ptr(), page_table.stride(0), k_pages.shape[0], k_pages.data_ptr(),
                                             v_pages.data_ptr(), a.bias.data_ptr(), a.bias.shape[1], N.ptr(a.talk), a.window, float(a.scale),
                                             float(a.softcap), weights.data_ptr(), KW, STEPS_PER_CTA, int(tensor_cores), _status(q.device).data_ptr(), st), "gated_attn_tiles")
    return out


def gated_attention_reference(q, a: GatedAttention, pos, req, page_table, k_pages, v_pages) -> torch.Tensor:
    """The same in plain fp32 math, sequence by sequence (CPU path)."""
    n, H, G, D, Dv = q.shape[0], a.heads, a.kv_heads, a.dim, a.vdim
    out = torch.zeros(n, H * Dv, dtype=q.dtype, device=q.device)
    R, nb = H // G, a.bias.shape[1]
    for r in torch.unique(req).tolist():
        rows = (req == r).nonzero()[:, 0]
        p = pos[rows].long()
        first, top = max(0, int(p.min()) - a.window + 1) // PAGE, int(p.max()) // PAGE + 1      # pages behind every window are gone
        pages = page_table[r, first:top].long()
        k = k_pages[pages].float()[..., :D].permute(1, 0, 2, 3).reshape(G, -1, D).repeat_interleave(R, 0)
        v = v_pages[pages].float()[..., :Dv].permute(1, 0, 2, 3).reshape(G, -1, Dv).repeat_interleave(R, 0)
        dist = p[:, None] - (torch.arange(k.shape[1], device=q.device) + first * PAGE)[None, :]
        s = torch.einsum("nhd,hjd->hnj", q[rows][..., :D].float(), k) * a.scale
        if a.softcap > 0:
            s = a.softcap * torch.tanh(s / a.softcap)
        s = s + a.bias[:, dist.clamp(0, nb - 1)]
        w = torch.sigmoid(s) * ((dist >= 0) & (dist < a.window))
        if a.talk is not None:
            w = torch.einsum("hg,gnj->hnj", a.talk, w)
        out[rows] = torch.einsum("hnj,hjd->nhd", w, v).reshape(len(rows), H * Dv).to(q.dtype)
    return out
