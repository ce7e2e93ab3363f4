"""Several fp32 residual streams per token (hyper-connections) around layer-normed sublayers (csrc/streams.cu).

A sublayer reads a weighed sum of the streams, ``u = sum_s way_in[s] x_s``, through a layer norm and, where the design has one, a causal
convolution that is added to its own input; its output, times a sigmoid gate computed from the normed row, joins them:
``x_t <- sum_s mix[s, t] x_s + way_out[t] y``.  :func:`step` is what stands between two sublayers, in one launch: the output of the one
before (a :class:`~prometorch_b200.ops.residual.Branch`, the rows of a mixture of experts, or both) into the streams, then the next
one's input.  :func:`pair_embed` starts the streams from a token, a pair and a position table.  CUDA tensors run the kernels, CPU tensors
the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .. import _native as N
from . import recurrence as R
from .experts import ExpertRows
from .paged import _status
from .residual import Branch, _bf16, _st


class DenseArgs(C.Structure):
    """``PtbDense`` of csrc/ptb200_types.h."""
    _fields_ = [("y", C.c_void_p), ("f32", C.c_int), ("splits", C.c_int), ("stride", C.c_longlong), ("ld", C.c_longlong)]

    @classmethod
    def of(cls, b: Optional[Branch]) -> "DenseArgs":
        if b is None:
            return cls()
        assert b.w is None and b.g == 1.0 and b.y.stride(-1) == 1
        return cls(*b.parts()[:5])


class PairEmbedArgs(C.Structure):
    """``PtbPairEmbed`` of csrc/ptb200_types.h."""
    _fields_ = [(n, C.c_void_p) for n in ("ids", "pos", "req", "last", "seqs", "table", "pairs", "at", "x", "status")] + \
        [("mul_before", C.c_longlong), ("mul_id", C.c_longlong)] + \
        [(n, C.c_int) for n in ("id_stride", "pos_stride", "req_stride", "slots", "n_seqs", "n", "V", "rows", "positions", "W", "streams", "bf16")]


class StreamStepArgs(C.Structure):
    """``PtbStreamStep`` of csrc/ptb200_types.h."""
    _fields_ = [(n, C.c_void_p) for n in ("x", "mix", "way_out", "way_in")] + [("y", DenseArgs), ("gate", DenseArgs)] + \
        [(n, C.c_void_p) for n in ("gate_bias", "index_of", "weight", "experts", "self")] + [("e_ld", C.c_longlong)] + \
        [(n, C.c_void_p) for n in ("norm", "h", "conv", "conv_state", "conv_out", "pos", "req", "index", "status")] + \
        [(n, C.c_int) for n in ("top", "e_rows", "taps", "slots", "pos_stride", "req_stride", "n", "m", "W", "streams", "bf16")] + [("eps", C.c_float)]


@N.register_decls
def _decls(L):
    for n, t in (("ptb_pair_embed", PairEmbedArgs), ("ptb_stream_step", StreamStepArgs)):
        getattr(L, n).argtypes = [C.POINTER(t), C.c_void_p]
        getattr(L, n).restype = C.c_int


MAX_STREAMS = 16


@dataclass
class PairEmbedding:
    """``table[id] + pairs[(id before * mul_before + id * mul_id) mod rows] + at[position]``; a sequence's first token takes the row behind
    the hashed ones."""
    table: torch.Tensor                # [V, W]
    pairs: torch.Tensor                # [rows + 1, W]
    at: torch.Tensor                   # [positions, W]
    mul_before: int
    mul_id: int

    @property
    def rows(self) -> int:
        return self.pairs.shape[0] - 1


def pair_embed(ids: torch.Tensor, e: PairEmbedding, streams: int, last: torch.Tensor, pos: torch.Tensor, req: torch.Tensor,
               seqs: Optional[R.Sequences] = None) -> torch.Tensor:
    """``x [n, streams, W]`` fp32; ``last [slots, 1]`` int32 brings every sequence's token before the batch and takes its last one along
    (``seqs`` as in ``ops/recurrence.py``)."""
    n, (V, W) = ids.shape[0], e.table.shape
    x = torch.empty(n, streams, W, dtype=torch.float32, device=e.table.device)
    if x.is_cuda:
        assert last.dtype == ids.dtype == pos.dtype == req.dtype == torch.int32 and all(t.is_contiguous() for t in (last, e.table, e.pairs, e.at))
        a = PairEmbedArgs(ids.data_ptr(), pos.data_ptr(), req.data_ptr(), last.data_ptr(), seqs.device.data_ptr() if seqs else 0, e.table.data_ptr(),
                          e.pairs.data_ptr(), e.at.data_ptr(), x.data_ptr(), _status(x.device).data_ptr(), e.mul_before, e.mul_id, ids.stride(0), pos.stride(0),
                          req.stride(0), last.shape[0], len(seqs.host) if seqs else 0, n, V, e.rows, e.at.shape[0], W, streams, _bf16(e.table))
        N.check(N.lib().ptb_pair_embed(C.byref(a), _st(x)), "pair_embed")
        return x
    row = torch.full((n,), e.rows, dtype=torch.long)
    for lo, count, at, slot in (seqs or R.Sequences.of_rows(pos, req)).host:
        t = torch.cat([last[slot].long(), ids[lo:lo + count].long()])
        pair = (t[:-1] * e.mul_before + t[1:] * e.mul_id) % e.rows
        row[lo + (at == 0):lo + count] = pair[int(at == 0):]
        last[slot, 0] = t[-1]
    return x.copy_((e.table[ids.long()].float() + e.pairs[row].float() + e.at[pos.long()].float())[:, None, :].expand_as(x))


@dataclass
class Connection:
    """How a sublayer reads the streams and joins them (all fp32)."""
    way_in: torch.Tensor               # [S]
    mix: torch.Tensor                  # [S, S]: from, to
    way_out: torch.Tensor              # [S]
    norm: torch.Tensor                 # [W] weight of the layer norm
    conv: torch.Tensor                 # [taps, W], the current token's tap last
    gate_bias: torch.Tensor            # [W]


@dataclass
class Output:
    """What a sublayer leaves: a product, the rows of its experts, or both; ``gate``: the gate's product, before bias and sigmoid."""
    link: Connection
    gate: Branch
    y: Optional[Branch] = None
    rows: Optional[ExpertRows] = None


def _value(b: Branch, W: int) -> torch.Tensor:
    """The first ``W`` columns: the rows of a matrix may have been rounded up."""
    return (b.y.float().sum(0) if b.y.dim() == 3 else b.y.float())[:, :W]


def _norm(u: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return torch.nn.functional.layer_norm(u, u.shape[-1:], w, None, eps)


def _launch(x, before: Optional[Output], way_in, norm, eps, dtype, index=None, conv=None, state=None, pos=None, req=None):
    n, S, W = x.shape
    m = n if index is None else index.shape[0]
    assert x.is_contiguous() and x.dtype == torch.float32
    a = StreamStepArgs(x=x.data_ptr(), way_in=N.ptr(way_in), norm=N.ptr(norm), index=N.ptr(index), status=_status(x.device).data_ptr(), n=n, m=m, W=W, streams=S,
                       bf16=int(dtype == torch.bfloat16), eps=float(eps))
    h = hc = None
    if norm is not None:
        h = torch.empty(m, W, dtype=dtype, device=x.device)
        a.h = h.data_ptr()
    if conv is not None:
        hc = torch.empty_like(h)
        assert state.dtype == dtype and state.is_contiguous() and pos.dtype == req.dtype == torch.int32
        a.conv, a.taps, a.conv_state, a.slots, a.conv_out = conv.data_ptr(), conv.shape[0], state.data_ptr(), state.shape[0], hc.data_ptr()
        a.pos, a.pos_stride, a.req, a.req_stride = pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0)
    if before is not None:
        link, r = before.link, before.rows
        a.mix, a.way_out, a.gate_bias = link.mix.data_ptr(), link.way_out.data_ptr(), link.gate_bias.data_ptr()
        a.y, a.gate = DenseArgs.of(before.y), DenseArgs.of(before.gate)
        if r is not None:
            assert r.y.dtype == r.h.dtype == dtype and r.h.is_contiguous() and r.y.stride(1) == 1
            a.index_of, a.weight, a.top, a.experts, a.e_rows, a.e_ld = r.index.data_ptr(), r.weight.data_ptr(), r.index.shape[1], r.y.data_ptr(), r.y.shape[0], r.y.stride(0)
            setattr(a, "self", r.h.data_ptr())
    N.check(N.lib().ptb_stream_step(C.byref(a), _st(x)), "stream_step")
    return h, hc


def step(x: torch.Tensor, before: Optional[Output], nxt: Optional[Connection], eps: float, dtype, state: Optional[torch.Tensor], pos: torch.Tensor,
         req: torch.Tensor, seqs: Optional[R.Sequences] = None) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
    """``x [n, S, W]`` takes the output ``before`` along (in place); returns the next sublayer's normed row and what it reads, the row plus its
    convolution over time (``state [slots, taps - 1, W]`` in ``dtype``), both ``[n, W]``; None without ``nxt``."""
    if x.is_cuda:
        h, hc = _launch(x, before, nxt.way_in if nxt else None, nxt.norm if nxt else None, eps, dtype, None, nxt.conv if nxt and seqs is None else None, state, pos, req)
    else:
        if before is not None:
            link = before.link
            y = sum(v for v in (_value(before.y, x.shape[2]) if before.y else None, before.rows.combine() if before.rows else None) if v is not None)
            y = y * torch.sigmoid(_value(before.gate, x.shape[2]) + link.gate_bias)
            x.copy_(torch.einsum("nsw,st->ntw", x, link.mix) + link.way_out[:, None] * y[:, None, :])
        h = hc = None
        if nxt is not None:
            h = _norm(torch.einsum("nsw,s->nw", x, nxt.way_in), nxt.norm, eps).to(dtype)
    if nxt is not None and hc is None:
        hc = R.short_conv(h, nxt.conv, state, pos, req, seqs, add=True)
    return h, hc


def rows(x: torch.Tensor, norm: torch.Tensor, eps: float, index: Optional[torch.Tensor] = None, dtype=torch.float32) -> torch.Tensor:
    """The layer norm of the sum of the streams of ``x[index]`` (``index`` int64; None: every row) in ``dtype``."""
    if x.is_cuda:
        if index is not None and not index.numel():
            return torch.empty(0, x.shape[2], dtype=dtype, device=x.device)
        return _launch(x, None, None, norm, eps, dtype, index)[0]
    return _norm((x if index is None else x[index]).sum(1), norm, eps).to(dtype)
