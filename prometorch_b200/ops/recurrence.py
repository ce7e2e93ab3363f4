"""Recurrent layers with a matrix state per head (csrc/recurrence.cu, csrc/recurrence_chunk.cu): linear attention with a fixed decay,
the gated delta rule with a decay per key channel or per head, state-space steps, and the short causal convolution and the gated norm that go
with them.

A sequence's state is one slot of ``[slots, H, dim, vdim]`` fp32 (and ``[slots, taps - 1, channels]`` of convolution inputs); a token
at position 0 starts from zero whatever the slot holds.  A decode pass gives one token per row (``seqs`` None: slot ``req[i]``,
position ``pos[i]``); a prompt pass gives :class:`Sequences`.  CUDA tensors run the kernels, CPU tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union

import torch

from .. import _native as N
from .paged import _status


class RecurrenceArgs(C.Structure):
    """``PtbRecurrence`` of csrc/ptb200_types.h."""
    _fields_ = [("x", C.c_void_p), ("ld", C.c_longlong), ("q_col", C.c_int), ("k_col", C.c_int), ("v_col", C.c_int),
                ("silu", C.c_int), ("delta", C.c_int), ("bf16", C.c_int),
                ("beta", C.c_void_p), ("ld_beta", C.c_longlong), ("a", C.c_void_p), ("ld_a", C.c_longlong),
                ("decay", C.c_void_p), ("dt_bias", C.c_void_p),
                ("state", C.c_void_p), ("slots", C.c_int), ("n", C.c_int), ("H", C.c_int), ("G", C.c_int), ("D", C.c_int), ("Dv", C.c_int),
                ("seqs", C.c_void_p), ("n_seqs", C.c_int), ("pos_stride", C.c_int), ("req_stride", C.c_int), ("pad", C.c_int),
                ("pos", C.c_void_p), ("req", C.c_void_p), ("out", C.c_void_p), ("status", C.c_void_p),
                ("chunks", C.c_void_p), ("first_chunk", C.c_void_p), ("n_chunks", C.c_int), ("rank", C.c_int),
                ("low", C.c_void_p), ("ld_low", C.c_longlong), ("low_w", C.c_void_p), ("skip", C.c_void_p)]


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_short_conv.argtypes = [vp, ll, vp, vp, ci, ci, ci, vp, vp, ci, ci, vp, ci, vp, ci, vp, ci, vp, ci, vp]
    L.ptb_short_conv.restype = ci
    L.ptb_recurrence.argtypes = [C.POINTER(RecurrenceArgs), vp]
    L.ptb_recurrence.restype = ci
    L.ptb_group_norm_gate.argtypes = [vp, vp, vp, ci, ll, vp, ci, ci, ci, cf, ci, ci, ci, ci, vp]
    L.ptb_group_norm_gate.restype = ci
    L.ptb_recurrence_chunked.argtypes = [C.POINTER(RecurrenceArgs), vp, ll, vp]
    L.ptb_recurrence_chunked.restype = ci
    L.ptb_recurrence_chunked_bytes.argtypes = [C.POINTER(RecurrenceArgs)]
    L.ptb_recurrence_chunked_bytes.restype = ll


CHUNK = 64                             # rows of a chunk of csrc/recurrence_chunk.cu
CHUNKED_FROM = 32                      # longest sequence of a prompt pass from which it runs in chunks


@dataclass
class Sequences:
    """The sequences of a prompt pass: on the device ``[sequences, 4]`` int32 (first row, rows, position of the first, slot), and
    their cut into chunks for the matrix form: ``[chunks, 4]`` (first row, rows, sequence, unused) and every sequence's first chunk."""
    host: List[Tuple[int, int, int, int]]
    device: torch.Tensor
    chunks: Optional[torch.Tensor] = None
    first_chunk: Optional[torch.Tensor] = None

    @classmethod
    def of(cls, offs: List[int], starts: List[int], rows: List[int], device) -> "Sequences":
        host = [(lo, hi - lo, at, r) for lo, hi, at, r in zip(offs, offs[1:], starts, rows)]
        chunks, first = [], []
        for i, (lo, n, _, _) in enumerate(host):
            first.append(len(chunks))
            chunks += [(lo + j, min(CHUNK, n - j), i, 0) for j in range(0, n, CHUNK)]
        up = lambda t: torch.tensor(t, dtype=torch.int32).to(device)
        return cls(host, up(host), up(chunks), up(first))

    @classmethod
    def of_rows(cls, pos: torch.Tensor, req: torch.Tensor) -> "Sequences":
        """One token per row (CPU path of a decode pass)."""
        return cls([(i, 1, p, r) for i, (p, r) in enumerate(zip(pos.tolist(), req.tolist()))], pos)


def _st(t):
    return torch.cuda.current_stream(t.device).cuda_stream


def _check(t: torch.Tensor):
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"the recurrence kernels take bf16 or fp32, got {t.dtype}")
    assert t.stride(1) == 1


# ------------------------------------------------------------------------------------------ short convolution
def short_conv(x: torch.Tensor, weight: torch.Tensor, state: torch.Tensor, pos: torch.Tensor, req: torch.Tensor,
               seqs: Optional[Sequences] = None, bias: Optional[torch.Tensor] = None, add: bool = False) -> torch.Tensor:
    """``x [n, C]`` (any row pitch), ``weight [taps, C]`` fp32 with the current token's tap last: per channel the weighted sum of a
    token and the taps - 1 before it, plus ``bias [C]`` fp32, then SiLU; with ``add`` the input plus that sum
    instead; ``state [slots, taps - 1, C]`` in the type of x brings the inputs from before the batch and takes the last ones along.  Returns ``[n, C]``."""
    n, Ch = x.shape
    taps = weight.shape[0]
    out = torch.empty(n, Ch, dtype=x.dtype, device=x.device)
    if x.is_cuda:
        _check(x)
        assert state.dtype == x.dtype and state.is_contiguous() and weight.is_contiguous()
        N.check(N.lib().ptb_short_conv(x.data_ptr(), x.stride(0), weight.data_ptr(), N.ptr(bias), int(add), Ch, taps, state.data_ptr(), out.data_ptr(), n, state.shape[0],
                                       pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0), seqs.device.data_ptr() if seqs else 0,
                                       len(seqs.host) if seqs else 0, _status(x.device).data_ptr(), int(x.dtype == torch.bfloat16), _st(x)), "short_conv")
        return out
    for lo, count, at, slot in (seqs or Sequences.of_rows(pos, req)).host:
        before = state[slot].float()
        before[:max(0, taps - 1 - at)] = 0                      # rows from before position 0
        full = torch.cat([before, x[lo:lo + count].float()])
        y = sum(full[i:i + count] * weight[i].float() for i in range(taps))
        y = y if bias is None else y + bias
        out[lo:lo + count] = (x[lo:lo + count].float() + y if add else torch.nn.functional.silu(y)).to(out.dtype)
        state[slot] = full[full.shape[0] - (taps - 1):].to(state.dtype)
    return out


# ------------------------------------------------------------------------------------------ recurrences
@dataclass
class DeltaRule:
    """The gated delta rule of one layer: per head ``S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q`` with q and k made unit
    vectors (q also times dim^-1/2), ``beta`` a sigmoid and ``g = exp(-rate softplus(a + dt_bias))`` per head and key channel, or with
    ``head_decay`` one number per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rate: torch.Tensor                 # [H] fp32: exp(A_log)
    dt_bias: torch.Tensor              # [H dim] fp32 ([H] with head_decay)
    head_decay: bool = False


@dataclass
class DecayAttention:
    """Linear attention of one layer: ``S <- decay_h S + k v^T; o = S^T q``; ``silu``: q, k and v pass SiLU first."""
    heads: int
    dim: int
    vdim: int
    decay: torch.Tensor                # [H] fp32
    silu: bool = True


@dataclass
class StateSpace:
    """The recurrence of a state-space layer: per head ``S <- exp(-rate dt) S + dt k v^T; o = S^T q + skip v`` with the step
    ``dt = softplus(a + dt_bias)``; q and k are shared by the heads of a group."""
    heads: int
    groups: int
    dim: int                           # rows of the state: size of q and k
    vdim: int
    rate: torch.Tensor                 # [H] fp32: exp(A_log)
    dt_bias: torch.Tensor              # [H] fp32
    skip: torch.Tensor                 # [H] fp32


def _unit(x):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def _runs_chunked(x: torch.Tensor, D: int, Dv: int, seqs: Optional[Sequences], chunked: Optional[bool]) -> bool:
    """Whether the kernels of csrc/recurrence_chunk.cu take this pass: bf16 prompts of some length, head sizes up to 128."""
    if seqs is None or x.dtype != torch.bfloat16 or max(D, Dv) > 128 or chunked is False:
        return False
    return bool(chunked) or max(c for _, c, _, _ in seqs.host) >= CHUNKED_FROM


def _run(args: RecurrenceArgs, x: torch.Tensor, seqs: Optional[Sequences], pos, req, state: torch.Tensor, out: torch.Tensor, chunked: bool):
    args.x, args.ld, args.bf16 = x.data_ptr(), x.stride(0), int(x.dtype == torch.bfloat16)
    args.state, args.slots, args.n, args.out, args.status = state.data_ptr(), state.shape[0], x.shape[0], out.data_ptr(), _status(x.device).data_ptr()
    args.pos, args.pos_stride, args.req, args.req_stride = pos.data_ptr(), pos.stride(0), req.data_ptr(), req.stride(0)
    if seqs is not None:
        args.seqs, args.n_seqs = seqs.device.data_ptr(), len(seqs.host)
        args.chunks, args.n_chunks, args.first_chunk = seqs.chunks.data_ptr(), seqs.chunks.shape[0], seqs.first_chunk.data_ptr()
    if chunked:
        work = torch.empty(int(N.lib().ptb_recurrence_chunked_bytes(C.byref(args))), dtype=torch.uint8, device=x.device)
        N.check(N.lib().ptb_recurrence_chunked(C.byref(args), work.data_ptr(), work.numel(), _st(x)), "recurrence_chunked")
    else:
        N.check(N.lib().ptb_recurrence(C.byref(args), _st(x)), "recurrence")


def delta_rule(x: torch.Tensor, r: DeltaRule, beta: torch.Tensor, a: Union[torch.Tensor, Tuple[torch.Tensor, torch.Tensor]], state: torch.Tensor,
               pos: torch.Tensor, req: torch.Tensor, seqs: Optional[Sequences] = None, chunked: Optional[bool] = None) -> torch.Tensor:
    """``x [n, 2 G dim + H vdim]``: q, k and v after their convolutions; ``beta [n, H]`` before its sigmoid (type of x); ``a [n, H
    dim]`` fp32, or its factors ``(low [n, rank], w [>= H dim, rank])`` in the type of x, whose product the chunk kernel forms itself; one
    decay per head: ``a [n, H]`` in the type of x.  Advances ``state [slots, H, dim, vdim]``; returns o ``[n, H vdim]`` fp32."""
    n, H, G, D, Dv = x.shape[0], r.heads, r.kv_heads, r.dim, r.vdim
    out = torch.empty(n, H * Dv, dtype=torch.float32, device=x.device)
    if x.is_cuda:
        _check(x)
        assert beta.dtype == x.dtype and state.is_contiguous()
        chunked = _runs_chunked(x, D, Dv, seqs, chunked)
        args = RecurrenceArgs(q_col=0, k_col=G * D, v_col=2 * G * D, delta=1, beta=beta.data_ptr(), ld_beta=beta.stride(0), decay=r.rate.data_ptr(),
                              dt_bias=r.dt_bias.data_ptr(), H=H, G=G, D=D, Dv=Dv)
        if r.head_decay:
            assert a.dtype == x.dtype and a.shape[1] == H and a.stride(1) == 1
            args.delta, args.a, args.ld_a = 2, a.data_ptr(), a.stride(0)
        elif isinstance(a, tuple):
            low, w = a
            rank = w.shape[1]
            if chunked and rank % 8 == 0 and rank <= 256 and low.stride(0) % 8 == 0 and low.data_ptr() % 16 == 0 and w.is_contiguous():
                assert low.dtype == w.dtype == x.dtype and low.shape[1] == rank and w.shape[0] >= H * D and low.stride(1) == 1
                args.low, args.ld_low, args.low_w, args.rank = low.data_ptr(), low.stride(0), w.data_ptr(), rank
            else:
                from .residual import linear_f32
                a = linear_f32(low, w)
        if not isinstance(a, tuple) and not r.head_decay:
            assert a.dtype == torch.float32 and a.stride(1) == 1
            args.a, args.ld_a = a.data_ptr(), a.stride(0)
        _run(args, x, seqs, pos, req, state, out, chunked)
        return out
    if isinstance(a, tuple):
        a = (a[0].float() @ a[1].float().t())[:, :H * D]
    f = x.float()
    q = (_unit(f[:, :G * D].reshape(n, G, D)) * D ** -0.5).repeat_interleave(H // G, 1)
    k = _unit(f[:, G * D:2 * G * D].reshape(n, G, D)).repeat_interleave(H // G, 1)
    v = f[:, 2 * G * D:].reshape(n, H, Dv)
    g = torch.exp(-r.rate[:, None] * torch.nn.functional.softplus(a.float() + r.dt_bias, threshold=50.0).view(n, H, -1))       # [n, H, D or 1]
    b = torch.sigmoid(beta.float())
    o = out.view(n, H, Dv)
    for lo, count, at, slot in (seqs or Sequences.of_rows(pos, req)).host:
        S = state[slot].clone() if at > 0 else torch.zeros_like(state[slot])
        for i in range(lo, lo + count):
            S *= g[i][:, :, None]
            u = b[i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
            S += k[i][:, :, None] * u[:, None, :]
            o[i] = torch.einsum("hdv,hd->hv", S, q[i])
        state[slot] = S
    return out


def decay_attention(x: torch.Tensor, r: DecayAttention, cols: Tuple[int, int, int], state: torch.Tensor, pos: torch.Tensor, req: torch.Tensor,
                    seqs: Optional[Sequences] = None, chunked: Optional[bool] = None) -> torch.Tensor:
    """``x [n, *]``: a packed projection with q, k and v (head by head) at the columns ``cols``.  Advances ``state [slots, H, dim,
    vdim]``; returns o ``[n, H vdim]`` fp32."""
    n, H, D, Dv = x.shape[0], r.heads, r.dim, r.vdim
    out = torch.empty(n, H * Dv, dtype=torch.float32, device=x.device)
    if x.is_cuda:
        _check(x)
        assert state.is_contiguous()
        args = RecurrenceArgs(q_col=cols[0], k_col=cols[1], v_col=cols[2], silu=int(r.silu), delta=0, decay=r.decay.data_ptr(), H=H, G=H, D=D, Dv=Dv)
        _run(args, x, seqs, pos, req, state, out, _runs_chunked(x, D, Dv, seqs, chunked))
        return out
    act = torch.nn.functional.silu if r.silu else (lambda t: t)
    q, k, v = (act(x[:, c:c + H * d].float()).reshape(n, H, d) for c, d in zip(cols, (D, D, Dv)))
    o = out.view(n, H, Dv)
    for lo, count, at, slot in (seqs or Sequences.of_rows(pos, req)).host:
        S = state[slot].clone() if at > 0 else torch.zeros_like(state[slot])
        for i in range(lo, lo + count):
            S = S * r.decay[:, None, None] + k[i][:, :, None] * v[i][:, None, :]
            o[i] = torch.einsum("hdv,hd->hv", S, q[i])
        state[slot] = S
    return out


def state_space(x: torch.Tensor, r: StateSpace, cols: Tuple[int, int, int], a: torch.Tensor, state: torch.Tensor, pos: torch.Tensor, req: torch.Tensor,
                seqs: Optional[Sequences] = None, chunked: Optional[bool] = None) -> torch.Tensor:
    """``x [n, *]``: q and k (group by group) and v (head by head) at the columns ``cols``; ``a [n, H]`` in the type of x.  Advances ``state
    [slots, H, dim, vdim]``; returns o ``[n, H vdim]`` fp32."""
    n, H, G, D, Dv = x.shape[0], r.heads, r.groups, r.dim, r.vdim
    out = torch.empty(n, H * Dv, dtype=torch.float32, device=x.device)
    if x.is_cuda:
        _check(x)
        assert a.dtype == x.dtype and a.shape[1] == H and a.stride(1) == 1 and state.is_contiguous()
        args = RecurrenceArgs(q_col=cols[0], k_col=cols[1], v_col=cols[2], delta=3, a=a.data_ptr(), ld_a=a.stride(0), decay=r.rate.data_ptr(),
                              dt_bias=r.dt_bias.data_ptr(), skip=r.skip.data_ptr(), H=H, G=G, D=D, Dv=Dv)
        _run(args, x, seqs, pos, req, state, out, _runs_chunked(x, D, Dv, seqs, chunked))
        return out
    q, k, v = (x[:, c:c + h * d].float().reshape(n, h, d) for c, h, d in zip(cols, (G, G, H), (D, D, Dv)))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    dt = torch.nn.functional.softplus(a.float() + r.dt_bias, threshold=50.0)
    g, o = torch.exp(-r.rate * dt), out.view(n, H, Dv)
    for lo, count, at, slot in (seqs or Sequences.of_rows(pos, req)).host:
        S = state[slot].clone() if at > 0 else torch.zeros_like(state[slot])
        for i in range(lo, lo + count):
            S = S * g[i][:, None, None] + k[i][:, :, None] * (dt[i][:, None] * v[i])[:, None, :]
            o[i] = torch.einsum("hdv,hd->hv", S, q[i]) + r.skip[:, None] * v[i]
        state[slot] = S
    return out


# ------------------------------------------------------------------------------------------ output norm and gate
def group_norm_gate(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float, dtype, act: str = "sigmoid",
                    groups: Optional[int] = None, gate_first: bool = False) -> torch.Tensor:
    """``o [n, K]`` fp32 in groups of ``len(weight)`` columns: RMS norm of every group times the fp32 ``weight``, times the sigmoid (or
    ``act="silu"``) of ``gate [n, K]`` (any row pitch; bf16 or fp32).  With ``groups`` the weight is ``[K]`` and that many equal groups are normed;
    ``gate_first``: the gate multiplies ``o`` ahead of the norm.  Returns ``[n, K]`` in ``dtype``."""
    n, K = o.shape
    gs = K // groups if groups else weight.shape[0]
    assert K % gs == 0 and weight.shape[0] == (K if groups else gs)
    if o.is_cuda:
        out = torch.empty(n, K, dtype=dtype, device=o.device)
        assert o.is_contiguous() and gate.stride(1) == 1
        N.check(N.lib().ptb_group_norm_gate(o.data_ptr(), weight.data_ptr(), gate.data_ptr(), int(gate.dtype == torch.bfloat16), gate.stride(0),
                                            out.data_ptr(), n, K // gs, gs, float(eps), int(act == "silu"), int(gate_first), int(bool(groups)),
                                            int(dtype == torch.bfloat16), _st(o)), "group_norm_gate")
        return out
    g = (torch.nn.functional.silu if act == "silu" else torch.sigmoid)(gate.float())
    x = (o.float() * g if gate_first else o.float()).reshape(n, K // gs, gs)
    y = (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (weight.view(-1, gs) if groups else weight)).reshape(n, K)
    return (y if gate_first else y * g).to(dtype)
