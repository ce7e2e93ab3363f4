"""Elementwise norms (dynamic tanh: ``tanh(alpha x) w + b``, no statistics of the row) around an fp32 residual stream, and the soft cap
of the logits (csrc/tanh_norm.cu).

:func:`residual` is what stands between two sublayers, in one launch: the norm on a sublayer's output, the sum, and the norm ahead of
the next one.  The output comes as a :class:`~prometorch_b200.ops.residual.Branch` (a product, or its split-K partials) or as the rows of
a mixture of experts, which are weighed and summed on the way.  CUDA tensors run the kernels, CPU tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch

from .. import _native as N
from .experts import ExpertRows
from .paged import _status
from .residual import Branch, _bf16, _st


@dataclass
class TanhNorm:
    alpha: float
    w: torch.Tensor                    # [W] fp32
    b: torch.Tensor                    # [W] fp32

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return torch.tanh(x * self.alpha) * self.w + self.b

    def parts(self) -> tuple:
        return float(self.alpha), self.w.data_ptr(), self.b.data_ptr()


class TanhResidualArgs(C.Structure):
    """``PtbTanhResidual`` of csrc/ptb200_types.h."""
    _fields_ = [("x", C.c_void_p), ("y", C.c_void_p), ("f32", C.c_int), ("splits", C.c_int), ("stride", C.c_longlong), ("ld", C.c_longlong),
                ("index", C.c_void_p), ("weight", C.c_void_p), ("top", C.c_int), ("y_rows", C.c_int),
                ("post_alpha", C.c_float), ("pre_alpha", C.c_float), ("post_w", C.c_void_p), ("post_b", C.c_void_p), ("pre_w", C.c_void_p),
                ("pre_b", C.c_void_p), ("ids", C.c_void_p), ("id_stride", C.c_int), ("V", C.c_int), ("table", C.c_void_p),
                ("out", C.c_void_p), ("n", C.c_int), ("W", C.c_int), ("bf16", C.c_int), ("pad", C.c_int), ("status", C.c_void_p)]


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_tanh_residual.argtypes = [C.POINTER(TanhResidualArgs), vp]
    L.ptb_tanh_rows.argtypes = [vp, vp, ci, cf, vp, vp, vp, ci, ci, vp, ci, vp]
    L.ptb_softcap.argtypes = [vp, vp, ci, ci, ll, cf, vp]
    for n in ("ptb_tanh_residual", "ptb_tanh_rows", "ptb_softcap"):
        getattr(L, n).restype = ci


def rows(x: torch.Tensor, norm: TanhNorm, index: Optional[torch.Tensor] = None, dtype=torch.float32) -> torch.Tensor:
    """``norm(x[index])`` in ``dtype`` (``index`` int64; None: every row)."""
    if not x.is_cuda:
        return norm(x if index is None else x[index]).to(dtype)
    m = x.shape[0] if index is None else index.shape[0]
    out = torch.empty(m, x.shape[1], dtype=dtype, device=x.device)
    N.check(N.lib().ptb_tanh_rows(x.data_ptr(), N.ptr(index), x.shape[0], *norm.parts(), out.data_ptr(), m, x.shape[1], _status(x.device).data_ptr(),
                                  _bf16(out), _st(x)), "tanh_rows")
    return out


def residual(x: torch.Tensor, y: Union[Branch, ExpertRows], post: TanhNorm, pre: Optional[TanhNorm], dtype=torch.float32,
             again: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> Optional[torch.Tensor]:
    """``x += post(y)`` in place (fp32), then, with ``again = (ids, table)``, ``x += table[ids]``; returns ``pre(x)`` in ``dtype`` (None
    without ``pre``)."""
    n, W = x.shape
    if not x.is_cuda:
        if isinstance(y, ExpertRows):
            f = y.combine()
        else:
            f = (y.y.float().sum(0) if y.y.dim() == 3 else y.y.float()) * y.g
        x += post(f)
        if again is not None:
            x += again[1][again[0].long()].float()
        return None if pre is None else pre(x).to(dtype)
    out = torch.empty(n, W, dtype=dtype, device=x.device) if pre is not None else None
    a = TanhResidualArgs(x=x.data_ptr(), n=n, W=W, bf16=int(dtype == torch.bfloat16), status=_status(x.device).data_ptr(), out=N.ptr(out))
    if isinstance(y, ExpertRows):
        a.y, a.f32, a.splits, a.ld = y.y.data_ptr(), int(y.y.dtype == torch.float32), 1, y.y.stride(0)
        a.index, a.weight, a.top, a.y_rows = y.index.data_ptr(), y.weight.data_ptr(), y.index.shape[1], y.y.shape[0]
    else:
        assert y.w is None and y.g == 1.0
        a.y, a.f32, a.splits, a.stride, a.ld = y.parts()[:5]
    assert x.is_contiguous() and x.dtype == torch.float32 and y.y.stride(-1) == 1
    a.post_alpha, a.post_w, a.post_b = post.parts()
    if pre is not None:
        a.pre_alpha, a.pre_w, a.pre_b = pre.parts()
    if again is not None:
        ids, table = again
        assert table.is_contiguous() and table.dtype == dtype
        a.ids, a.id_stride, a.table, a.V = ids.data_ptr(), ids.stride(0), table.data_ptr(), table.shape[0]
    N.check(N.lib().ptb_tanh_residual(C.byref(a), _st(x)), "tanh_residual")
    return out


def softcap(z: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap tanh(z / cap)`` of fp32 logits ``[m, V]`` (any row pitch)."""
    if not z.is_cuda:
        return torch.tanh(z / cap) * cap
    out = torch.empty(z.shape, dtype=torch.float32, device=z.device)
    assert z.dtype == torch.float32 and z.stride(1) == 1
    N.check(N.lib().ptb_softcap(z.data_ptr(), out.data_ptr(), z.shape[0], z.shape[1], z.stride(0), float(cap), _st(z)), "softcap")
    return out
