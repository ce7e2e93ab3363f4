"""Ops around an fp32 residual stream (csrc/residual.cu, csrc/gemm_sm100.cu): embedding into it, a norm on a sublayer's output
followed by the sum, the sum followed by the next sublayer's norm, and the last norm over chosen rows.

The stream is a pair ``(x, xb)``: the fp32 sum and its copy in the compute type, which the projections read (the same tensor when
the compute type is fp32).  A norm's weight is a scale ``g``, a vector ``w``, or both.  CUDA tensors run the kernels; CPU tensors
take the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from .. import _native as N
from .gemm import _skinny_splits, linear
from .gemm import _status as _gemm_status
from .paged import _status

Stream = Tuple[torch.Tensor, torch.Tensor]


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_embed_residual.argtypes = [vp, ci, vp, ci, ci, cf, ci, vp, vp, vp, ci, vp]
    L.ptb_post_norm_add.argtypes = [vp, ll, vp, cf, cf, vp, vp, ci, ci, ci, vp]
    L.ptb_row_norm.argtypes = [vp, vp, ci, vp, cf, cf, vp, ci, ci, vp, ci, vp]
    L.ptb_gemm_bf16_splitk_f32.argtypes = [vp, ll, vp, ll, vp, ll, ci, ci, ci, ci, vp, vp, ci, vp]
    L.ptb_gemm_bf16_splitk_post_norm.argtypes = [vp, ll, vp, ll, ci, ci, ci, ci, vp, vp, cf, cf, vp, vp, vp, ci, vp]
    L.ptb_residual_norm.argtypes = [vp, vp, ci, ci, ll, ll, vp, cf, vp, ci, ci, ll, ll, vp, cf, cf, vp, vp, ci, ci, ci, vp, vp]
    for n in ("ptb_residual_norm", "ptb_embed_residual", "ptb_post_norm_add", "ptb_row_norm", "ptb_gemm_bf16_splitk_f32", "ptb_gemm_bf16_splitk_post_norm"):
        getattr(L, n).restype = ci


def _st(t):
    return torch.cuda.current_stream(t.device).cuda_stream


def _bf16(t) -> int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"the residual-stream kernels take bf16 or fp32, got {t.dtype}")
    return int(t.dtype == torch.bfloat16)


def _rms(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def embed_residual(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0, copy: bool = True) -> Stream:
    """``ids [n]`` int32 (any stride); ``table [V, W]`` in the compute type.  Without ``copy`` the stream is (x, x): for a decoder
    whose projections read a normalised row, never the stream itself."""
    n, (V, W) = ids.shape[0], table.shape
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        return x, (x if table.dtype == torch.float32 or not copy else x.to(table.dtype))
    x = torch.empty(n, W, dtype=torch.float32, device=table.device)
    xb = torch.empty(n, W, dtype=table.dtype, device=table.device) if _bf16(table) and copy else x
    N.check(N.lib().ptb_embed_residual(ids.data_ptr(), ids.stride(0), table.data_ptr(), V, W, float(scale), n, x.data_ptr(),
                                       xb.data_ptr() if xb is not x else 0, _status(x.device).data_ptr(), _bf16(table), _st(x)), "embed_residual")
    return x, xb


def post_norm_add(y: torch.Tensor, stream: Stream, g: float, eps: float, w: Optional[torch.Tensor] = None) -> Stream:
    """``x += y / rms(y) * g * w`` in place; returns the stream."""
    x, xb = stream
    if not y.is_cuda:
        v = _rms(y.float(), eps) * g
        x += v if w is None else v * w
        if xb is not x:
            xb.copy_(x)
        return stream
    n, W = x.shape
    assert x.is_contiguous() and xb.is_contiguous() and y.stride(1) == 1 and y.dtype == xb.dtype
    N.check(N.lib().ptb_post_norm_add(y.data_ptr(), y.stride(0), N.ptr(w), float(g), float(eps), x.data_ptr(), xb.data_ptr() if xb is not x else 0,
                                      n, W, _bf16(y), _st(y)), "post_norm_add")
    return stream


def linear_post_norm_add(a: torch.Tensor, weight: torch.Tensor, stream: Stream, g: float, eps: float, w: Optional[torch.Tensor] = None) -> Stream:
    """``y = a weight^T`` then :func:`post_norm_add`.  For decode-sized batches the sum of the split-K partials, the norm and the
    residual sum are one launch behind the product, and y stays in fp32."""
    x, xb = stream
    splits = _skinny_splits(a, weight)
    if splits and weight.shape[0] <= 8192 and xb is not x:
        M, K, Nn = a.shape[0], a.shape[1], weight.shape[0]
        work = torch.empty(splits * M * Nn, dtype=torch.float32, device=a.device)
        N.check(N.lib().ptb_gemm_bf16_splitk_post_norm(a.data_ptr(), a.stride(0), weight.data_ptr(), weight.stride(0), M, Nn, K, splits,
                                                       work.data_ptr(), N.ptr(w), float(g), float(eps), x.data_ptr(), xb.data_ptr(),
                                                       _gemm_status(a.device).data_ptr(), 0, _st(a)), "gemm_bf16_splitk_post_norm")
        return stream
    return post_norm_add(linear(a, weight), stream, g, eps, w)


def row_norm(stream: Stream, g: float, eps: float, w: Optional[torch.Tensor] = None, index: Optional[torch.Tensor] = None,
             dtype=None) -> torch.Tensor:
    """``x[index] / rms * g * w`` in the compute type (``index`` int64; None: every row), which is ``dtype`` or that of the copy."""
    x, xb = stream
    dtype = dtype or xb.dtype
    if not x.is_cuda:
        v = _rms(x if index is None else x[index], eps) * g
        return (v if w is None else v * w).to(dtype)
    m = x.shape[0] if index is None else index.shape[0]
    out = torch.empty(m, x.shape[1], dtype=dtype, device=x.device)
    N.check(N.lib().ptb_row_norm(x.data_ptr(), N.ptr(index), x.shape[0], N.ptr(w), float(g), float(eps), out.data_ptr(), m, x.shape[1],
                                 _status(x.device).data_ptr(), _bf16(out), _st(x)), "row_norm")
    return out


@dataclass
class Branch:
    """A sublayer's output on its way into the stream: ``y [n, W]``, or split-K partials ``[splits, n, W]`` fp32
    (:func:`linear_branch`), times ``g``; with ``w`` it is RMS-normed first."""
    y: torch.Tensor
    g: float = 1.0
    w: Optional[torch.Tensor] = None

    def parts(self) -> tuple:
        y = self.y
        if y.dim() == 3:
            return y.data_ptr(), 1, y.shape[0], y.stride(0), y.stride(1), N.ptr(self.w), float(self.g)
        return y.data_ptr(), int(y.dtype == torch.float32), 1, 0, y.stride(0), N.ptr(self.w), float(self.g)


def linear_branch(a: torch.Tensor, weight: torch.Tensor, g: float = 1.0, w: Optional[torch.Tensor] = None) -> Branch:
    """``a weight^T`` as a branch: decode-sized batches leave the split-K partials for :func:`residual_norm` to sum."""
    splits = _skinny_splits(a, weight)
    if not splits:
        return Branch(linear(a, weight), g, w)
    M, K, Nn = a.shape[0], a.shape[1], weight.shape[0]
    work = torch.empty(splits, M, Nn, dtype=torch.float32, device=a.device)
    real = N.lib().ptb_gemm_bf16_splitk_partials(a.data_ptr(), a.stride(0), weight.data_ptr(), weight.stride(0), M, Nn, K, splits, work.data_ptr(),
                                                 _gemm_status(a.device).data_ptr(), 0, _st(a))
    N.check(min(real, 0), "gemm_bf16_splitk_partials")
    return Branch(work[:real], g, w)


def residual_norm(x: torch.Tensor, branches: Sequence[Branch], eps: float, w: Optional[torch.Tensor] = None, dtype=None) -> Optional[torch.Tensor]:
    """``x += sum of the branches`` in place (fp32), then ``x / rms(x) * w`` in ``dtype`` (None without ``w``): the sum after a
    sublayer and the norm ahead of the next one in one launch.  At most two branches."""
    n, W = x.shape
    if not x.is_cuda:
        for b in branches:
            y = b.y.float()
            y = y.sum(0) if y.dim() == 3 else y
            x += (y if b.w is None else _rms(y, eps) * b.w) * b.g
        return None if w is None else (_rms(x, eps) * w).to(dtype or x.dtype)
    none = (0, 0, 0, 0, 0, 0, 0.0)
    p = [b.parts() for b in branches] + [none] * (2 - len(branches))
    out = torch.empty(n, W, dtype=dtype or x.dtype, device=x.device) if w is not None else None
    assert len(branches) <= 2 and x.is_contiguous() and x.dtype == torch.float32 and all(b.y.stride(-1) == 1 for b in branches)
    N.check(N.lib().ptb_residual_norm(x.data_ptr(), *p[0], *p[1], float(eps), N.ptr(w), N.ptr(out), n, W,
                                      _bf16(out) if out is not None else 0, _status(x.device).data_ptr(), _st(x)), "residual_norm")
    return out


def linear_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``x weight^T`` with an fp32 result (logits): the products of bf16 operands are not rounded on the way out."""
    if not (x.is_cuda and x.dtype == torch.bfloat16):
        return torch.nn.functional.linear(x.float(), weight.float())
    if x.shape[1] % 8 or weight.shape[0] % 8:                # operands the TMA kernel cannot address
        return torch.nn.functional.linear(x.float(), weight.float())
    M, K, Nn = x.shape[0], x.shape[1], weight.shape[0]
    out = torch.empty(M, Nn, dtype=torch.float32, device=x.device)
    splits = _skinny_splits(x, weight)
    if splits:
        work = torch.empty(splits * M * Nn, dtype=torch.float32, device=x.device)
        N.check(N.lib().ptb_gemm_bf16_splitk_f32(x.data_ptr(), x.stride(0), weight.data_ptr(), weight.stride(0), out.data_ptr(), Nn, M, Nn, K,
                                                 splits, work.data_ptr(), _gemm_status(x.device).data_ptr(), 0, _st(x)), "gemm_bf16_splitk_f32")
        return out
    from .gemm import gemm_bf16
    return gemm_bf16(x, weight, out=out)
