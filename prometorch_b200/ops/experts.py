"""A mixture of experts for inference (csrc/experts.cu, csrc/experts_sm100.cu): a router (sigmoid, or softmax over all its outputs) with a
correction that has a say in the choice only, and gated experts ``down (silu(gate h) * (up h))``, each token using ``top`` of them.  Router
outputs behind the experts are identities: they return the token's row itself.  A shared expert runs for every token: of a width near the
others' as more experts of the same grouped products (:meth:`Experts.of`), else by itself (:class:`SharedExpert`).

:func:`run` sorts the (token, expert) pairs by expert on the device, runs every expert over its rows (one grouped product for gate
and up, one for down) and returns :class:`ExpertRows`: the rows where they lie, their places and weights.  What sums them up is the kernel
that adds them to the stream (``ops/tanh_norm.py``, ``ops/streams.py``).  Nothing depends on the counts on the host, so a decode pass can be a CUDA graph.
CUDA tensors run the kernels, CPU tensors the plain math."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional

import torch

from .. import _native as N
from .paged import _status
from .gemm import linear_swiglu
from .residual import Branch, _st, linear_branch, linear_f32


@N.register_decls
def _decls(L):
    vp, ci, cf, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
    L.ptb_expert_route.argtypes = [vp, ci, ll, ll, vp, ci, ci, ci, ci, ci, ci, cf, vp, vp, vp, vp, vp, vp, vp]
    L.ptb_expert_gemm_simt.argtypes = [vp, vp, ll, vp, ci, vp, vp, ci, ci, ci, ci, ci, vp, vp]
    L.ptb_expert_gather.argtypes = [vp, ll, vp, vp, vp, ci, ci, ci, vp, vp]
    L.ptb_expert_gemm.argtypes = [vp, ll, vp, ci, vp, vp, ci, ci, ci, ci, ci, ci, vp, vp]
    L.ptb_expert_route_rows.argtypes = [vp, ll, vp, ci, vp, ci, ci, ci, ci, ci, ci, cf, vp, vp, vp, vp, vp, vp, ci, vp]
    for n in ("ptb_expert_route", "ptb_expert_route_rows", "ptb_expert_gemm_simt", "ptb_expert_gather", "ptb_expert_gemm"):
        getattr(L, n).restype = ci


@dataclass
class Experts:
    """One layer's experts in the layout the kernels read; ``ff`` is rounded up to a multiple of eight with zeros."""
    gate_up: torch.Tensor              # [E, 2 ff, W]: gate rows, then up rows
    down: torch.Tensor                 # [E, W, ff]
    router: torch.Tensor               # [outputs rounded up to eight, W]
    correction: torch.Tensor           # [outputs] fp32: the experts, then the identities
    top: int
    scale: float                       # sigmoid scores: weights are scores over the sum of the chosen ones, times scale; softmax: the scores times scale
    softmax: bool = False
    always: int = 0                    # the last experts, behind the routed ones: every token uses them, with the weight 1

    def __post_init__(self):
        self.done = torch.zeros(ROUTE_ROWS + 1, dtype=torch.int32, device=self.router.device)      # counters of the row router, zero between launches

    @property
    def count(self) -> int:
        return self.gate_up.shape[0]

    @property
    def routed(self) -> int:
        return self.count - self.always

    @property
    def width(self) -> int:
        """Experts of a token."""
        return self.top + self.always

    @property
    def outputs(self) -> int:
        return self.correction.shape[0]

    @classmethod
    def of(cls, gate: List[torch.Tensor], up: List[torch.Tensor], down: List[torch.Tensor], router: torch.Tensor, correction: torch.Tensor, top: int,
           scale: float, softmax: bool = False, shared: Optional[tuple] = None) -> "Experts":
        """``shared``: gate, up and down of an expert for every token, cut into experts of the others' width."""
        always = 0
        if shared is not None:
            ff, wide = gate[0].shape[0], shared[0].shape[0]
            always = -(-wide // ff)
            more = lambda t, d: list(torch.nn.functional.pad(t, (0, 0, 0, always * ff - wide) if d == 0 else (0, always * ff - wide)).split(ff, d))
            gate, up, down = gate + more(shared[0], 0), up + more(shared[1], 0), down + more(shared[2], 1)
        pad = lambda t, d: torch.nn.functional.pad(t, (0, 0, 0, -t.shape[0] % 8) if d == 0 else (0, -t.shape[1] % 8))
        return cls(torch.stack([torch.cat([pad(g, 0), pad(u, 0)]) for g, u in zip(gate, up)]), torch.stack([pad(t, 1) for t in down]), pad(router, 0).contiguous(),
                   correction.float().contiguous(), top, scale, softmax, always)


@dataclass
class ExpertRows:
    """Outputs of the chosen experts: row ``index[t, i]`` of ``y`` belongs to token t with the weight ``weight[t, i]``; where the index is -1 it is the
    token's own row of ``h``."""
    y: torch.Tensor                    # [n top, W], sorted by expert
    index: torch.Tensor                # [n, top] int32
    weight: torch.Tensor               # [n, top] fp32
    h: Optional[torch.Tensor] = None   # [n, W] what the experts read

    def combine(self) -> torch.Tensor:
        i = self.index.long()
        if self.h is None:
            return (self.y.float()[i] * self.weight[..., None]).sum(1)
        rows = torch.where((i < 0)[..., None], self.h.float()[:, None, :], self.y.float()[i.clamp_min(0)])
        return (rows * self.weight[..., None]).sum(1)


@dataclass
class Routing:
    index: torch.Tensor                # [n, top] int32: place of every pair in the order by expert
    weight: torch.Tensor               # [n, top] fp32
    token: torch.Tensor                # [n top] int32: the token of every place
    offsets: torch.Tensor              # [E + 1] int32: first place of every expert


ROUTE_ROWS = 64                        # tokens up to which the kernel that chooses forms the logits as well


def route(h: torch.Tensor, e: Experts) -> Routing:
    n, E, O, k, W = h.shape[0], e.routed, e.outputs, e.width, h.shape[1]
    if h.is_cuda:
        i32 = lambda *s: torch.empty(*s, dtype=torch.int32, device=h.device)
        r = Routing(i32(n, k), torch.empty(n, k, dtype=torch.float32, device=h.device), i32(n * k), i32(e.count + 1))
        few = n <= ROUTE_ROWS and O * W <= 1 << 21
        work = i32(2 * n * k + (n * O if few else E))
        out = (r.index.data_ptr(), r.weight.data_ptr(), r.token.data_ptr(), r.offsets.data_ptr(), work.data_ptr())
        if few:
            assert h.dtype == e.router.dtype and h.stride(1) == 1
            N.check(N.lib().ptb_expert_route_rows(h.data_ptr(), h.stride(0), e.router.data_ptr(), W, e.correction.data_ptr(), n, E, O, e.always, int(e.softmax), e.top, float(e.scale), *out,
                                                  e.done.data_ptr(), int(h.dtype == torch.bfloat16), _st(h)), "expert_route_rows")
            return r
        z = linear_f32(h, e.router)
        N.check(N.lib().ptb_expert_route(z.data_ptr(), 1, 0, z.stride(0), e.correction.data_ptr(), n, E, O, e.always, int(e.softmax), e.top, float(e.scale), *out, _status(h.device).data_ptr(), _st(h)),
                "expert_route")
        return r
    z = linear_f32(h, e.router)
    s = torch.softmax(z[:, :O], -1) if e.softmax else torch.sigmoid(z[:, :O])
    chosen = torch.topk(s + e.correction, e.top, -1).indices
    w = s.gather(1, chosen)
    w = w * e.scale if e.softmax else w / (w.sum(-1, keepdim=True) + 1e-20) * e.scale
    chosen = torch.where(chosen < E, chosen, e.count)            # identities last
    chosen = torch.cat([chosen, torch.arange(E, e.count).expand(n, e.always)], 1)
    w = torch.cat([w, w.new_ones(n, e.always)], 1)
    order = torch.sort(chosen.flatten(), stable=True).indices
    index = torch.empty_like(order)
    index[order] = torch.arange(n * k)
    index[chosen.flatten() == e.count] = -1
    offsets = torch.cat([torch.zeros(1, dtype=torch.long), torch.bincount(chosen.flatten(), minlength=e.count)[:e.count].cumsum(0)])
    return Routing(index.view(n, k).int(), w, (order // k).int(), offsets.int())


GATED_FROM = 128                       # rows above which the shared expert runs as a grouped product of one expert
FEW_ROWS = 48                          # mean rows of an expert below which its weights are the 128-row operand


def products(h: torch.Tensor, e: Experts, r: Routing, simt: bool = False) -> torch.Tensor:
    """The experts over their rows: ``[n top, W]`` in the order by expert.  bf16 rows of a multiple of eight go to the tensor cores;
    everything else, or all with ``simt``, to the kernel that takes any size."""
    n, W = h.shape
    rows, F, E = n * e.width, e.down.shape[2], e.count
    if h.is_cuda:
        bf16, st, status = h.dtype == torch.bfloat16, _st(h), _status(h.device).data_ptr()
        act, y = torch.empty(rows, F, dtype=h.dtype, device=h.device), torch.empty(rows, W, dtype=h.dtype, device=h.device)
        assert h.stride(1) == 1 and e.gate_up.dtype == h.dtype
        if bf16 and W % 8 == 0 and h.stride(0) % 8 == 0 and not simt:
            x = torch.empty(rows, W, dtype=h.dtype, device=h.device)
            few = int(rows < FEW_ROWS * E)
            N.check(N.lib().ptb_expert_gather(h.data_ptr(), h.stride(0), r.token.data_ptr(), r.offsets[E:].data_ptr(), x.data_ptr(), rows, W, n, status, st), "expert_gather")
            N.check(N.lib().ptb_expert_gemm(x.data_ptr(), W, e.gate_up.data_ptr(), 1, act.data_ptr(), r.offsets.data_ptr(), rows, E, F, W, few, 0, status, st), "expert_gemm")
            N.check(N.lib().ptb_expert_gemm(act.data_ptr(), F, e.down.data_ptr(), 0, y.data_ptr(), r.offsets.data_ptr(), rows, E, W, F, few, 0, status, st), "expert_gemm")
            return y
        N.check(N.lib().ptb_expert_gemm_simt(h.data_ptr(), r.token.data_ptr(), h.stride(0), e.gate_up.data_ptr(), 1, act.data_ptr(), r.offsets.data_ptr(), rows, E, F, W,
                                             int(bf16), status, st), "expert_gemm_simt")
        N.check(N.lib().ptb_expert_gemm_simt(act.data_ptr(), 0, F, e.down.data_ptr(), 0, y.data_ptr(), r.offsets.data_ptr(), rows, E, W, F, int(bf16), status, st),
                "expert_gemm_simt")
        return y
    x, at = h.float()[r.token.long()], r.offsets.tolist()
    y = torch.zeros(rows, W)
    for i in range(E):
        lo, hi = at[i], at[i + 1]
        if lo < hi:
            g, u = (x[lo:hi] @ e.gate_up[i].float().t()).split([F, F], -1)
            y[lo:hi] = (torch.nn.functional.silu(g) * u) @ e.down[i].float().t()
    return y.to(h.dtype)


def run(h: torch.Tensor, e: Experts) -> ExpertRows:
    """``h [n, W]`` through its tokens' experts."""
    r = route(h, e)
    return ExpertRows(products(h, e, r), r.index, r.weight, h)


SHARED_PARTS = 2                       # a shared expert of at most this many times the others' width joins their grouped products


@dataclass
class SharedExpert:
    """A gated expert that every token uses; ``ff`` is rounded up to a multiple of eight with zeros."""
    gate_up: torch.Tensor              # [2 ff, W]: gate rows, then up rows
    down: torch.Tensor                 # [W rounded up to eight, ff]

    @classmethod
    def of(cls, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> "SharedExpert":
        pad = lambda t: torch.nn.functional.pad(t, (0, 0, 0, -t.shape[0] % 8))
        return cls(torch.cat([pad(gate), pad(up)]), pad(torch.nn.functional.pad(down, (0, -down.shape[1] % 8))))


def run_shared(h: torch.Tensor, e: SharedExpert) -> Branch:
    """``h [n, W]`` through the shared expert, as a branch for the kernel that adds it to the stream."""
    n, W = h.shape
    F = e.down.shape[1]
    if h.is_cuda and h.dtype == torch.bfloat16 and n > GATED_FROM and W % 8 == 0 and h.stride(0) % 8 == 0:
        act = torch.empty(n, F, dtype=h.dtype, device=h.device)
        offsets = torch.arange(0, n + 1, n, dtype=torch.int32, device=h.device)          # [0, n]
        N.check(N.lib().ptb_expert_gemm(h.data_ptr(), h.stride(0), e.gate_up.data_ptr(), 1, act.data_ptr(), offsets.data_ptr(), n, 1, F, W, 0, 0,
                                        _status(h.device).data_ptr(), _st(h)), "expert_gemm")
    else:
        act = linear_swiglu(h, e.gate_up)
    return linear_branch(act, e.down)
