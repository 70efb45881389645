"""MoE operators: router, expert FFNs over routed rows, deterministic combine.

CPU tensors run the oracles in :mod:`flyingfish_b200.ops.ref`. CUDA tensors run the sm_100a
kernels of ``csrc/moe.cu``: one router kernel (logits + deterministic top-k for softmax /
sigmoid / grouped no-aux scoring), a device-side count/scan/permute that needs no host sync
(the reference reads the per-expert counts back to the host, src/backend/cuda/moe/prefill.rs:1137),
a grouped tcgen05 GEMM over the expert segments with SwiGLU in the epilogue, and a combine that
sums contributions in ascending expert id.
"""
from __future__ import annotations

import ctypes
from ctypes import c_float

import torch

from . import ref
from .lib import check, kernels, ptr, status_tensor, stream_ptr


def route(x: torch.Tensor, w_router: torch.Tensor, top_k: int, score: str = "softmax",
          bias: torch.Tensor | None = None, n_groups: int = 1, topk_groups: int = 1, routed_scaling: float = 1.0,
          renormalize: bool = True, exact: bool = False, experts: int | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """Returns (weights fp32 [rows, k], expert ids int32 [rows, k]). ``exact``: the logits stay in FP32 (otherwise they are
    rounded to the activations' type). ``experts``: rows of ``w_router`` that count, where it carries padding."""
    if not x.is_cuda:
        w = w_router[:experts] if experts is not None else w_router
        return ref.moe_route(x, w, top_k, score, bias, n_groups, topk_groups, routed_scaling, renormalize, torch.float32 if exact else None)
    from . import moe_cuda
    return moe_cuda.route(x, w_router, top_k, score, bias, n_groups, topk_groups, routed_scaling, renormalize, exact, experts)


class ExpertRows:
    """What the routed experts of a batch leave behind for the kernel that sums them (``residual_ops.step``): their output rows,
    the row of every choice (negative: none), the choices and weights, and the experts' input (the output of an identity
    choice: an id from ``experts`` on)."""

    def __init__(self, y, pos, ids, weights, h, experts: int):
        self.y, self.pos, self.ids, self.weights, self.h, self.experts = y, pos, ids, weights, h, experts

    def total(self) -> torch.Tensor:
        """The weighted sum in FP32 (CPU)."""
        out = torch.zeros(self.h.shape, dtype=torch.float32)
        for j in range(self.ids.shape[1]):
            ident = self.ids[:, j] >= self.experts
            row = torch.where(ident[:, None], self.h.float(), self.y[self.pos.view(self.ids.shape)[:, j].clamp(min=0).long()].float())
            out += self.weights[:, j, None] * row
        return out


def expert_rows(x: torch.Tensor, weights: torch.Tensor, ids: torch.Tensor, gu: torch.Tensor, down: torch.Tensor, limit: float = 0.0) -> ExpertRows:
    """SwiGLU experts on the rows that chose them, without the final sum. ``gu`` [E, 2f, h] with gate / up rows interleaved per
    64, ``down`` [E, h, f]; ids from ``E`` on are not served here (identity outputs). ``limit > 0``: the clamped gate (``ref.silu_mul`` mode 5) in place of SiLU.
    BF16 or FP32."""
    if x.is_cuda:
        from . import moe_cuda
        return moe_cuda.expert_rows(x, weights, ids, gu, down, limit)
    e = gu.shape[0]
    y = torch.zeros(ids.numel(), x.shape[1], dtype=x.dtype)
    pos = torch.where(ids < e, torch.arange(ids.numel()).view(ids.shape), -1).reshape(-1)
    for k in range(e):
        r, c = torch.nonzero(ids == k, as_tuple=True)
        if r.numel():
            y[r * ids.shape[1] + c] = ref.linear(ref.linear_swiglu(x[r], gu[k], 5 if limit else 0, limit), down[k])
    return ExpertRows(y, pos, ids, weights, x, e)


def experts_forward(x: torch.Tensor, weights: torch.Tensor, ids: torch.Tensor, w_gate_up: torch.Tensor,
                    w_down: torch.Tensor, mode: int = 0) -> torch.Tensor:
    """Weighted sum of the selected experts' SwiGLU FFNs for every row (no shared expert)."""
    if not x.is_cuda:
        return ref.moe_forward(x, weights, ids, w_gate_up, w_down, None, None, mode)
    from . import moe_cuda
    return moe_cuda.experts_forward(x, weights, ids, w_gate_up, w_down, mode)


def add_shared(routed: torch.Tensor, shared: torch.Tensor) -> torch.Tensor:
    """Adds the shared expert's output in the storage dtype (one rounding)."""
    if not routed.is_cuda:
        return (routed.to(torch.float32) + shared.to(torch.float32)).to(routed.dtype)
    from . import residual_add
    return residual_add(routed, shared)


def routed_rows(x: torch.Tensor, w_router: torch.Tensor, top_k: int, score: str, bias: torch.Tensor | None, outputs: int, gu: torch.Tensor,
                down: torch.Tensor, limit: float = 0.0) -> ExpertRows:
    """:func:`route` with FP32 logits over the first ``outputs`` rows of ``w_router`` and renormalised weights, then
    :func:`expert_rows`."""
    if x.is_cuda:
        from . import moe_cuda
        return moe_cuda.routed_rows(x, w_router, top_k, score, bias, outputs, gu, down, limit)
    weights, ids = route(x, w_router, top_k, score, bias, exact=True, experts=outputs)
    return expert_rows(x, weights, ids, gu, down, limit)
