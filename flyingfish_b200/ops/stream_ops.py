"""Residual streams with fixed hyper-connections (input-independent coefficients; ``mhc_ops`` has the form whose
coefficients are computed from the streams). CUDA: ``csrc/streams.cu``; CPU: FP32 arithmetic on the same layouts.

The streams are FP32, ``[rows, S, width]``. ``coef`` packs ``[read of the next sub-layer (S) | write (S) | matrix (S x S,
from x to)]``; ``true_width`` is the width the norm divides by where ``width`` carries padding."""
from __future__ import annotations

from ctypes import c_float

import torch

from . import _count, _require
from .lib import check, kernels, ptr, status_tensor, stream_ptr

MAX_STREAMS = 16


def _norm(u: torch.Tensor, w: torch.Tensor, eps: float, true_width: int) -> torch.Tensor:
    r = torch.rsqrt((u * u).sum(-1, keepdim=True) / true_width + eps)
    return (u * r * w.float()).to(w.dtype)


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float, read: torch.Tensor, norm_w: torch.Tensor, eps: float,
          true_width: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Every stream = ``table[ids] * scale``; returns (streams, ``rmsnorm(sum_s read_s x_s) * norm_w``)."""
    rows, streams = ids.numel(), read.numel()
    vocab, width = table.shape
    if not table.is_cuda:
        e = table[ids.long()].float() * scale
        x = e[:, None].repeat(1, streams, 1).contiguous()
        return x, _norm(torch.einsum("rsw,s->rw", x, read), norm_w, eps, true_width)
    _require(ids.dtype == torch.int32 and table.is_contiguous() and width % 8 == 0, "stream embed: int32 ids, rows of 8 elements")
    _require(norm_w.dtype == table.dtype and norm_w.numel() == width, "stream embed: norm weight")
    x = torch.empty(rows, streams, width, dtype=torch.float32, device=table.device)
    n = torch.empty(rows, width, dtype=table.dtype, device=table.device)
    rc = kernels().ff_stream_embed(ptr(ids), ptr(table), c_float(scale), ptr(read), ptr(norm_w), ptr(x), ptr(n), rows, streams, width,
                                   true_width, vocab, c_float(eps), int(table.dtype == torch.float32), ptr(status_tensor(table.device)),
                                   stream_ptr())
    check(rc, "ff_stream_embed")
    _count()
    return x, n


def step(x: torch.Tensor, y: torch.Tensor, scale: torch.Tensor, coef: torch.Tensor, norm_w: torch.Tensor, eps: float,
         true_width: int, write: bool = True) -> torch.Tensor:
    """``x_t <- sum_s M[s, t] x_s + b_t (y * scale)`` in place (``write``), then ``rmsnorm(sum_t a_t x_t) * norm_w``."""
    rows, streams, width = x.shape
    if not x.is_cuda:
        a, b, m = coef[:streams], coef[streams: 2 * streams], coef[2 * streams:].view(streams, streams)
        new = torch.einsum("st,rsw->rtw", m, x) + b[None, :, None] * (y.float() * scale.float())[:, None]
        if write:
            x.copy_(new)
        return _norm(torch.einsum("rsw,s->rw", new, a), norm_w, eps, true_width)
    _require(x.dtype == torch.float32 and x.is_contiguous() and width % 8 == 0, "stream step: FP32 streams, rows of 8 elements")
    _require(y.shape == (rows, width) and y.is_contiguous() and y.dtype == scale.dtype == norm_w.dtype, "stream step: operand types")
    _require(coef.numel() == streams * (streams + 2) and coef.dtype == torch.float32, "stream step: coefficient table")
    n = torch.empty(rows, width, dtype=y.dtype, device=y.device)
    rc = kernels().ff_stream_step(ptr(x), ptr(y), ptr(scale), ptr(coef), ptr(norm_w), ptr(n), rows, streams, width, true_width, c_float(eps),
                                  int(y.dtype == torch.float32), int(write), stream_ptr())
    check(rc, "ff_stream_step")
    _count()
    return n
