"""FP32 residual stream. Parallel layers (:func:`embed`, :func:`step`): the sums a layer ends with, and the one or two norms the next
one starts with, in one kernel. Sequential layers with norms on both sides of a sub-layer (:func:`embed_normed`, :func:`add_normed`):
the norm behind one sub-layer, the sum and the norm in front of the next. CUDA: ``csrc/residual.cu``; CPU: FP32 arithmetic on the same
layouts.

The stream is FP32 ``[rows, width]``; norm weights are FP32 vectors with any offset already added; ``true_width`` is the width the
norms divide by where ``width`` carries padding. A layer may have a second mixer beside the first, each normed on its way into the sum
(:class:`Beside`), and tokens a second embedding that depends on the token before (:func:`bigram_rows`, :class:`Second`)."""
from __future__ import annotations

from ctypes import c_float, c_longlong
from dataclasses import dataclass

import torch

from . import _count, _require
from .lib import check, kernels, ptr, status_tensor, stream_ptr
from .moe_ops import ExpertRows


def _norms(x: torch.Tensor, w1: torch.Tensor, w2: torch.Tensor | None, eps: float, true_width: int, dtype) -> tuple:
    n = x * torch.rsqrt((x * x).sum(-1, keepdim=True) / true_width + eps)
    return (n * w1).to(dtype), None if w2 is None else (n * w2).to(dtype)


def _outputs(x: torch.Tensor, w1: torch.Tensor, w2: torch.Tensor | None, dtype) -> tuple:
    for w in (w1, w2):
        _require(w is None or (w.dtype == torch.float32 and w.numel() == x.shape[1] and w.is_contiguous()), "residual norms: FP32 weights")
    new = lambda: torch.empty(x.shape, dtype=dtype, device=x.device)
    return new(), None if w2 is None else new()


@dataclass
class Second:
    """A second embedding table, its row per row of the batch, and the FP32 weight of the norm of the sum of both."""
    table: torch.Tensor
    rows: torch.Tensor
    w: torch.Tensor


@dataclass
class Beside:
    """Rows of a second mixer and the FP32 weights of the norms of the first and the second."""
    a: torch.Tensor
    w_first: torch.Tensor
    w: torch.Tensor


def bigram_rows(ids: torch.Tensor, last: torch.Tensor, row_start: torch.Tensor, slots: torch.Tensor, buckets: int, mul_prev: int, mul_cur: int
                ) -> torch.Tensor:
    """int32 ``(previous token * mul_prev + token * mul_cur) % buckets`` per row, ``buckets`` for a sequence's first token. ``last``
    [slots] int32: the token before a sequence's next one, negative at its start; takes the batch's last tokens."""
    out = torch.empty(ids.numel(), dtype=torch.int32, device=ids.device)
    if not ids.is_cuda:
        for s in range(slots.numel()):
            r0, r1, slot = int(row_start[s]), int(row_start[s + 1]), int(slots[s])
            prev = int(last[slot])
            for r in range(r0, r1):
                t = int(ids[r])
                out[r] = buckets if prev < 0 else (prev * mul_prev + t * mul_cur) % buckets
                prev = t
            if r1 > r0:
                last[slot] = prev
        return out
    _require(ids.dtype == last.dtype == row_start.dtype == slots.dtype == torch.int32 and row_start.numel() == slots.numel() + 1, "bigram_rows: int32 metadata")
    check(kernels().ff_bigram_rows(ptr(ids), ptr(out), ptr(last), ptr(row_start), ptr(slots), slots.numel(), buckets, c_longlong(mul_prev),
                                   c_longlong(mul_cur), stream_ptr()), "ff_bigram_rows")
    _count()
    return out


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float, w1: torch.Tensor, w2: torch.Tensor | None, eps: float,
          true_width: int, second: Second | None = None) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor | None]:
    """(stream ``table[ids] * scale``, its norm times ``w1``, its norm times ``w2``). ``second``: the stream is the norm of the sum with
    another table's rows."""
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        if second is not None:
            x = _norms(x + second.table[second.rows.long()].float(), second.w, None, eps, true_width, torch.float32)[0]
        return (x,) + _norms(x, w1, w2, eps, true_width, table.dtype)
    rows, (vocab, width) = ids.numel(), table.shape
    _require(ids.dtype == torch.int32 and table.is_contiguous() and width % 8 == 0, "residual embed: int32 ids, rows of 8 elements")
    x = torch.empty(rows, width, dtype=torch.float32, device=table.device)
    n1, n2 = _outputs(x, w1, w2, table.dtype)
    e = (None, None, 0, None)
    if second is not None:
        _require(second.table.dtype == table.dtype and second.table.is_contiguous() and second.table.shape[1] == width and
                 second.rows.dtype == torch.int32 and second.rows.numel() == rows, "residual embed: second table")
        e = (ptr(second.table), ptr(second.rows), second.table.shape[0], ptr(second.w))
    rc = kernels().ff_residual_embed(ptr(ids), ptr(table), c_float(scale), *e, ptr(x), ptr(w1), ptr(w2), ptr(n1), ptr(n2), rows, width, true_width,
                                     vocab, c_float(eps), int(table.dtype == torch.float32), ptr(status_tensor(table.device)), stream_ptr())
    check(rc, "ff_residual_embed")
    _count()
    return x, n1, n2


def step(x: torch.Tensor, a: torch.Tensor, b: torch.Tensor | None, experts: ExpertRows | None, w1: torch.Tensor, w2: torch.Tensor | None,
         eps: float, true_width: int, beside: Beside | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """``x += a + b + (weighted sum of the experts' rows)`` in place; returns the norms as :func:`embed` does. ``beside``: in place of
    ``a`` the norm of ``a`` and the norm of a second mixer's rows, each with its weight."""
    if not x.is_cuda:
        if beside is None:
            x += a.float()
        else:
            x += _norms(a.float(), beside.w_first, None, eps, true_width, torch.float32)[0] + \
                _norms(beside.a.float(), beside.w, None, eps, true_width, torch.float32)[0]
        if b is not None:
            x += b.float()
        if experts is not None:
            x += experts.total()
        return _norms(x, w1, w2, eps, true_width, a.dtype)
    rows, width = x.shape
    _require(x.dtype == torch.float32 and x.is_contiguous() and width % 8 == 0, "residual step: FP32 rows of 8 elements")
    ok = lambda t: t is None or (t.shape == x.shape and t.is_contiguous() and t.dtype == a.dtype)
    _require(ok(a) and ok(b) and (beside is None or ok(beside.a)) and (experts is None or ok(experts.h)), "residual step: rows of one type")
    n1, n2 = _outputs(x, w1, w2, a.dtype)
    e, top, ldy, first = experts, 0, 0, 0
    if e is not None:
        top, ldy, first = e.ids.shape[1], e.y.stride(0), e.experts
        _require(e.y.dtype == a.dtype and e.ids.is_contiguous() and e.weights.is_contiguous() and e.weights.dtype == torch.float32 and
                 e.ids.dtype == e.pos.dtype == torch.int32, "residual step: expert rows")
    g = lambda name: None if e is None else getattr(e, name)
    two = (None, None, None) if beside is None else (ptr(beside.a), ptr(beside.w_first), ptr(beside.w))
    rc = kernels().ff_residual_step(ptr(x), ptr(a), *two, ptr(b), ptr(g("y")), ptr(g("pos")), ptr(g("ids")), ptr(g("weights")), ptr(g("h")), top,
                                    first, ldy, ptr(w1), ptr(w2), ptr(n1), ptr(n2), rows, width, true_width, c_float(eps),
                                    int(a.dtype == torch.float32), stream_ptr())
    check(rc, "ff_residual_step")
    _count()
    return n1, n2


# ------------------------------------------------------------------------------------------
# norms on both sides of a sub-layer
# ------------------------------------------------------------------------------------------
@dataclass
class Norm:
    """``kind`` "rms": ``x / rms(x) * w``; "tanh": ``tanh(alpha x) * w + b``; "copy": the row in the operand type. FP32 vectors."""
    kind: str = "copy"
    w: torch.Tensor | None = None
    b: torch.Tensor | None = None
    alpha: float = 0.0

    KINDS = {"copy": 0, "rms": 1, "tanh": 2}

    def __call__(self, x: torch.Tensor, eps: float, true_width: int) -> torch.Tensor:
        """FP32 rows normed (the oracle)."""
        if self.kind == "rms":
            return x * torch.rsqrt((x * x).sum(-1, keepdim=True) / true_width + eps) * self.w
        return torch.tanh(self.alpha * x) * self.w + self.b if self.kind == "tanh" else x

    def args(self, width: int) -> tuple:
        for v in (self.w, self.b):
            _require(v is None or (v.dtype == torch.float32 and v.numel() == width and v.is_contiguous()), "norm: FP32 vectors of the width")
        return self.KINDS[self.kind], ptr(self.w), ptr(self.b), c_float(self.alpha)


def embed_normed(ids: torch.Tensor, table: torch.Tensor, scale: float, outer: Norm, eps: float, true_width: int
                 ) -> tuple[torch.Tensor, torch.Tensor]:
    """(FP32 stream ``table[ids] * scale``, its norm)."""
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        return x, outer(x, eps, true_width).to(table.dtype)
    rows, (vocab, width) = ids.numel(), table.shape
    _require(ids.dtype == torch.int32 and table.is_contiguous() and width % 8 == 0, "residual embed: int32 ids, rows of 8 elements")
    x = torch.empty(rows, width, dtype=torch.float32, device=table.device)
    n = torch.empty(rows, width, dtype=table.dtype, device=table.device)
    rc = kernels().ff_residual_embed_normed(ptr(ids), ptr(table), c_float(scale), ptr(x), *outer.args(width), ptr(n), rows, width, true_width,
                                            vocab, c_float(eps), int(table.dtype == torch.float32), ptr(status_tensor(table.device)), stream_ptr())
    check(rc, "ff_residual_embed_normed")
    _count()
    return x, n


def add_normed(x: torch.Tensor, y: torch.Tensor, inner: Norm, outer: Norm, eps: float, true_width: int) -> torch.Tensor:
    """``x += inner(y)`` in place (FP32); returns ``outer(x)`` in the type of ``y``."""
    if not x.is_cuda:
        x += inner(y.float(), eps, true_width)
        return outer(x, eps, true_width).to(y.dtype)
    rows, width = x.shape
    _require(x.dtype == torch.float32 and x.is_contiguous() and width % 8 == 0, "residual step: FP32 rows of 8 elements")
    _require(y.shape == x.shape and y.is_contiguous(), "residual step: rows of the stream's shape")
    n = torch.empty(rows, width, dtype=y.dtype, device=x.device)
    rc = kernels().ff_residual_add_normed(ptr(x), ptr(y), *inner.args(width), *outer.args(width), ptr(n), rows, width, true_width, c_float(eps),
                                          int(y.dtype == torch.float32), stream_ptr())
    check(rc, "ff_residual_add_normed")
    _count()
    return n
