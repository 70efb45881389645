"""State-space recurrence of Mamba-2 (scalar decay per head, input and output maps shared by groups of heads) over packed rows of several
sequences, its state addressed by slot. CUDA: the scalar-gate kernels of ``csrc/mlstm.cu`` (token by token for decoding and 32-bit
prompts, 64 tokens at a time for BF16 prompts); CPU: the recurrence in FP32. The convolution in front: :func:`delta_ops.short_conv`.

Packed rows hold ``[C groups | B groups | x heads]``, ``dk`` / ``dv`` wide (multiples of 16, zeros behind a group's or head's own
elements)."""
from __future__ import annotations

from ctypes import c_float

import torch

from . import _count, _require, workspace
from .lib import check, kernels, ptr, stream_ptr
from .mlstm_ops import CHUNK_MAX_KEY, CHUNK_MIN_ROWS, FILL_CTAS, SEGMENT_ROWS, TILE


class SsdState:
    """S [slots, heads, dk, dv] of one layer, FP32, zero at the start of a sequence."""

    def __init__(self, slots: int, heads: int, groups: int, dk: int, dv: int, device):
        self.heads, self.groups, self.dk, self.dv, self.tiles = heads, groups, dk, dv, (dv + TILE - 1) // TILE
        self.S = torch.zeros(slots, heads, dk, dv, dtype=torch.float32, device=device)

    def reset(self, slot: int) -> None:
        self.S[slot].zero_()

    def bytes_per_slot(self) -> int:
        return 4 * self.S[0].numel()


def _cpu(x, steps, bias, a, skip, st: SsdState, row_start, slots, out) -> None:
    H, G, dk, dv = st.heads, st.groups, st.dk, st.dv
    C, B = (x[:, i * G * dk: (i + 1) * G * dk].float().view(-1, G, dk).repeat_interleave(H // G, 1) for i in (0, 1))
    v = x[:, 2 * G * dk: 2 * G * dk + H * dv].float().view(-1, H, dv)
    dt = torch.nn.functional.softplus(steps[:, :H].float() + bias, threshold=1e9)
    for s in range(slots.numel()):
        S = st.S[int(slots[s])]
        for t in range(int(row_start[s]), int(row_start[s + 1])):
            S = torch.exp(a * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * v[t][:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, C[t]) + skip[:, None] * v[t]
        st.S[int(slots[s])] = S


def state_space(x: torch.Tensor, steps: torch.Tensor, bias: torch.Tensor, a: torch.Tensor, skip: torch.Tensor, state: SsdState,
                row_start: torch.Tensor, slots: torch.Tensor, out: torch.Tensor, max_rows: int) -> None:
    """Runs the rows ``row_start[s] .. row_start[s + 1]`` of every sequence through its state (updated in place) and writes the heads'
    outputs to the same rows of ``out`` (FP32 [all rows, heads, dv]). ``steps`` (the type of ``x``) [all rows, >= heads]: logits of the
    step sizes; FP32 per head: their ``bias``, ``a`` = -exp(A_log), and ``skip``, the factor of the input in the output."""
    if not x.is_cuda:
        _cpu(x, steps, bias, a, skip, state, row_start, slots, out)
        return
    st, n = state, slots.numel()
    _require(x.dim() == 2 and x.stride(1) == 1 and x.shape[1] >= 2 * st.groups * st.dk + st.heads * st.dv, "state_space: packed rows")
    _require(steps.dtype == x.dtype and steps.stride(1) == 1 and steps.shape[1] >= st.heads, "state_space: step logits")
    _require(all(t.dtype == torch.float32 and t.numel() == st.heads and t.is_contiguous() for t in (bias, a, skip)), "state_space: FP32 vectors")
    _require(row_start.dtype == slots.dtype == torch.int32 and row_start.numel() == n + 1 and out.is_contiguous() and out.dtype == torch.float32,
             "state_space: metadata")
    args = (ptr(x), ptr(steps), ptr(bias), ptr(a), ptr(skip), ptr(st.S), ptr(out), ptr(row_start), ptr(slots), n, x.stride(0), steps.stride(0),
            st.heads, st.groups, st.dk, st.dv)
    if x.dtype == torch.float32 or max_rows < CHUNK_MIN_ROWS or st.dk > CHUNK_MAX_KEY:
        check(kernels().ff_ssd_recurrent(*args, int(x.dtype == torch.float32), stream_ptr()), "ff_ssd_recurrent")
        _count()
        return
    segs, scratch = 1, None
    if n * st.heads * st.tiles < FILL_CTAS and max_rows >= 2 * SEGMENT_ROWS:
        segs = (max_rows + SEGMENT_ROWS - 1) // SEGMENT_ROWS
        scratch = workspace(x.device).ensure("mlstm_segments", n * segs * st.heads * (st.dk * st.dv + st.tiles * (st.dk + 3)))
    check(kernels().ff_ssd_chunked(*args, segs, SEGMENT_ROWS, ptr(scratch), stream_ptr()), "ff_ssd_chunked")
    _count(1 if segs == 1 else 3)


def gated_out(o: torch.Tensor, z: torch.Tensor, w: torch.Tensor, vdim: int, parts: int, eps: float) -> torch.Tensor:
    """``y / rms(y) * w`` with ``y = o silu(z)``, normed in ``parts`` equal pieces of the heads' own elements (``vdim`` of each) ->
    [rows, heads * dv] of the type of ``z``. ``w`` FP32 [heads * dv]."""
    rows, heads, dv = o.shape
    if not o.is_cuda:
        g = z.float()
        y = (o.reshape(rows, heads * dv) * g * torch.sigmoid(g)).view(rows, heads, dv)[..., :vdim].reshape(rows, parts, -1)
        y = (y * torch.rsqrt((y * y).mean(-1, keepdim=True) + eps)).view(rows, heads, vdim)
        out = torch.zeros(rows, heads, dv)
        out[..., :vdim] = y
        return (out.view(rows, heads * dv) * w).to(z.dtype)
    _require(o.dtype == torch.float32 and o.is_contiguous() and z.shape == (rows, heads * dv) and z.stride(1) == 1, "gated_out: operands")
    _require(w.dtype == torch.float32 and w.numel() == heads * dv and w.is_contiguous(), "gated_out: weight")
    y = torch.empty(rows, heads * dv, dtype=z.dtype, device=o.device)
    check(kernels().ff_ssd_out(ptr(o), ptr(z), z.stride(0), ptr(w), ptr(y), rows, heads, vdim, dv, parts, c_float(eps),
                               int(z.dtype == torch.float32), stream_ptr()), "ff_ssd_out")
    _count()
    return y
