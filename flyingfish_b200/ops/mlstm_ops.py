"""Matrix memory with exponential gates (the mLSTM of xLSTM) over packed rows of several sequences, its state addressed by slot.
CUDA: ``csrc/mlstm.cu`` (token by token for decoding and 32-bit prompts, 64 tokens at a time for BF16 prompts); CPU: the
recurrence in FP32.

Packed rows hold ``[q heads | k heads | v heads | gate heads]``, heads ``dk`` / ``dv`` wide (multiples of 16, zeros behind a head's
own elements)."""
from __future__ import annotations

from ctypes import c_float

import torch

from . import _count, _require, workspace
from .lib import check, kernels, ptr, stream_ptr

TILE = 64                    # value columns one CTA owns
CHUNK = 64                   # tokens of a chunk
CHUNK_MIN_ROWS = 12          # shortest longest portion of a launch for which the chunked form is used
CHUNK_MAX_KEY = 256
SEGMENT_ROWS = 512           # rows of a segment where a prompt is cut into segments that run side by side
FILL_CTAS = 256              # launches with fewer CTAs than this cut long prompts into segments


class MemoryState:
    """State of one layer run for ``slots`` sequences: S [slots, heads, dk, dv], n and the running maximum m (a copy per tile of
    64 value columns), all FP32 and zero at the start of a sequence."""

    def __init__(self, slots: int, heads: int, dk: int, dv: int, device):
        self.heads, self.dk, self.dv, self.tiles = heads, dk, dv, (dv + TILE - 1) // TILE
        z = lambda *s: torch.zeros(*s, dtype=torch.float32, device=device)
        self.S, self.n, self.m = z(slots, heads, dk, dv), z(slots, heads, self.tiles, dk), z(slots, heads, self.tiles)

    def reset(self, slot: int) -> None:
        for t in (self.S, self.n, self.m):
            t[slot].zero_()

    def bytes_per_slot(self) -> int:
        return sum(t[0].numel() * 4 for t in (self.S, self.n, self.m))


def _cpu(x, gates, bias, cap, st: MemoryState, row_start, slots, qscale, out) -> None:
    H, dk, dv = st.heads, st.dk, st.dv
    z = cap * torch.tanh((gates[:, : 2 * H].float() + bias) / cap)
    li, lf = z[:, :H], torch.nn.functional.logsigmoid(z[:, H:])
    q = x[:, : H * dk].float().view(-1, H, dk) * qscale
    k = x[:, H * dk: 2 * H * dk].float().view(-1, H, dk)
    v = x[:, 2 * H * dk: 2 * H * dk + H * dv].float().view(-1, H, dv)
    for s in range(slots.numel()):
        sl = int(slots[s])
        S, n, m = st.S[sl], st.n[sl, :, 0], st.m[sl, :, 0]
        for t in range(int(row_start[s]), int(row_start[s + 1])):
            new = torch.maximum(lf[t] + m, li[t])
            keep, add = torch.exp(lf[t] + m - new), torch.exp(li[t] - new)
            S = keep[:, None, None] * S + (add[:, None] * k[t])[:, :, None] * v[t][:, None, :]
            n = keep[:, None] * n + add[:, None] * k[t]
            m = new
            den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            out[t] = torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None]
        st.S[sl] = S
        st.n[sl] = n[:, None]
        st.m[sl] = m[:, None]


def memory(x: torch.Tensor, gates: torch.Tensor, gate_bias: torch.Tensor, cap: float, state: MemoryState, row_start: torch.Tensor,
           slots: torch.Tensor, qscale: float, out: torch.Tensor, max_rows: int) -> None:
    """Runs the rows ``row_start[s] .. row_start[s + 1]`` of every sequence through its state (updated in place) and writes the
    heads' outputs to the same rows of ``out`` (FP32 [all rows, heads, dv]). ``gates`` FP32 [all rows, >= 2 heads]: logits of the
    input gates, then of the forget gates; ``max_rows``: the longest sequence's rows."""
    if not x.is_cuda:
        _cpu(x, gates, gate_bias, cap, state, row_start, slots, qscale, out)
        return
    st, n = state, slots.numel()
    _require(x.dim() == 2 and x.stride(1) == 1 and x.shape[1] >= 2 * st.heads * (st.dk) + st.heads * st.dv, "memory: packed rows")
    _require(gates.dtype == gate_bias.dtype == out.dtype == torch.float32 and gates.stride(1) == 1 and gate_bias.numel() == 2 * st.heads, "memory: FP32 gates")
    _require(row_start.dtype == slots.dtype == torch.int32 and row_start.numel() == n + 1 and out.is_contiguous(), "memory: metadata")
    args = (ptr(x), ptr(gates), ptr(gate_bias), ptr(st.S), ptr(st.n), ptr(st.m), ptr(out), ptr(row_start), ptr(slots), n, x.stride(0),
            gates.stride(0), st.heads, st.dk, st.dv, st.tiles, c_float(qscale), c_float(cap))
    if x.dtype == torch.float32 or max_rows < CHUNK_MIN_ROWS or st.dk > CHUNK_MAX_KEY:
        check(kernels().ff_mlstm_recurrent(*args, int(x.dtype == torch.float32), stream_ptr()), "ff_mlstm_recurrent")
        _count()
        return
    segs, scratch = 1, None
    if n * st.heads * st.tiles < FILL_CTAS and max_rows >= 2 * SEGMENT_ROWS:
        segs = (max_rows + SEGMENT_ROWS - 1) // SEGMENT_ROWS
        scratch = workspace(x.device).ensure("mlstm_segments", n * segs * st.heads * (st.dk * st.dv + st.tiles * (st.dk + 3)))
    check(kernels().ff_mlstm_chunked(*args, segs, SEGMENT_ROWS, ptr(scratch), stream_ptr()), "ff_mlstm_chunked")
    _count(1 if segs == 1 else 3)


def head_out(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, vdim: int, eps: float) -> torch.Tensor:
    """``o / rms(o) * w * sigmoid(gate)`` per head (``vdim`` elements count) -> [rows, heads * dv] of the gate's type. ``w`` FP32."""
    rows, heads, dv = o.shape
    if not o.is_cuda:
        y = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / vdim + eps)
        return (y.reshape(rows, heads * dv) * w * torch.sigmoid(gate.float())).to(gate.dtype)
    _require(o.dtype == torch.float32 and o.is_contiguous() and gate.shape == (rows, heads * dv) and gate.stride(1) == 1, "head_out: operands")
    _require(w.dtype == torch.float32 and w.numel() == heads * dv and w.is_contiguous(), "head_out: weight")
    y = torch.empty(rows, heads * dv, dtype=gate.dtype, device=o.device)
    check(kernels().ff_mlstm_out(ptr(o), ptr(gate), gate.stride(0), ptr(w), ptr(y), rows, heads, vdim, dv, c_float(eps),
                                 int(gate.dtype == torch.float32), stream_ptr()), "ff_mlstm_out")
    _count()
    return y
