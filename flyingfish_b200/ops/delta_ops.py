"""Gated delta rule with a decay per key channel, and the short convolution in front of such recurrences, over packed rows of several
sequences, their state addressed by slot. CUDA: ``csrc/short_conv.cu``, ``csrc/delta.cu`` (token by token for decoding and 32-bit
prompts) and ``csrc/delta_chunk.cu`` (BF16 prompts); CPU: the recurrence in FP32.

Convolved rows hold ``[q heads | k heads | v heads]``, heads ``dk`` / ``dv`` wide (multiples of 16, zeros behind a head's own
elements)."""
from __future__ import annotations

from ctypes import c_float
from dataclasses import dataclass

import torch

from . import _count, _require, workspace
from .lib import check, kernels, ptr, stream_ptr

CONV_MAX_TAPS = 8
CHUNK = 64                   # tokens of a chunk
CHUNK_MIN_ROWS = 12          # shortest longest portion of a launch for which the chunked form is used
CHUNK_MAX_KEY = 128
SCRATCH_BYTES = 512 << 20    # the chunked form takes the chunks of a batch in rounds whose scratch stays below this


@dataclass
class ConvWeights:
    """Depthwise causal convolution over ``nh`` heads of ``dn`` channels and ``vh`` heads of ``dv``: FP32 ``w`` [taps, channels], the
    last row weighs the current token, and ``bias`` [channels] or None."""
    w: torch.Tensor
    bias: torch.Tensor | None
    nh: int
    dn: int
    vh: int
    dv: int

    @property
    def taps(self) -> int:
        return self.w.shape[0]

    @property
    def channels(self) -> int:
        return self.nh * self.dn + self.vh * self.dv


class ConvState:
    """The last ``taps - 1`` inputs of ``slots`` sequences, FP32, zero at the start of a sequence."""

    def __init__(self, slots: int, conv: ConvWeights, device):
        self.x = torch.zeros(slots, conv.taps - 1, conv.channels, dtype=torch.float32, device=device)

    def reset(self, slot: int) -> None:
        self.x[slot].zero_()

    def bytes_per_slot(self) -> int:
        return 4 * self.x[0].numel()


def short_conv(x: torch.Tensor, conv: ConvWeights, state: ConvState, row_start: torch.Tensor, slots: torch.Tensor, max_rows: int,
               unit_scale: float | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """SiLU of the convolution of the first ``conv.channels`` columns of ``x`` -> [rows, channels] of its type; the states take the last
    inputs. ``unit_scale``: also FP32 [rows, nh], ``1 / sqrt(sum of squares + 1e-6)`` of the first ``nh`` heads, times ``unit_scale``
    for the first half of them (queries)."""
    rows, ch = x.shape[0], conv.channels
    if not x.is_cuda:
        out = torch.empty(rows, ch, dtype=x.dtype)
        for s in range(slots.numel()):
            r0, r1, sl = int(row_start[s]), int(row_start[s + 1]), int(slots[s])
            full = torch.cat([state.x[sl], x[r0:r1, :ch].float()])
            y = sum(full[j: j + r1 - r0] * conv.w[j] for j in range(conv.taps))
            if conv.bias is not None:
                y = y + conv.bias
            out[r0:r1] = (y * torch.sigmoid(y)).to(x.dtype)
            state.x[sl] = full[full.shape[0] - (conv.taps - 1):]
        if unit_scale is None:
            return out, None
        h = out[:, : conv.nh * conv.dn].float().view(rows, conv.nh, conv.dn)
        unit = torch.rsqrt((h * h).sum(-1) + 1e-6)
        unit[:, : conv.nh // 2] *= unit_scale
        return out, unit
    _require(x.dim() == 2 and x.stride(1) == 1 and x.shape[1] >= ch and state.x.shape[1:] == (conv.taps - 1, ch), "short_conv: rows and state")
    _require(row_start.dtype == slots.dtype == torch.int32 and row_start.numel() == slots.numel() + 1, "short_conv: metadata")
    out = torch.empty(rows, ch, dtype=x.dtype, device=x.device)
    unit = None if unit_scale is None else torch.empty(rows, conv.nh, dtype=torch.float32, device=x.device)
    rc = kernels().ff_short_conv(ptr(x), ptr(out), ptr(conv.w), ptr(conv.bias), ptr(state.x), ptr(unit), ptr(row_start), ptr(slots), slots.numel(),
                                 max_rows, x.stride(0), conv.nh, conv.dn, conv.vh, conv.dv, conv.taps, c_float(unit_scale or 1.0),
                                 int(x.dtype == torch.float32), stream_ptr())
    check(rc, "ff_short_conv")
    _count()
    return out, unit


class DeltaState:
    """S [slots, heads, dk, dv] of one layer, FP32, zero at the start of a sequence."""

    def __init__(self, slots: int, heads: int, kv_heads: int, dk: int, dv: int, device):
        self.heads, self.kv_heads, self.dk, self.dv = heads, kv_heads, dk, dv
        self.S = torch.zeros(slots, heads, dk, dv, dtype=torch.float32, device=device)

    def reset(self, slot: int) -> None:
        self.S[slot].zero_()

    def bytes_per_slot(self) -> int:
        return 4 * self.S[0].numel()


def _cpu(x, unit, decay, beta, rate, dt_bias, st: DeltaState, row_start, slots, out) -> None:
    H, G, dk, dv = st.heads, st.kv_heads, st.dk, st.dv
    head = lambda a, b: x[:, a:b].float().view(-1, G, dk)
    q, k = ((head(i * G * dk, (i + 1) * G * dk) * unit[:, i * G: (i + 1) * G, None]).repeat_interleave(H // G, 1) for i in (0, 1))
    v = x[:, 2 * G * dk: 2 * G * dk + H * dv].float().view(-1, H, dv)
    b = torch.sigmoid(beta[:, :H].float())
    g = torch.exp(rate[:, None] * torch.nn.functional.softplus(decay[:, : H * dk] + dt_bias, threshold=1e9).view(-1, H, dk))
    for s in range(slots.numel()):
        S = st.S[int(slots[s])]
        for t in range(int(row_start[s]), int(row_start[s + 1])):
            S = g[t][:, :, None] * S
            u = b[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, q[t])
        st.S[int(slots[s])] = S


def delta_rule(x: torch.Tensor, unit: torch.Tensor, decay: torch.Tensor, beta: torch.Tensor, rate: torch.Tensor, dt_bias: torch.Tensor,
               state: DeltaState, row_start: torch.Tensor, slots: torch.Tensor, out: torch.Tensor, max_rows: int) -> None:
    """Runs the rows ``row_start[s] .. row_start[s + 1]`` of every sequence through its state (updated in place) and writes the heads'
    outputs to the same rows of ``out`` (FP32 [all rows, heads, dv]). ``x``, ``unit``: what :func:`short_conv` gives; ``decay`` FP32
    [all rows, heads * dk] and ``beta`` (the type of ``x``) [all rows, >= heads]: logits; ``rate`` [heads] = -exp(A_log) and ``dt_bias``
    [heads * dk] FP32."""
    if not x.is_cuda:
        _cpu(x, unit, decay, beta, rate, dt_bias, state, row_start, slots, out)
        return
    st, n = state, slots.numel()
    _require(x.dim() == 2 and x.stride(1) == 1 and x.shape[1] >= 2 * st.kv_heads * st.dk + st.heads * st.dv, "delta_rule: packed rows")
    _require(unit.dtype == decay.dtype == rate.dtype == dt_bias.dtype == out.dtype == torch.float32 and unit.is_contiguous() and
             decay.stride(1) == 1 and beta.stride(1) == 1 and beta.dtype == x.dtype, "delta_rule: operand types")
    _require(unit.shape[1] == 2 * st.kv_heads and decay.shape[1] >= st.heads * st.dk and beta.shape[1] >= st.heads and rate.numel() == st.heads and
             dt_bias.numel() == st.heads * st.dk, "delta_rule: operand shapes")
    _require(row_start.dtype == slots.dtype == torch.int32 and row_start.numel() == n + 1 and out.is_contiguous(), "delta_rule: metadata")
    args = (ptr(x), ptr(unit), ptr(decay), ptr(beta), ptr(rate), ptr(dt_bias), ptr(st.S), ptr(out), ptr(row_start), ptr(slots), n, x.stride(0),
            decay.stride(0), beta.stride(0), st.heads, st.kv_heads, st.dk, st.dv)
    if x.dtype == torch.float32 or max_rows < CHUNK_MIN_ROWS or st.dk > CHUNK_MAX_KEY:
        check(kernels().ff_delta_recurrent(*args, int(x.dtype == torch.float32), stream_ptr()), "ff_delta_recurrent")
        _count()
        return
    chunks = (max_rows + CHUNK - 1) // CHUNK
    record = kernels().ff_delta_chunk_record(st.dk, st.dv) * n * st.heads
    rounds = -(-chunks // max(1, SCRATCH_BYTES // record))
    per_round = -(-chunks // rounds)
    scratch = workspace(x.device).ensure("delta_chunks", record * per_round // 4)
    check(kernels().ff_delta_chunked(*args, chunks, per_round, ptr(scratch), stream_ptr()), "ff_delta_chunked")
    _count(2 * -(-chunks // per_round))


def head_out(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, vdim: int, eps: float) -> torch.Tensor:
    """``o / rms(o) * w * sigmoid(gate)`` per head (``vdim`` elements count) -> [rows, heads * dv] of the gate's type. ``w`` FP32 [dv],
    shared by the heads."""
    rows, heads, dv = o.shape
    if not o.is_cuda:
        y = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / vdim + eps) * w
        return (y.reshape(rows, heads * dv) * torch.sigmoid(gate.float())).to(gate.dtype)
    _require(o.dtype == torch.float32 and o.is_contiguous() and gate.shape == (rows, heads * dv) and gate.stride(1) == 1, "head_out: operands")
    _require(w.dtype == torch.float32 and w.numel() == dv and w.is_contiguous(), "head_out: weight")
    y = torch.empty(rows, heads * dv, dtype=gate.dtype, device=o.device)
    check(kernels().ff_delta_out(ptr(o), ptr(gate), gate.stride(0), ptr(w), ptr(y), rows, heads, vdim, dv, c_float(eps),
                                 int(gate.dtype == torch.float32), stream_ptr()), "ff_delta_out")
    _count()
    return y
