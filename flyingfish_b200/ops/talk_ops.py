"""Windowed attention whose heads' weights are mixed by a matrix before they meet the values (talking heads behind the soft-max). CUDA:
``csrc/talk_simt.cu`` (any head width, BF16 or FP32); CPU: FP32 arithmetic.

The heads do not separate: a row's weights of every head, normalised, go into every head's sum. ``one`` adds a fixed 1 to the soft-max's
denominator."""
from __future__ import annotations

from ctypes import c_float

import torch

from . import _count, _require, _rows2d
from .lib import check, kernels, ptr, status_tensor, stream_ptr


def _cpu(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, hq, hkv, dim, vdim, scale, window, talk, one) -> torch.Tensor:
    out = torch.zeros(q.shape[0], hq * vdim)
    page, per = kcache.shape[2], hq // hkv
    for b in range(block_table.shape[0]):
        n, ctx, r0 = int(q_lens[b]), int(ctx_lens[b]), int(q_start[b])
        if n == 0 or ctx == 0:
            continue
        blocks = block_table[b, : (ctx + page - 1) // page].long()
        rows = lambda c, w: c[blocks].permute(1, 0, 2, 3).reshape(hkv, -1, w)[:, :ctx].float().repeat_interleave(per, 0)
        pos, key = torch.arange(ctx - n, ctx)[:, None], torch.arange(ctx)[None, :]
        see = (key <= pos) & (pos - key < window)
        s = torch.einsum("nhd,hkd->hnk", q[r0: r0 + n, : hq * dim].float().view(n, hq, dim), rows(kcache, dim)) * scale
        s = s.masked_fill(~see, float("-inf"))
        m = s.amax(-1, keepdim=True).clamp(min=0.0 if one else None)
        e = torch.exp(s - m)
        w = e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if one else 0.0))
        w = torch.einsum("hg,gnk->hnk", talk, w)
        out[r0: r0 + n] = torch.einsum("hnk,hkd->nhd", w, rows(vcache, vdim)).reshape(n, hq * vdim)
    return out.to(q.dtype)


def talk_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor, q_start: torch.Tensor,
                   q_lens: torch.Tensor, ctx_lens: torch.Tensor, max_q_len: int, hq: int, hkv: int, scale: float, window: int,
                   talk: torch.Tensor, one: bool, out: torch.Tensor) -> torch.Tensor:
    """``q`` [rows, >= hq * dim]: rows ``q_start[s] .. + q_lens[s]`` of sequence s, the last of them seeing ``ctx_lens[s]`` keys. ``talk``
    FP32 [hq, hq]. Writes ``out`` [rows, hq * vdim]."""
    dim, vdim = kcache.shape[3], vcache.shape[3]
    if not q.is_cuda:
        out.copy_(_cpu(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, hq, hkv, dim, vdim, scale, window, talk, one))
        return out
    rows, ldq = _rows2d(q)
    _require(q.dtype == kcache.dtype == vcache.dtype == out.dtype and kcache.is_contiguous() and vcache.is_contiguous(), "talk_attention: one type throughout")
    _require(talk.dtype == torch.float32 and talk.shape == (hq, hq) and talk.is_contiguous() and out.stride(1) == 1 and out.shape == (rows, hq * vdim),
             "talk_attention: mixing matrix, output")
    _require(block_table.dtype == q_start.dtype == q_lens.dtype == ctx_lens.dtype == torch.int32, "talk_attention: int32 metadata")
    rc = kernels().ff_talk_simt(ptr(q), ptr(kcache), ptr(vcache), ptr(block_table), ptr(q_start), ptr(q_lens), ptr(ctx_lens), ptr(talk), ptr(out),
                                block_table.shape[0], rows, 1, hq, hkv, dim, vdim, ldq, out.stride(0), kcache.shape[2], block_table.stride(0),
                                kcache.shape[0], window, c_float(scale), c_float(float(one)), int(q.dtype == torch.float32),
                                ptr(status_tensor(q.device)), stream_ptr())
    check(rc, "ff_talk_simt")
    _count()
    return out


def talk_prefill(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, max_q_len: int, hq: int, hkv: int, scale: float, window: int, talk,
                 one: bool, out: torch.Tensor) -> torch.Tensor:
    """Portions of prompts: see :func:`talk_attention`."""
    return talk_attention(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, max_q_len, hq, hkv, scale, window, talk, one, out)


def talk_decode(q, kcache, vcache, block_table, ctx_lens, max_ctx: int, hq: int, hkv: int, scale: float, window: int, talk, one: bool,
                out: torch.Tensor) -> torch.Tensor:
    """One row per sequence: see :func:`talk_attention`."""
    n = block_table.shape[0]
    start = torch.arange(n, dtype=torch.int32, device=q.device)
    return talk_attention(q, kcache, vcache, block_table, start, torch.ones_like(start), ctx_lens, 1, hq, hkv, scale, window, talk, one, out)
