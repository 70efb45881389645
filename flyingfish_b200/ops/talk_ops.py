"""Windowed attention whose heads' weights are mixed by a matrix before they meet the values (talking heads behind the soft-max). CUDA:
``csrc/talk_tc.cu`` (tensor cores: BF16, heads of up to 128 elements) and ``csrc/talk_simt.cu`` (any head width, BF16 or FP32); CPU: FP32
arithmetic.

The heads do not separate: a row's weights of every head, normalised, go into every head's sum. ``one`` adds a fixed 1 to the soft-max's
denominator."""
from __future__ import annotations

from ctypes import c_float

import torch

from . import BF16, _count, _require, SideLane, _rows2d, workspace
from .lib import check, kernels, ptr, status_tensor, stream_ptr

PAGE = 64
ROWS = 128                    # query rows of a tile of the prompt kernels
ROUND_BYTES = 160 << 20       # prompts: scratch of a round
DECODE_CTAS = 592             # decode: CTAs a launch should have
DECODE_SPLITS = 32
_lanes: dict[int, SideLane] = {}


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
        m = s.amax(-1, keepdim=True)
        m = m.clamp(min=0.0) if one else m
        e = torch.exp(s - m)
        w = e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if one else 0.0))
        w = torch.einsum("hg,gnk->hnk", talk, w)
        out[r0: r0 + n] = torch.einsum("hnk,hkd->nhd", w, rows(vcache, vdim)).reshape(n, hq * vdim)
    return out.to(q.dtype)


def _simt(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, hq: int, hkv: int, scale: float, window: int, talk, one: bool, out) -> None:
    rows, ldq = _rows2d(q)
    rc = kernels().ff_talk_simt(ptr(q), ptr(kcache), ptr(vcache), ptr(block_table), ptr(q_start), ptr(q_lens), ptr(ctx_lens), ptr(talk), ptr(out),
                                block_table.shape[0], rows, 1, hq, hkv, kcache.shape[3], vcache.shape[3], ldq, out.stride(0), kcache.shape[2],
                                block_table.stride(0), kcache.shape[0], window, c_float(scale), c_float(float(one)), int(q.dtype == torch.float32),
                                ptr(status_tensor(q.device)), stream_ptr())
    check(rc, "ff_talk_simt")
    _count()


def _check(q, kcache, vcache, hq: int, talk, out, *metadata) -> bool:
    """Whether the tensor-core kernels take these operands."""
    rows, ldq = _rows2d(q)
    dim, vdim = kcache.shape[3], vcache.shape[3]
    _require(q.dtype == kcache.dtype == vcache.dtype == out.dtype and kcache.is_contiguous() and vcache.is_contiguous(), "talk attention: one type throughout")
    _require(talk.dtype == torch.float32 and talk.shape == (hq, hq) and talk.is_contiguous() and out.stride(1) == 1 and out.shape == (rows, hq * vdim),
             "talk attention: mixing matrix, output")
    _require(all(t.dtype == torch.int32 for t in metadata), "talk attention: int32 metadata")
    return q.dtype == BF16 and max(dim, vdim) <= 128 and dim % 16 == vdim % 16 == 0 and kcache.shape[2] == PAGE and ldq % 8 == out.stride(0) % 8 == 0


def _band(max_ctx: int, window: int, rows: int) -> int:
    """Pages that ``rows`` consecutive positions see at most."""
    return min(-(-max_ctx // PAGE), (window + rows + 61) // PAGE + 1)


def talk_prefill(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor, q_start: torch.Tensor,
                 q_lens: torch.Tensor, ctx_lens: torch.Tensor, max_q_len: int, max_ctx: int, hq: int, hkv: int, scale: float, window: int,
                 talk: torch.Tensor, one: bool, out: torch.Tensor) -> torch.Tensor:
    """Portions of prompts. ``q`` [rows, >= hq * dim]: rows ``q_start[s] .. + q_lens[s]`` of sequence s, the last of them seeing
    ``ctx_lens[s]`` (at most ``max_ctx``) keys through ``window``. ``talk`` FP32 [hq, hq]. Writes ``out`` [rows, hq * vdim]."""
    dim, vdim = kcache.shape[3], vcache.shape[3]
    if not q.is_cuda:
        out.copy_(_cpu(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, hq, hkv, dim, vdim, scale, window, talk, one))
        return out
    tensor = _check(q, kcache, vcache, hq, talk, out, block_table, q_start, q_lens, ctx_lens)
    if not tensor or hq > 32:
        _simt(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, hq, hkv, scale, window, talk, one, out)
        return out
    rows, batch = q.shape[0], block_table.shape[0]
    band, tiles = _band(max_ctx, window, ROWS), -(-max_q_len // ROWS)
    rounds = -(-tiles // max(1, ROUND_BYTES // (batch * hq * ROWS * band * PAGE * 2)))
    rounds += rounds > 1 and rounds % 2    # two streams share them
    per_round = -(-tiles // rounds)
    floats = batch * per_round * hq * ROWS * (band * (PAGE // 2 + 2) + 1)

    def run(first: int, step: int) -> None:
        scratch = workspace(q.device).ensure("talk_weights", floats)
        rc = kernels().ff_talk_prefill(ptr(q), ptr(kcache), ptr(vcache), ptr(block_table), ptr(q_start), ptr(q_lens), ptr(ctx_lens), ptr(talk), ptr(out),
                                       ptr(scratch), batch, rows, max_q_len, hq, hkv, dim, vdim, q.stride(0), out.stride(0), block_table.stride(0),
                                       kcache.shape[0], window, band, per_round, first, step, c_float(scale), c_float(float(one)),
                                       ptr(status_tensor(q.device)), stream_ptr())
        check(rc, "ff_talk_prefill")
    if rounds == 1:
        run(0, 1)
    else:                              # every other round on a second stream: a round's tail runs under the next one
        lane = _lanes.get(q.device.index)
        if lane is None:
            lane = _lanes[q.device.index] = SideLane(q.device)
        lane.fork()
        with lane:
            run(1, 2)
        run(0, 2)
        lane.join()
    _count(3 * -(-tiles // per_round))
    return out


def talk_decode(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_table: torch.Tensor, ctx_lens: torch.Tensor, max_ctx: int, hq: int,
                hkv: int, scale: float, window: int, talk: torch.Tensor, one: bool, out: torch.Tensor) -> torch.Tensor:
    """One row per sequence: as :func:`talk_prefill`."""
    dim, vdim, batch = kcache.shape[3], vcache.shape[3], block_table.shape[0]
    if not q.is_cuda or not _check(q, kcache, vcache, hq, talk, out, block_table, ctx_lens) or hq > 64 or hq // hkv > 16:
        start = torch.arange(batch, dtype=torch.int32, device=q.device)
        args = (q, kcache, vcache, block_table, start, torch.ones_like(start), ctx_lens, hq, hkv)
        if q.is_cuda:
            _simt(*args, scale, window, talk, one, out)
        else:
            out.copy_(_cpu(*args, dim, vdim, scale, window, talk, one))
        return out
    band = _band(max_ctx, window, 1)
    splits = max(1, min(-(-DECODE_CTAS // (hkv * batch)), band, DECODE_SPLITS))
    ws = workspace(q.device)
    scores, ml = ws.ensure("talk_scores", batch * hq * band * PAGE), ws.ensure("talk_ml", batch * splits * hq * 2)
    part = ws.ensure("attn_o", batch * splits * hq * vdim) if splits > 1 else None
    rc = kernels().ff_talk_decode(ptr(q), ptr(kcache), ptr(vcache), ptr(block_table), ptr(ctx_lens), ptr(talk), ptr(out), ptr(scores), ptr(ml), ptr(part),
                                  batch, hq, hkv, dim, vdim, q.stride(0), out.stride(0), block_table.stride(0), kcache.shape[0], window, band, splits,
                                  c_float(scale), c_float(float(one)), ptr(status_tensor(q.device)), stream_ptr())
    check(rc, "ff_talk_decode")
    _count(2 if splits == 1 else 3)
    return out
