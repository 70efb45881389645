"""Multi-head latent attention operators: latent cache write, absorbed attention over the paged
latent cache, per-head batched projections. CUDA: ``csrc/mla.cu`` (+ the grouped tcgen05 GEMM for the
per-head W_UK / W_UV products); CPU: FP32 oracles. :func:`latent_norm_kv` and :func:`latent_attention` are the forms for any
widths, windows and 32-bit, with ``ops.head_linear`` for the per-head products."""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_longlong
from dataclasses import dataclass

import torch

from . import _count, _head_gate_ld, _require, attn_decode, attn_prefill, linear, workspace
from .lib import check, kernels, ptr, status_tensor, stream_ptr

F32 = torch.float32


def cache_write(c: torch.Tensor, k_rope: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor) -> None:
    """cache: [blocks, 1, block_size, kv_lora + rope]; row r goes to ``slots[r]`` (negative skips)."""
    nb, _, bs, d = cache.shape
    if not c.is_cuda:
        ok = slots >= 0
        blk = torch.div(slots[ok], bs, rounding_mode="floor").long()
        off = (slots[ok] % bs).long()
        cache[blk, 0, off, :] = torch.cat([c, k_rope], dim=1)[ok].to(cache.dtype)
        return
    _require(c.shape[1] == 512 and k_rope.shape[1] == 64 and bs == 64 and d == 576, "MLA kernel: kv_lora 512 + rope 64")
    _require(c.stride(1) == 1 and k_rope.stride(1) == 1 and cache.is_contiguous(), "mla cache_write: layout")
    check(kernels().ff_mla_cache_write(ptr(c), ptr(k_rope), ptr(slots), ptr(cache), c.shape[0], c.stride(0),
                                       k_rope.stride(0), nb, ptr(status_tensor(c.device)), stream_ptr()), "ff_mla_cache_write")
    _count()


def attention(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, q_start: torch.Tensor,
              q_lens: torch.Tensor, ctx_lens: torch.Tensor, max_q: int, max_ctx: int, scale: float, kv_lora: int,
              window: int = 0, head_gate: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """q: [rows, heads, kv_lora + rope] (absorbed queries). Returns out_lat [rows, heads, kv_lora]. ``window > 0``: a query sees its last
    ``window`` keys; ``head_gate`` ([rows, heads]): a head's result is multiplied by its sigmoid."""
    rows, heads, d = q.shape
    batch = block_table.shape[0]
    if not q.is_cuda:
        _require(window == 0 and head_gate is None and out is None, "MLA oracle: see latent_attention")
        out = torch.zeros(rows, heads, kv_lora, dtype=q.dtype)
        bs = cache.shape[2]
        for b in range(batch):
            ql, ctx, qs = int(q_lens[b]), int(ctx_lens[b]), int(q_start[b])
            if ql == 0:
                continue
            nblk = (ctx + bs - 1) // bs
            kv = cache[block_table[b, :nblk].long(), 0].reshape(nblk * bs, d)[:ctx].to(F32)
            qq = q[qs: qs + ql].to(F32)
            s = torch.einsum("qhd,kd->hqk", qq, kv) * scale
            pos_q = torch.arange(ql)[:, None] + (ctx - ql)
            vis = torch.arange(ctx)[None, :] <= pos_q
            s = s.masked_fill(~vis[None], float("-inf"))
            p = torch.softmax(s, dim=-1)
            out[qs: qs + ql] = torch.einsum("hqk,kd->qhd", p, kv[:, :kv_lora]).to(q.dtype)
        return out
    _require(d <= 576 and kv_lora <= 512 and d % 16 == 0 and kv_lora % 16 == 0 and q.is_contiguous() and cache.shape[2] == 64 and
             cache.shape[3] == d and cache.is_contiguous(), "MLA kernel: contiguous [rows, heads, d], d up to 576 and latents up to 512 wide")
    lib = kernels()
    po, pml = c_longlong(0), c_longlong(0)
    if window:
        max_ctx = min(max_ctx, window + max_q + 63)
    nsplit = lib.ff_mla_plan(batch, heads, max_q, max_ctx, kv_lora, ctypes.byref(po), ctypes.byref(pml))
    ws = workspace(q.device)
    part_o = ws.ensure("attn_o", po.value // 4) if nsplit > 1 else None
    part_ml = ws.ensure("attn_ml", pml.value // 4) if nsplit > 1 else None
    if out is None:
        out = torch.empty(rows, heads, kv_lora, dtype=torch.bfloat16, device=q.device)
    _require(out.numel() == rows * heads * kv_lora and out.is_contiguous() and out.dtype == torch.bfloat16, "MLA kernel: output")
    rc = lib.ff_mla_attn(ptr(q), ptr(cache), ptr(block_table), ptr(q_start), ptr(q_lens), ptr(ctx_lens), ptr(out),
                         ptr(part_o), ptr(part_ml), batch, heads, max_q, block_table.shape[1], cache.shape[0], nsplit,
                         c_float(scale), d, kv_lora, window, ptr(head_gate), _head_gate_ld(head_gate, rows, heads), ptr(status_tensor(q.device)), stream_ptr())
    check(rc, "ff_mla_attn")
    _count(2 if nsplit > 1 else 1)
    return out


def per_head_linear(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``y[r, h] = x[r, h] @ w[h].T`` for x [rows, heads, k], w [heads, n, k] -> [rows, heads, n]."""
    rows, heads, k = x.shape
    n = w.shape[1]
    if not x.is_cuda:
        return torch.einsum("rhk,hnk->rhn", x.to(torch.float64), w.to(torch.float64)).to(x.dtype)
    from . import moe_cuda
    _require(n % 128 == 0 and k % 8 == 0, "per_head_linear: n % 128 == 0")
    pad = (rows + 15) // 16 * 16
    xs = torch.zeros(heads, pad, k, dtype=torch.bfloat16, device=x.device)
    xs[:, :rows] = x.permute(1, 0, 2)
    seg_off = (torch.arange(heads + 1, dtype=torch.int32, device=x.device) * pad)
    counts = torch.full((heads,), rows, dtype=torch.int32, device=x.device)
    y = moe_cuda.grouped_gemm(xs.view(heads * pad, k), w.contiguous(), seg_off, counts, heads * pad, epi=0)
    return y.view(heads, pad, n)[:, :rows].permute(1, 0, 2).contiguous()


# ------------------------------------------------------------------------------------------
# any widths, windows, BF16 and FP32
# ------------------------------------------------------------------------------------------
def latent_norm_kv(p: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor, q_full: torch.Tensor, q_rot_col: int, latent_col: int, rank: int,
                   rank_pad: int, weight: torch.Tensor, cos_sin: torch.Tensor, eps: float) -> None:
    """Packed rows ``p`` with the rotated query parts ([heads, rot_pad] from ``q_rot_col``) and, from ``latent_col``, the latent
    (``rank`` of ``rank_pad`` columns) and the rotated key part. The latent is normed (``weight`` FP32 [rank_pad]) and goes with the
    turned key to ``slots`` of ``cache`` [blocks, 1, bs, rank_pad + rot_pad]; the turned query parts go to the last columns of
    ``q_full`` [rows, heads, rank_pad + rot_pad]. Neighbours turn (``cos_sin``: :func:`ops.rope_angles`)."""
    rows, heads, width = q_full.shape
    rot = width - rank_pad
    half = cos_sin.shape[1]
    nb, one, bs, cw = cache.shape
    _require(one == 1 and cw == width and cache.is_contiguous() and q_full.is_contiguous() and p.dtype == cache.dtype == q_full.dtype and
             p.shape[0] == rows and p.stride(1) == 1 and 2 * half <= rot, "latent_norm_kv: operands")
    _require(weight.dtype == F32 and weight.numel() == rank_pad and cos_sin.shape == (rows, half, 2) and cos_sin.dtype == F32, "latent_norm_kv: tables")
    if not p.is_cuda:
        c, s = cos_sin[..., 0], cos_sin[..., 1]

        def turn(x, c, s):
            u, v = x[..., 0: 2 * half: 2].clone(), x[..., 1: 2 * half: 2].clone()
            x[..., 0: 2 * half: 2], x[..., 1: 2 * half: 2] = u * c - v * s, v * c + u * s
            return x
        q = p[:, q_rot_col: q_rot_col + heads * rot].to(F32, copy=True).view(rows, heads, rot)
        q_full[..., rank_pad:] = turn(q, c[:, None], s[:, None]).to(p.dtype)
        lat = p[:, latent_col: latent_col + rank_pad].to(F32)
        lat = lat * torch.rsqrt((lat * lat).sum(-1, keepdim=True) / rank + eps) * weight
        k = turn(p[:, latent_col + rank_pad: latent_col + width].to(F32, copy=True), c, s)
        ok = slots >= 0
        at = slots[ok].long()
        cache[at // bs, 0, at % bs] = torch.cat([lat, k], 1)[ok].to(cache.dtype)
        return
    rc = kernels().ff_latent_norm_kv(ptr(p), ptr(slots), ptr(cache), ptr(q_full), rows, heads, rank, rank_pad, rot, q_rot_col, latent_col, bs, nb,
                                     p.stride(0), c_float(eps), ptr(weight), ptr(cos_sin), half, int(p.dtype == F32), ptr(status_tensor(p.device)),
                                     stream_ptr())
    check(rc, "ff_latent_norm_kv")
    _count()


def latent_attention(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, q_start: torch.Tensor, q_lens: torch.Tensor,
                     ctx_lens: torch.Tensor, max_q: int, max_ctx: int, scale: float, rank: int, window: int = 0,
                     head_gate: torch.Tensor | None = None, out: torch.Tensor | None = None, decode: bool = False) -> torch.Tensor:
    """Absorbed attention over the paged rows ``[latent (rank columns) | rotated key]``: q [rows, heads, width] -> [rows, heads * rank].
    All heads read one key row and its first ``rank`` columns as the value, which is multi-query attention: rows of up to 128
    columns take the kernels of ``ops.attn_prefill`` (tcgen05) and ``ops.attn_decode``, wider ones ``csrc/mla.cu``, still wider ones and FP32
    ``csrc/attention_simt.cu``. ``q_start`` / ``q_lens``: the rows of every sequence; with ``decode`` each has ``max_q``."""
    rows, heads, width = q.shape
    flat, vals = q.reshape(rows, heads * width), cache[..., :rank]
    if out is None:
        out = torch.empty(rows, heads * rank, dtype=q.dtype, device=q.device)
    kw = dict(window=window, vdim=rank, head_gate=head_gate, out=out)
    wide = q.is_cuda and q.dtype != F32 and width > 128
    if wide and width <= 576 and rank <= 512:
        attention(q, cache, block_table, q_start, q_lens, ctx_lens, max_q, max_ctx, scale, rank, window, head_gate, out)
        return out
    if decode:
        reach = min(max_ctx, window + cache.shape[2]) if window else max_ctx
        return attn_decode(flat, cache, vals, block_table, ctx_lens, heads, 1, width, scale, nq=max_q, max_ctx=reach, **kw)
    return attn_prefill(flat, cache, vals, block_table, q_start, q_lens, ctx_lens, max_q, heads, 1, width, scale, **kw)


# ------------------------------------------------------------------------------------------
# prompts: keys and values expanded from the latents
# ------------------------------------------------------------------------------------------
EXPAND_MIN_ROWS = 64             # portions of fewer rows stay in the latent space
EXPAND_MAX_KEYS = 1 << 16        # most key rows expanded at a time


def expands(q: torch.Tensor, width: int, dim: int, rot: int, vdim: int, longest: int) -> bool:
    """Whether :func:`expanded_attention` serves a batch whose longest portion has ``longest`` rows: on the tensor cores a head of
    dim + rot elements costs a fraction of one as wide as the latent, which pays for the expansion from a few dozen rows on. Narrow
    latents have the tcgen05 kernel in the latent space."""
    return q.is_cuda and q.dtype == torch.bfloat16 and width > 128 and dim <= 128 and rot <= 64 and vdim <= 128 and longest >= EXPAND_MIN_ROWS


@dataclass
class KeyPages:
    """Cache pages a batch of portions can see, one sequence after the other."""
    count: int
    offsets: torch.Tensor            # int32 [sequences]: page t of a sequence is expanded page offsets + t
    blocks: torch.Tensor             # int32 [count]: the pages' blocks

    @classmethod
    def of(cls, q_lens: list[int], ctx_lens: list[int], block_table, window: int, page: int, device) -> "KeyPages | None":
        """``block_table``: rows of block ids on the host. None when the pages hold more than ``EXPAND_MAX_KEYS`` keys."""
        offsets, blocks = [], []
        for row, n, ctx in zip(block_table, q_lens, ctx_lens):
            first = max(ctx - n - window + 1, 0) // page if window else 0
            offsets.append(len(blocks) - first)
            blocks += row[first: (ctx + page - 1) // page].tolist()
        if len(blocks) * page > EXPAND_MAX_KEYS:
            return None
        both = torch.tensor(offsets + blocks, dtype=torch.int32, device=device)
        return cls(len(blocks), both[: len(offsets)], both[len(offsets):])


def expanded_attention(q: torch.Tensor, q_full: torch.Tensor, cache: torch.Tensor, w_kv: torch.Tensor, pages: KeyPages, block_table: torch.Tensor,
                       q_start: torch.Tensor, q_lens: torch.Tensor, ctx_lens: torch.Tensor, max_q: int, dim: int, vdim: int, rank: int, scale: float,
                       window: int, head_gate: torch.Tensor | None, out: torch.Tensor) -> torch.Tensor:
    """Prefill attention with every visible latent expanded once: ``w_kv`` ([heads * (dim + vdim), rank], all key matrices, then all value
    matrices) makes keys and values of the pages, then the tcgen05 prefill kernel reads them beside the cache's rotated key parts.
    q: rows with the heads' unrotated parts (``dim`` each); ``q_full`` [rows, heads, rank + rot] holds the rotated ones behind
    ``rank`` columns. out: [rows, heads * vdim]."""
    rows, heads, width = q_full.shape
    nb, one, bs, cw = cache.shape
    _require(one == 1 and bs == 64 and cw == width and cache.is_contiguous() and q_full.is_contiguous() and q.stride(1) == 1 and out.is_contiguous(),
             "expanded_attention: layout")
    latents = torch.empty(pages.count * bs, rank, dtype=q.dtype, device=q.device)
    check(kernels().ff_mla_gather(ptr(cache), ptr(pages.blocks), ptr(latents), pages.count, rank, cw, nb, ptr(status_tensor(q.device)), stream_ptr()),
          "ff_mla_gather")
    both = linear(latents, w_kv)
    rc = kernels().ff_attn_prefill_latent(ptr(q), ptr(q_full), ptr(both), ptr(cache), ptr(block_table), ptr(q_start), ptr(q_lens), ptr(ctx_lens),
                                          ptr(pages.offsets), ptr(out), block_table.shape[0], rows, max_q, heads, dim, width - rank, vdim, q.stride(0),
                                          width, rank, both.stride(0), both.shape[0], cw, rank, out.stride(0), block_table.shape[1], nb, c_float(scale),
                                          window, ptr(head_gate), _head_gate_ld(head_gate, rows, heads), ptr(status_tensor(q.device)), stream_ptr())
    check(rc, "ff_attn_prefill_latent")
    _count(2)
    return out
