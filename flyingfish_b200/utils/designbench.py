"""A design's throughput and kernels beside the closest other model at equal size (``bench.py --design duponex``).

The closest model of a Duponex shape is the Gemma layout (QK-norm, local attention in every layer, extra norms per
sub-layer, operator-by-operator decode step): same width, heads and layers, a sliding window as long as the block, and a
gated feed-forward of the width that makes the layers' weights equal. Prompts end inside a block, so both attentions see
the same keys. Weights are random. Every kernel of the design is timed beside its like kernel on the same rows; a
fraction of the roofline is algorithmic bytes (or FLOPs) over time over the measured peak, and ``distance`` is the ratio
of the two fractions (above 1: the design's kernel is further from its roofline).
"""
from __future__ import annotations

import dataclasses

import torch

from .. import ops
from ..config import ModelSpec, Settings, named_shape
from ..ops import stream_ops
from .kbench import Flusher, peaks, time_op

SIZES = ("duponex-2b-shape", "duponex-8b-shape")


def closest_spec(spec: ModelSpec) -> ModelSpec:
    """Gemma-layout shape with the layer weights of a Duponex shape of equal layers."""
    l = spec.layer_specs[0]
    f = (l.heads * l.vdim + 2 * l.ffn) // 3 // 128 * 128
    return ModelSpec(name=spec.name.replace("duponex", "gemma-layout"), arch="gemma", layers=spec.layers, hidden=spec.hidden,
                     heads=l.heads, kv_heads=l.kv_heads, head_dim=l.dim, ffn=f, vocab=spec.vocab, qk_norm=True, swiglu_mode=2,
                     rms_eps=spec.rms_eps, extra={"gemma": {"window": l.chunk, "global_every": spec.layers + 1}})


def _device_ms(fn, n: int) -> float:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


def model_throughput(spec: ModelSpec, prompt: int, batches, steps: int, warmup: int, device) -> dict:
    """Prefill tokens/s (8 prompts together, and one of 8192 tokens) and decode tokens/s per batch size."""
    from ..api import Model
    long = 8192
    m = Model.load(spec, Settings(capacity=long + 64, max_batch=max(max(batches), 8), kv_tokens=max(batches) * (prompt + 128) + 2 * long),
                   device=device)
    eng = m.engine
    g = torch.Generator().manual_seed(1)
    prompts = lambda n, k: [torch.randint(0, spec.vocab, (k,), generator=g).tolist() for _ in range(n)]

    def prefill(n, k):
        seqs = [eng.add_sequence(p) for p in prompts(n, k)]
        ms = _device_ms(lambda: eng.prefill(seqs), 1)
        return seqs, n * k / ms * 1e3

    def drop(seqs):
        for s in seqs:
            eng.free_sequence(s.seq_id)
    out: dict = {"prefill_tokens_per_s": {}, "decode_tokens_per_s": {}, "decode_ms": {}, "decode_e2e_ms": {}}
    for n, k in ((8, prompt), (1, long)):
        rates = []
        for _ in range(4):
            seqs, r = prefill(n, k)
            drop(seqs)
            rates.append(r)
        out["prefill_tokens_per_s"][f"{n}x{k}"] = max(rates[1:])
    for b in batches:
        seqs, _ = prefill(b, prompt)
        for _ in range(warmup):
            eng.decode(seqs)
        out["decode_e2e_ms"][str(b)] = _device_ms(lambda: eng.decode(seqs), steps)
        # device-timed: the captured step replayed back to back (the weights read per step exceed the L2)
        graph = eng.capture(b).graph
        out["decode_ms"][str(b)] = _device_ms(graph.replay, steps)
        out["decode_tokens_per_s"][str(b)] = b / out["decode_ms"][str(b)] * 1e3
        drop(seqs)
    ops.check_status()
    out["layer_weights"] = spec.dense_param_count() - 2 * spec.vocab * spec.hidden if spec.layer_specs is not None else \
        spec.layers * (spec.hidden * spec.qkv_dim + spec.q_dim * spec.hidden + 3 * spec.hidden * spec.ffn)
    del m, eng
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------
# kernel by kernel
# ------------------------------------------------------------------------------------------
class _Paged:
    """Random caches of ``batch`` sequences of ``ctx`` tokens for both attentions."""

    def __init__(self, batch: int, ctx: int, hkv: int, d: int, dev):
        per = (ctx + 63) // 64
        self.k, self.v = (torch.randn(batch * per, hkv, 64, d, device=dev).to(torch.bfloat16) for _ in range(2))
        self.table = torch.randperm(batch * per, device=dev).to(torch.int32).view(batch, per)
        self.ctx = torch.full((batch,), ctx, dtype=torch.int32, device=dev)


def kernel_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    """One line per pair: the design's kernel and its like on ``rows`` rows (``rows`` <= 128: a decode step of that batch at
    context ``ctx``; more: prefill of rows / ctx prompts)."""
    l, other = spec.layer_specs[0], closest_spec(spec)
    dev, bf = torch.device(device), torch.bfloat16
    W, S, H, G, d, f = spec.hidden, int(spec.extra["duponex"]["streams"]), l.heads, l.kv_heads, l.dim, l.ffn
    rn = lambda *s: torch.randn(*s, device=dev).to(bf)
    pk, flush = peaks(), Flusher(dev)
    decode = rows <= 128
    res: list[dict] = []

    def bound(byts, flops):
        return max(byts / (pk["hbm_gbs"] * 1e9), flops / (pk["bf16_tflops"] * 1e12)) * 1e6

    def pair(name, mine, mine_cost, like_name, like, like_cost):
        a, b = (time_op(fn, iters, 3, flush, graph=True)["us_median"] for fn in (mine, like))
        fa, fb = bound(*mine_cost) / a, bound(*like_cost) / b
        res.append({"kernel": name, "us": round(a, 2), "frac": round(fa, 3), "like": like_name, "like_us": round(b, 2),
                    "like_frac": round(fb, 3), "distance": round(fb / fa, 2)})

    def gemm_cost(n, k, out_cols=None):
        return (2 * (rows * k + n * k + rows * (out_cols or n)), 2 * rows * n * k)
    x, n1, a1 = rn(rows, W), rn(W), rn(rows, H * d)
    # projections
    nq, no = H * d + 2 * G * d + H * d, H * d + 2 * G * d
    wq, bq, wqo = rn(nq, W), rn(nq), rn(no, W)
    pair("qkv+gate projection, bias", lambda: ops.linear(x, wq, bias=bq), gemm_cost(nq, W), "qkv projection",
         lambda: ops.linear(x, wqo), gemm_cost(no, W))
    wo, bo = rn(W, H * d), rn(W)
    pair("output projection, bias", lambda: ops.linear(a1, wo, bias=bo), gemm_cost(W, H * d), "output projection",
         lambda: ops.linear(a1, wo), gemm_cost(W, H * d))
    wu, wgu, h1, h2 = rn(f, W), rn(2 * other.ffn, W), rn(rows, f), rn(rows, other.ffn)
    pair("up projection, squared ReLU", lambda: ops.linear(x, wu, act="relu2"), gemm_cost(f, W), "gate/up projection, tanh-GELU",
         lambda: ops.linear_swiglu(x, wgu, mode=2), gemm_cost(2 * other.ffn, W, other.ffn))
    wd, wdo = rn(W, f), rn(W, other.ffn)
    pair("down projection", lambda: ops.linear(h1, wd), gemm_cost(W, f), "down projection", lambda: ops.linear(h2, wdo), gemm_cost(W, other.ffn))
    del wq, wqo, wo, wu, wgu, wd, wdo, h1, h2
    # streams against add + norm (the residual stays in memory: each launch works on the same buffer)
    xs, coef, scale = torch.randn(rows, S, W, device=dev), torch.randn(S * (S + 2), device=dev) * 0.1, rn(W)
    r16 = rn(rows, W)
    pair("stream step + norm", lambda: stream_ops.step(xs, x, scale, coef, n1, 1e-5, W), (rows * W * (8 * S + 4), 0), "add + norm",
         lambda: ops.add_rmsnorm(x, r16, n1, 1e-5), (rows * W * 8, 0))
    ids, table = torch.randint(0, 1024, (rows,), device=dev).to(torch.int32), rn(1024, W)
    read = torch.randn(S, device=dev)
    pair("stream embed + norm", lambda: stream_ops.embed(ids, table, 2.0, read, n1, 1e-5, W), (rows * W * (4 * S + 4), 0), "embed + norm",
         lambda: ops.embed_rmsnorm(ids, table, n1, 1e-5), (rows * W * 6, 0))
    del xs
    # head norm + cache write against head norm, rotation and cache write
    batch = rows if decode else rows // ctx
    pg = _Paged(batch, ctx, G, d, dev)
    slots = torch.randperm(pg.k.shape[0] * 64, device=dev)[:rows].to(torch.int32)
    pos = torch.arange(rows, device=dev).to(torch.int32) % ctx
    qkvg, first = rn(rows, nq), rn(rows, nq)
    v0 = (H + G) * d
    byts = 2 * rows * d * (2 * H + 2 * G + 2 * G + G)
    qk = rn(rows, no)
    pair("head norm + value mix + cache write", lambda: ops.head_norm_kv(qkvg, slots, pg.k, pg.v, H, G, d, d, 1e-5, first_v=first[:, v0: v0 + G * d], mix=0.3),
         (byts, 0), "rotation + cache write", lambda: ops.rope_kv_paged(qk, pos, slots, pg.k, pg.v, H, G, d, 1e4),
         (2 * rows * d * (2 * H + 2 * G + 2 * G), 0))
    # attention
    gate = qkvg[:, no:]
    out = torch.empty(rows, H * d, dtype=bf, device=dev)
    if decode:
        seen = l.keys_seen(ctx)
        cost = lambda gated: (2 * rows * (2 * seen * G * d + (3 if gated else 2) * H * d), 4 * rows * seen * H * d)
        pair("decode attention, block-local, gated", lambda: ops.attn_decode(qkvg, pg.k, pg.v, pg.table, pg.ctx, H, G, d, l.scale, max_ctx=ctx,
             out=out, chunk=l.chunk, gate=gate), cost(True), "decode attention, window",
             lambda: ops.attn_decode(qk, pg.k, pg.v, pg.table, pg.ctx, H, G, d, l.scale, max_ctx=ctx, window=l.chunk), cost(False))
    else:
        qs, ql = (torch.arange(batch, device=dev) * ctx).to(torch.int32), torch.full((batch,), ctx, dtype=torch.int32, device=dev)
        pairs = batch * l.pairs_seen(ctx)
        wpairs = batch * sum(min(i + 1, l.chunk) for i in range(ctx))
        cost = lambda p: (2 * rows * (2 * H * d + 2 * G * d), 4 * p * H * d)
        pair("prefill attention, block-local, gated", lambda: ops.attn_prefill(qkvg, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, H, G, d, l.scale,
             out=out, chunk=l.chunk, gate=gate), cost(pairs), "prefill attention, window",
             lambda: ops.attn_prefill(qk, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, H, G, d, l.scale, window=l.chunk), cost(wpairs))
    ops.check_status()
    return res


def run(device, steps: int, warmup: int, sizes=SIZES, batches=(1, 8, 64), prompt: int = 1024, layers: int | None = None) -> dict:
    out: dict = {"design": "duponex", "prompt": prompt, "peaks": peaks(), "sizes": {}}
    for name in sizes:
        spec = named_shape(name)
        if layers:
            spec = dataclasses.replace(spec, layers=layers, layer_specs=spec.layer_specs[:layers])
        other = closest_spec(spec)
        out["sizes"][name] = {
            "closest": {"name": other.name, "ffn": other.ffn},
            "duponex": model_throughput(spec, prompt, batches, steps, warmup, device),
            "closest_model": model_throughput(other, prompt, batches, steps, warmup, device),
            "kernels": {"decode rows 64, context 1024": kernel_table(spec, 64, 1024, 30, device),
                        "prefill 8 x 1024": kernel_table(spec, 8192, 1024, 15, device),
                        "prefill 1 x 8192": kernel_table(spec, 8192, 8192, 15, device)}}
    return out
