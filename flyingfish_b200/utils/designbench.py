"""A design's throughput and kernels beside the closest other model at equal size (``bench.py --design duponex|rudorax|kabavik|bazulorn``).

The closest model of a Rudorax shape is the Flint layout (QK-norm, windowed attention with sinks, routed and shared experts): same
width, heads, window, experts and number of layers (Rudorax: layer runs); a memory layer's kernels are timed beside those of the
gated delta net. The closest model of a Duponex shape is the Gemma layout (QK-norm, local attention in every layer, extra norms per
sub-layer, operator-by-operator decode step): same width, heads and layers, a sliding window as long as the block, and a
gated feed-forward of the width that makes the layers' weights equal. A Kabavik shape is measured beside the Gemma layout too, with a
feed-forward that makes the mean weights of a layer equal; the kernels of its latent layers beside those of the DeepSeek layout. A
Bazulorn shape is measured beside the Flint layout as well (same attention in every layer, same experts); its delta rule and its
state space beside the gated delta net with as many state elements, its short convolution beside that net's.
Prompts end inside a block, so both attentions see
the same keys. Weights are random. Every kernel of the design is timed beside its like kernel on the same rows; a
fraction of the roofline is algorithmic bytes (or FLOPs) over time over the measured peak, and ``distance`` is the ratio
of the two fractions (above 1: the design's kernel is further from its roofline).
"""
from __future__ import annotations

import dataclasses

import torch

from .. import ops
from ..config import ModelSpec, MoeSpec, Settings, named_shape
from ..ops import delta_ops, gdn_ops, mla_ops, mlstm_ops, moe_cuda, moe_ops, residual_ops, ssd_ops, stream_ops, talk_ops
from .kbench import Flusher, peaks, time_op

SIZES = {"duponex": ("duponex-2b-shape", "duponex-8b-shape"), "rudorax": ("rudorax-2k-shape", "rudorax-4k-shape"),
         "kabavik": ("kabavik-2k-shape", "kabavik-4k-shape"), "bazulorn": ("bazulorn-2k-shape", "bazulorn-4k-shape")}


def closest_spec(spec: ModelSpec) -> ModelSpec:
    """Gemma-layout shape with the layer weights of a Duponex shape of equal layers or the mean layer weights of a Kabavik shape;
    Flint-layout shape with the attention and experts of a Rudorax or Bazulorn shape."""
    l = spec.layer_specs[0]
    if spec.arch in ("rudorax", "bazulorn"):
        l = next(x for x in spec.layer_specs if x.mixer == "attention")
        m = l.moe
        return ModelSpec(name=spec.name.replace(spec.arch, "flint-layout"), arch="flint", layers=spec.layers, hidden=spec.hidden, heads=l.heads,
                         kv_heads=l.kv_heads, head_dim=l.dim, ffn=m.expert_ffn, vocab=spec.vocab, qk_norm=True, rms_eps=spec.rms_eps,
                         moe=MoeSpec(num_experts=m.num_experts, top_k=m.top_k, expert_ffn=m.expert_ffn, score="sigmoid", n_shared=1,
                                     shared_ffn=m.shared_ffn),
                         extra={"flint": {"window": l.window, "no_rope_layers": []}})
    f, window = (l.heads * l.vdim + 2 * l.ffn) // 3 // 128 * 128, l.chunk
    if spec.arch == "kabavik":
        f = (spec.run_params() // (spec.layers * spec.hidden) - 2 * (l.heads + l.kv_heads) * l.dim) // 3 // 128 * 128
        window = l.window
    return ModelSpec(name=spec.name.replace(spec.arch, "gemma-layout"), arch="gemma", layers=spec.layers, hidden=spec.hidden,
                     heads=l.heads, kv_heads=l.kv_heads, head_dim=l.dim, ffn=f, vocab=spec.vocab, qk_norm=True, swiglu_mode=2,
                     rms_eps=spec.rms_eps, extra={"gemma": {"window": window, "global_every": spec.layers + 1}})


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
    out["run_weights"] = spec.run_params() if spec.layer_specs is not None else \
        spec.layers * (spec.hidden * spec.qkv_dim + spec.q_dim * spec.hidden + 3 * spec.hidden *
                       (spec.ffn if spec.moe is None else spec.moe.top_k * spec.moe.expert_ffn + spec.moe.shared_ffn))
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


class _Pairs:
    """Times pairs of kernels on ``rows`` rows; a cost is (bytes, FLOPs)."""

    def __init__(self, rows: int, iters: int, dev):
        self.rows, self.iters, self.flush, self.pk, self.lines = rows, iters, Flusher(dev), peaks(), []

    def bound(self, byts, flops):
        return max(byts / (self.pk["hbm_gbs"] * 1e9), flops / (self.pk["bf16_tflops"] * 1e12)) * 1e6

    def __call__(self, name, mine, mine_cost, like_name, like, like_cost):
        a, b = (time_op(fn, self.iters, 3, self.flush, graph=True)["us_median"] for fn in (mine, like))
        fa, fb = self.bound(*mine_cost) / a, self.bound(*like_cost) / b
        self.lines.append({"kernel": name, "us": round(a, 2), "frac": round(fa, 3), "like": like_name, "like_us": round(b, 2),
                           "like_frac": round(fb, 3), "distance": round(fb / fa, 2)})

    def gemm(self, n, k, out_cols=None, out_bytes=2):
        return (2 * (self.rows * k + n * k) + out_bytes * self.rows * (out_cols or n), 2 * self.rows * n * k)


def kernel_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    """One line per pair: the design's kernel and its like on ``rows`` rows (``rows`` <= 128: a decode step of that batch at
    context ``ctx``; more: prefill of rows / ctx prompts)."""
    return {"duponex": _duponex_table, "rudorax": _rudorax_table, "kabavik": _kabavik_table,
            "bazulorn": _bazulorn_table}[spec.arch](spec, rows, ctx, iters, device)


def _duponex_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    l, other = spec.layer_specs[0], closest_spec(spec)
    dev, bf = torch.device(device), torch.bfloat16
    W, S, H, G, d, f = spec.hidden, int(spec.extra["duponex"]["streams"]), l.heads, l.kv_heads, l.dim, l.ffn
    rn = lambda *s: torch.randn(*s, device=dev).to(bf)
    decode = rows <= 128
    pair = _Pairs(rows, iters, dev)
    gemm_cost = pair.gemm
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
    return pair.lines


def _rudorax_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    l, mem = (next(x for x in spec.layer_specs if x.mixer == k) for k in ("attention", "mlstm"))
    dev, bf, f32 = torch.device(device), torch.bfloat16, torch.float32
    W, H, G, d, e = spec.hidden, l.heads, l.kv_heads, l.dim, l.moe
    rn = lambda *s: torch.randn(*s, device=dev).to(bf)
    fl = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda t: t.to(torch.int32)
    decode = rows <= 128
    pair = _Pairs(rows, iters, dev)
    x = rn(rows, W)
    nq, outs, f = H * d + 2 * G * d, e.num_experts + e.identity, e.expert_ffn
    # projections
    for name, n, k in (("qkv projection", nq, W), ("output projection", W, H * d)):
        w, r = rn(n, k), x if k == W else rn(rows, k)
        pair(name, lambda: ops.linear(r, w), pair.gemm(n, k), name, lambda: ops.linear(r, w), pair.gemm(n, k))
    # head norm + rotation + cache write against the two norms, the rotation and the cache write of the like layer
    batch = rows if decode else rows // ctx
    pg = _Paged(batch, ctx, G, d, dev)
    slots, pos = i32(torch.randperm(pg.k.shape[0] * 64, device=dev)[:rows]), i32(torch.arange(rows, device=dev)) % ctx
    qkv, qn, kn = rn(rows, nq), rn(d), rn(d)
    freqs, amp = l.rope.frequencies()
    fr = ops.rope_frequencies(freqs, dev)
    table = ops.rope_angles(pos, fr, amp)

    def like_norm_rope():
        q, k = qkv[:, : H * d].reshape(rows * H, d), qkv[:, H * d: (H + G) * d].reshape(rows * G, d)
        qkv[:, : H * d] = ops.rmsnorm(q.contiguous(), qn, 1e-5).view(rows, -1)
        qkv[:, H * d: (H + G) * d] = ops.rmsnorm(k.contiguous(), kn, 1e-5).view(rows, -1)
        ops.rope_kv_paged(qkv, pos, slots, pg.k, pg.v, H, G, d, 1e4)
    byts = 2 * rows * d * (2 * H + 2 * G + 2 * G)
    qnf, knf = qn.float(), kn.float()
    pair("head norm + rotation + cache write", lambda: ops.head_norm_kv(qkv, slots, pg.k, pg.v, H, G, d, d, 1e-5, q_weight=qnf, k_weight=knf, cos_sin=table),
         (byts, 0), "head norms, rotation + cache write", like_norm_rope, (byts, 0))
    pair("angles of a step", lambda: ops.rope_angles(pos, fr, amp), (rows * d * 4, 0), "angles of a step", lambda: ops.rope_table(pos, d, 1e4), (rows * d * 4, 0))
    # attention
    sinks = fl(H)
    if decode:
        cost = (2 * rows * (2 * l.keys_seen(ctx) * G * d + 2 * H * d), 4 * rows * l.keys_seen(ctx) * H * d)
        at = lambda: ops.attn_decode(qkv, pg.k, pg.v, pg.table, pg.ctx, H, G, d, l.scale, max_ctx=ctx, window=l.window, sinks=sinks)
    else:
        qs, ql = i32(torch.arange(batch, device=dev) * ctx), torch.full((batch,), ctx, dtype=torch.int32, device=dev)
        cost = (2 * rows * (2 * H * d + 2 * G * d), 4 * batch * l.pairs_seen(ctx) * H * d)
        at = lambda: ops.attn_prefill(qkv, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, H, G, d, l.scale, window=l.window, sinks=sinks)
    pair("attention, window + sinks", at, cost, "attention, window + sinks", at, cost)
    del pg, qkv
    # router, experts
    wr, corr = rn((outs + 15) // 16 * 16, W) * 0.02, fl(outs) * 0.01
    pair("router, 32-bit logits", lambda: moe_ops.route(x, wr, e.top_k, "softmax", corr, exact=True, experts=outs), pair.gemm(outs, W, out_bytes=8),
         "router", lambda: moe_ops.route(x, wr[: e.num_experts], e.top_k, "sigmoid"), pair.gemm(e.num_experts, W, out_bytes=4))
    weights, ids = moe_ops.route(x, wr, e.top_k, "softmax", corr, exact=True, experts=outs)
    lw, lids = moe_ops.route(x, wr[: e.num_experts], e.top_k, "sigmoid")
    gu, down = rn(e.num_experts, 2 * f, W), rn(e.num_experts, W, f)

    def expert_cost(ids):
        served = int((ids < e.num_experts).sum())
        touched = int(torch.unique(ids[ids < e.num_experts]).numel())
        return (2 * (touched * 3 * f * W + served * (2 * W + 3 * f)), 2 * served * 3 * f * W)
    holder = {}

    def like_experts():
        xs, p, so, ct, cap = moe_cuda.dispatch_local(x, lids, e.num_experts, 0, e.num_experts)
        rpe = rows * e.top_k / e.num_experts
        h = moe_cuda.grouped_gemm(xs, gu, so, ct, cap, epi=1, rows_per_expert=rpe)
        holder["y"], holder["pos"] = moe_cuda.grouped_gemm(h, down, so, ct, cap, epi=0, rows_per_expert=rpe), p
    add = lambda p, q: (p[0] + q[0], p[1] + q[1])

    def like_routed():
        moe_ops.route(x, wr[: e.num_experts], e.top_k, "sigmoid")
        like_experts()
    pair("router, dispatch, two grouped GEMMs", lambda: moe_ops.routed_rows(x, wr, e.top_k, "softmax", corr, outs, gu, down),
         add(expert_cost(ids), pair.gemm(outs, W, out_bytes=8)), "router, dispatch, two grouped GEMMs", like_routed,
         add(expert_cost(lids), pair.gemm(e.num_experts, W, out_bytes=4)))
    er = moe_ops.expert_rows(x, weights, ids, gu, down)
    like_experts()
    sg, sd = rn(2 * e.shared_ffn, W), rn(W, e.shared_ffn)
    cost = (2 * (3 * e.shared_ffn * W + rows * (2 * W + 2 * e.shared_ffn)), 6 * rows * e.shared_ffn * W)
    pair("shared expert", lambda: ops.linear(ops.linear_swiglu(x, sg), sd), cost, "shared expert",
         lambda: ops.linear(ops.silu_mul(ops.linear(x, sg)), sd), cost)
    # the layer's end: sums and the next norms
    xs, a, b, w1, w2, w16, r16 = fl(rows, W), rn(rows, W), rn(rows, W), fl(W), fl(W), rn(W), rn(rows, W)

    def like_end():
        y = moe_cuda.combine(holder["y"], holder["pos"], lids, lw, rows, W)
        ops.add_rmsnorm(a, r16, w16, 1e-5)
        ops.add_rmsnorm(moe_ops.add_shared(y, b), r16, w16, 1e-5)
    pair("residual step (all sums, two norms)", lambda: residual_ops.step(xs, a, b, er, w1, w2, 1e-5, W), (rows * W * (8 + 4 + 4 + 2 * e.top_k), 0),
         "expert sum, shared sum, two add + norm", like_end, (rows * W * (2 * e.top_k + 2 * 6), 0))
    tok, tab = i32(torch.randint(0, 1024, (rows,), device=dev)), rn(1024, W)
    pair("embed + two norms", lambda: residual_ops.embed(tok, tab, 2.0, w1, w2, 1e-5, W), (rows * W * 10, 0), "embed + norm",
         lambda: ops.embed_rmsnorm(tok, tab, w16, 1e-5), (rows * W * 6, 0))
    del gu, down, er, holder, xs
    # matrix memory against the gated delta net (128 x 128 heads, as many state elements)
    M, dk, dv = mem.heads, mem.dim_pad, mem.vdim_pad
    pn = mem.projection_cols
    wp = rn(pn, W)
    pair("memory projection", lambda: ops.linear(x, wp), pair.gemm(pn, W), "qkv projection, same size", lambda: ops.linear(x, wp), pair.gemm(pn, W))
    wg = rn(max(2 * M, 16), W) * 0.02
    pair("gate logits, 32-bit", lambda: ops.linear(x, wg, out_dtype=f32), pair.gemm(wg.shape[0], W, out_bytes=4), "projection of that size",
         lambda: ops.linear(x, wg), pair.gemm(wg.shape[0], W))
    del wp
    st = mlstm_ops.MemoryState(batch, M, dk, dv, dev)
    packed, gates, gb, o = rn(rows, pn), fl(rows, wg.shape[0]), fl(2 * M), torch.empty(rows, M, dv, device=dev)
    starts = i32(torch.arange(batch + 1, device=dev) * (rows // batch))
    sl = i32(torch.randperm(batch, device=dev))
    V = M * dv // 128
    q, k, v = (fl(rows, V, 128) for _ in range(3))
    beta, dec = torch.rand(rows, V, device=dev), -torch.rand(rows, V, device=dev)
    gst = torch.zeros(batch, V, 128, 128, device=dev)
    state = 8 * batch * M * dk * dv
    flops = 4 * rows * M * dk * dv + (0 if decode else 2 * rows * 64 * M * (dk + dv))       # prompts: and the triangle inside a chunk
    gflops = 4 * rows * V * 128 * 128 + (0 if decode else 2 * rows * 64 * V * 128 * 4)
    pair("memory recurrence" if decode else "memory, chunked", lambda: mlstm_ops.memory(packed, gates, gb, mem.gate_cap, st, starts, sl, mem.scale, o, rows // batch),
         (state + rows * M * (4 * dk + 2 * dv + 4 * dv + 8), flops), "gated delta net recurrence" if decode else "gated delta net, chunked",
         (lambda: gdn_ops.recurrent_slots(q, k, v, beta, dec, gst, starts, sl)) if decode else (lambda: gdn_ops.chunked_slots(q, k, v, beta, dec, gst, starts, sl)),
         (8 * batch * V * 128 * 128 + rows * V * 128 * (12 + 2), gflops))
    gate, wn, z = packed[:, M * (2 * dk + dv):], fl(M * dv), rn(rows, V * 128)
    on = rn(rows * V, 128)
    pair("head norm + output gate", lambda: mlstm_ops.head_out(o, gate, wn, dv, 1e-5), (rows * M * dv * 8, 0), "head norm, output gate",
         lambda: (ops.rmsnorm(on, qn, 1e-5).view(rows, -1).float() * torch.nn.functional.silu(z.float())).to(bf), (rows * M * dv * 8, 0))
    # vocabulary logits of a step
    if decode:
        wv = rn(spec.vocab, W)
        pair("logits, 32-bit, soft cap", lambda: ops.softcap(ops.linear(x, wv, out_dtype=f32), 30.0), pair.gemm(spec.vocab, W, out_bytes=4), "logits",
             lambda: ops.linear(x, wv), pair.gemm(spec.vocab, W))
    ops.check_status()
    return pair.lines


def _kabavik_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    win, lat, cap = (next(l for l in spec.layer_specs if pick(l)) for pick in (lambda l: l.qk_norm == "row", lambda l: l.mixer == "latent", lambda l: l.softcap))
    other = closest_spec(spec)
    dev, bf, f32 = torch.device(device), torch.bfloat16, torch.float32
    W, H, G, d, f, fo, side = spec.hidden, win.heads, win.kv_heads, win.dim, win.ffn, other.ffn, spec.side_dim
    rn = lambda *s: torch.randn(*s, device=dev).to(bf)
    fl = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda t: t.to(torch.int32)
    decode = rows <= 128
    pair = _Pairs(rows, iters, dev)
    x = rn(rows, W)
    nq = (H + 2 * G) * d
    # projections
    for name, n, k, like in (("qkv projection, bias", nq, W, "qkv projection"), ("output projection, bias", W, H * d, "output projection")):
        w, b, r = rn(n, k), rn(n), x if k == W else rn(rows, k)
        pair(name, lambda: ops.linear(r, w, bias=b), pair.gemm(n, k), like, lambda: ops.linear(r, w), pair.gemm(n, k))
    wgu, wgo, h1, h2, wd, wdo = rn(2 * f, W), rn(2 * fo, W), rn(rows, f), rn(rows, fo), rn(W, f), rn(W, fo)
    pair("gate/up projection, tanh-GELU", lambda: ops.linear_swiglu(x, wgu, mode=3), pair.gemm(2 * f, W, f), "gate/up projection, tanh-GELU",
         lambda: ops.linear_swiglu(x, wgo, mode=2), pair.gemm(2 * fo, W, fo))
    pair("down projection", lambda: ops.linear(h1, wd), pair.gemm(W, f), "down projection", lambda: ops.linear(h2, wdo), pair.gemm(W, fo))
    del wgu, wgo, h1, h2, wd, wdo
    # the residual between two sub-layers
    xs, y, r16, w16, vec = fl(rows, W), rn(rows, W), rn(rows, W), rn(W), lambda: fl(W)
    tanh = lambda: residual_ops.Norm("tanh", vec(), vec(), 0.7)
    n1, n2, n3, copy = tanh(), tanh(), residual_ops.Norm("rms", vec()), residual_ops.Norm()

    def like_step():
        ops.add_rmsnorm(ops.rmsnorm(y, w16, 1e-5), r16, w16, 1e-5)
    for name, a, b in (("residual step, two tanh norms", n1, n2), ("residual step, tanh norm and copy", n1, copy), ("residual step, RMS and tanh norm", n3, n2)):
        pair(name, lambda: residual_ops.add_normed(xs, y, a, b, 1e-5, W), (rows * W * 12, 0), "norm, add + norm", like_step, (rows * W * 12, 0))
    tok, tab = i32(torch.randint(0, 1024, (rows,), device=dev)), rn(1024, W)
    pair("embed + norm", lambda: residual_ops.embed_normed(tok, tab, 2.0, n1, 1e-5, W), (rows * W * 8, 0), "embed + norm",
         lambda: ops.embed_rmsnorm(tok, tab, w16, 1e-5), (rows * W * 6, 0))
    # token input
    wg, wp, es, g1 = rn(side, W), rn(W, side), rn(1024, 4 * side), rn(rows, side)
    cost = pair.gemm(side, W)
    pair("token gate, tanh-GELU, factors", lambda: ops.linear(x, wg, act="gelu_tanh", mul=(es[:, side: 2 * side], tok)), (cost[0] + 2 * rows * side, cost[1]),
         "projection of that size", lambda: ops.linear(x, wg), cost)
    pair("token projection", lambda: ops.linear(g1, wp), pair.gemm(W, side), "projection of that size", lambda: ops.linear(g1, wp), pair.gemm(W, side))
    del xs, tab, es
    # norms, rotation and cache write
    batch = rows if decode else rows // ctx
    pg = _Paged(batch, ctx, G, d, dev)
    slots, pos = i32(torch.randperm(pg.k.shape[0] * 64, device=dev)[:rows]), i32(torch.arange(rows, device=dev)) % ctx
    qkv, qn, kn, wq, wk = rn(rows, nq), rn(d), rn(d), fl(H * d), fl(G * d)
    freqs, amp = win.rope.frequencies()
    table = ops.rope_angles(pos, ops.rope_frequencies(freqs, dev), amp)

    def like_norm_rope():
        q, k = qkv[:, : H * d].reshape(rows * H, d), qkv[:, H * d: (H + G) * d].reshape(rows * G, d)
        qkv[:, : H * d] = ops.rmsnorm(q.contiguous(), qn, 1e-5).view(rows, -1)
        qkv[:, H * d: (H + G) * d] = ops.rmsnorm(k.contiguous(), kn, 1e-5).view(rows, -1)
        ops.rope_kv_paged(qkv, pos, slots, pg.k, pg.v, H, G, d, 1e4)
    byts = (2 * rows * d * (2 * H + 4 * G), 0)
    pair("row norms, rotation + cache write", lambda: ops.head_norm_kv(qkv, slots, pg.k, pg.v, H, G, d, d, 1e-5, q_weight=wq, k_weight=wk, cos_sin=table,
         whole=True, halves=True), byts, "head norms, rotation + cache write", like_norm_rope, byts)
    pair("head norms, temperature + cache write", lambda: ops.head_norm_kv(qkv, slots, pg.k, pg.v, H, G, d, d, 1e-5, q_weight=wq[:d], k_weight=wk[:d],
         temp=(pos, *cap.q_temp)), byts, "head norms, rotation + cache write", like_norm_rope, byts)
    # attention
    qs, ql = (i32(torch.arange(batch, device=dev) * (rows // batch)), torch.full((batch,), rows // batch, dtype=torch.int32, device=dev))
    seen = lambda l: batch * (l.keys_seen(ctx) if decode else l.pairs_seen(ctx))       # (query, key) pairs

    def cost(l, kv_width, pairs, q_width, flop_width):
        keys = rows * l.keys_seen(ctx) if decode else rows
        return 2 * (keys * kv_width + rows * H * q_width), 2 * pairs * H * flop_width
    plain = dataclasses.replace(win, keep_first=0)
    full = dataclasses.replace(win, window=0)
    for name, l, like_name, like in (("attention, window + kept positions", win, "attention, window", plain),
                                     ("attention, capped scores", cap, "attention, full", full)):
        def at(z):
            kw = dict(window=z.window, keep=z.keep_first if z.window else 0, softcap=z.softcap)
            if decode:
                return ops.attn_decode(qkv, pg.k, pg.v, pg.table, pg.ctx, H, G, d, l.scale, max_ctx=ctx, **kw)
            return ops.attn_prefill(qkv, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, H, G, d, l.scale, **kw)
        pair(name, lambda: at(l), cost(l, 2 * G * d, seen(l), 2 * d, 2 * d), like_name, lambda: at(like), cost(like, 2 * G * d, seen(like), 2 * d, 2 * d))
    del pg, qkv
    # latent attention
    R, T = lat.rank_pad, lat.rot_pad
    n = lat.projection_cols
    w = rn(n, W)
    pair("latent projection", lambda: ops.linear(x, w), pair.gemm(n, W), "projection of that size", lambda: ops.linear(x, w), pair.gemm(n, W))
    p, wn = rn(rows, n), fl(R)
    lg = _Paged(batch, ctx, 1, R + T, dev)
    lfreqs, lamp = lat.rope.frequencies()
    ltab = ops.rope_angles(pos, ops.rope_frequencies(lfreqs, dev), lamp)
    q = torch.empty(rows, H, R + T, dtype=bf, device=dev)
    rot, at0 = H * d, H * (d + T)
    byts = (2 * rows * (2 * H * T + 2 * (R + T)), 0)

    def like_latent():
        c = ops.rmsnorm(p[:, at0: at0 + R].contiguous(), w16[:R].contiguous(), 1e-5)
        kr, qr = p[:, at0 + R: at0 + R + T].contiguous(), p[:, rot: at0].contiguous()
        ops.rope_inplace(qr, pos, H, T, 1e4)
        ops.rope_inplace(kr, pos, 1, T, 1e4)
        mla_ops.cache_write(c, kr, slots, lg.k)
    pair("latent norm, rotations + cache write", lambda: mla_ops.latent_norm_kv(p, slots, lg.k, q, rot, at0, R, R, wn, ltab, 1e-5), byts,
         "norm, rotations, cache write", like_latent, byts)
    uk, uv, out = rn(H, R, d), rn(H, d, R), rn(rows, H * R)
    per_head = lambda a, b: (2 * (rows * H * (a + b) + H * a * b), 2 * rows * H * a * b)
    xq = p[:, :rot]
    pair("queries into the latent space", lambda: ops.head_linear(xq, uk, out=q.view(rows, -1), out_cols=R + T), per_head(d, R), "per-head projection",
         lambda: mla_ops.per_head_linear(xq.reshape(rows, H, d), uk), per_head(d, R))
    pair("results out of the latent space", lambda: ops.head_linear(out, uv), per_head(R, d), "per-head projection",
         lambda: mla_ops.per_head_linear(out.view(rows, H, R), uv), per_head(R, d))
    q.normal_()
    gate = p[:, at0 + R + T: at0 + R + T + H]
    unbound = dataclasses.replace(lat, window=0)
    lc = lambda l: cost(l, R + T, seen(l), 2 * R + T, 2 * R + T)
    like = lambda: mla_ops.attention(q, lg.k, lg.table, qs, ql, lg.ctx, rows // batch, ctx, lat.scale, R)
    if decode:
        pair("latent attention, window, gated", lambda: mla_ops.latent_attention(q, lg.k, lg.table, qs, ql, lg.ctx, 1, ctx, lat.scale, R, lat.window, gate, out,
             decode=True), lc(lat), "latent attention, full", like, lc(unbound))
    else:       # prompts: expansion and attention here, the latent space there; the cost is that of the expanded form for both
        def like_latent_attention():
            mla_ops.per_head_linear(xq.reshape(rows, H, d), uk)
            mla_ops.per_head_linear(like(), uv)
        pages = mla_ops.KeyPages.of([ctx] * batch, [ctx] * batch, lg.table.cpu(), lat.window, 64, dev)
        w_kv, res = rn(H * 2 * d, R), rn(rows, H * d)
        expansion, ec = pair.gemm(H * 2 * d, R), lambda l: cost(l, R + T, seen(l), 2 * d + T, 2 * d + T)
        add = lambda a, b: (a[0] + b[0], a[1] + b[1])
        pair("latents expanded, attention, window, gated", lambda: mla_ops.expanded_attention(xq, q, lg.k, w_kv, pages, lg.table, qs, ql, lg.ctx, ctx, d, d, R,
             lat.scale, lat.window, gate, res), add(expansion, ec(lat)), "queries to latents, attention, results out of latents",
             like_latent_attention,
             add(expansion, ec(unbound)))
    if decode:
        wv = rn(spec.vocab, W)
        pair("logits, 32-bit", lambda: ops.linear(x, wv, out_dtype=f32), pair.gemm(spec.vocab, W, out_bytes=4), "logits", lambda: ops.linear(x, wv),
             pair.gemm(spec.vocab, W))
    ops.check_status()
    return pair.lines


def _bazulorn_table(spec: ModelSpec, rows: int, ctx: int, iters: int, device) -> list[dict]:
    delta, both = (next(x for x in spec.layer_specs if x.mixer == k) for k in ("channel_delta", "attention"))
    ssd, e = both.beside, both.moe
    dev, bf, f32 = torch.device(device), torch.bfloat16, torch.float32
    W, H, G, d, f = spec.hidden, both.heads, both.kv_heads, both.dim, e.expert_ffn
    rn = lambda *s: torch.randn(*s, device=dev).to(bf)
    fl = lambda *s: torch.randn(*s, device=dev)
    i32 = lambda t: t.to(torch.int32)
    decode = rows <= 128
    batch = rows if decode else rows // ctx
    pair = _Pairs(rows, iters, dev)
    x = rn(rows, W)
    starts, sl = i32(torch.arange(batch + 1, device=dev) * (rows // batch)), i32(torch.randperm(batch, device=dev))
    # projections
    nd, nb = delta.projection_cols, both.projection_cols
    for name, n, k in (("delta projection", nd, W), ("projection of the pair, bias", nb, W), ("output projection", W, H * d)):
        w, r, b = rn(n, k), x if k == W else rn(rows, k), rn(n) if "bias" in name else None
        pair(name, lambda: ops.linear(r, w, bias=b), pair.gemm(n, k), "projection of that size", lambda: ops.linear(r, w), pair.gemm(n, k))
    wr, low = rn(delta.heads * delta.dim, delta.decay_rank), rn(rows, delta.decay_rank)
    n = wr.shape[0]
    pair("decay logits, 32-bit", lambda: ops.linear(low, wr, out_dtype=f32), pair.gemm(n, delta.decay_rank, out_bytes=4), "projection of that size",
         lambda: ops.linear(low, wr), pair.gemm(n, delta.decay_rank))
    # convolutions
    V = delta.heads
    for name, l, unit in (("short convolution, unit factors", delta, 0.1), ("short convolution, bias", ssd, None)):
        conv = delta_ops.ConvWeights(fl(l.conv, l.conv_pad), None if unit else fl(l.conv_pad), 2 * l.kv_heads, l.dim_pad, l.heads, l.vdim_pad)
        ch, cs = l.conv_pad, delta_ops.ConvState(batch, conv, dev)
        px, gw, hist = rn(rows, ch), rn(ch, 4), torch.zeros(batch, ch, 3, device=dev)
        cost = (rows * ch * 4 + batch * ch * 24, 0)
        pair(name, lambda: delta_ops.short_conv(px, conv, cs, starts, sl, rows // batch, unit_scale=unit), cost, "convolution of the gated delta net",
             lambda: gdn_ops.conv_batched(px, gw, hist, starts, sl), cost)
    del px, hist, cs
    # recurrences against the gated delta net
    def like_net(V):
        q, k, v = (fl(rows, V, 128) for _ in range(3))
        k = k / k.norm(dim=-1, keepdim=True)
        beta, dec, gst = torch.rand(rows, V, device=dev), -torch.rand(rows, V, device=dev), torch.zeros(batch, V, 128, 128, device=dev)
        run = gdn_ops.recurrent_slots if decode else gdn_ops.chunked_slots
        flops = 4 * rows * V * 128 * 128 + (0 if decode else 2 * rows * 64 * V * 128 * 4)
        return lambda: run(q, k, v, beta, dec, gst, starts, sl), (8 * batch * V * 128 * 128 + rows * V * 128 * 14, flops)
    form = "recurrence" if decode else "chunked"
    cx, unit, dz, db, o = rn(rows, delta.conv_pad), fl(rows, 2 * V).abs() * 0.01, fl(rows, V * 128), rn(rows, V), torch.empty(rows, V, 128, device=dev)
    unit = torch.rsqrt((cx[:, : 2 * V * 128].float().view(rows, 2 * V, 128) ** 2).sum(-1) + 1e-6)
    st, rate, dtb = delta_ops.DeltaState(batch, V, delta.kv_heads, 128, 128, dev), -torch.rand(V, device=dev), fl(V * 128) - 4.0
    like, like_cost = like_net(V)
    pair(f"delta rule by channel, {form}", lambda: delta_ops.delta_rule(cx, unit, dz, db, rate, dtb, st, starts, sl, o, rows // batch),
         (8 * batch * V * 128 * 128 + rows * V * 128 * (3 * 2 + 4 + 4), like_cost[1]), f"gated delta net, {form}", like, like_cost)
    gate, wn, z, qn, on = rn(rows, V * 128), fl(128), rn(rows, V * 128), rn(128), rn(rows * V, 128)
    like_out = lambda: (ops.rmsnorm(on, qn, 1e-5).view(rows, -1).float() * torch.nn.functional.silu(z.float())).to(bf)
    pair("head norm + output gate", lambda: delta_ops.head_out(o, gate, wn, 128, 1e-5), (rows * V * 128 * 8, 0), "head norm, output gate", like_out,
         (rows * V * 128 * 8, 0))
    del cx, dz, st, like
    M, dk, dv = ssd.heads, ssd.dim_pad, ssd.vdim_pad
    cx, steps, sb, sa, skip, o = rn(rows, ssd.conv_pad), rn(rows, M), fl(M) - 4.0, -torch.rand(M, device=dev), fl(M), torch.empty(rows, M, dv, device=dev)
    st = ssd_ops.SsdState(batch, M, ssd.kv_heads, dk, dv, dev)
    like, like_cost = like_net(M * dk * dv // (128 * 128))
    flops = 4 * rows * M * dk * dv + (0 if decode else 2 * rows * 64 * M * (dk + dv))
    pair(f"state space, {form}", lambda: ssd_ops.state_space(cx, steps, sb, sa, skip, st, starts, sl, o, rows // batch),
         (8 * batch * M * dk * dv + rows * (2 * ssd.conv_pad + M * dv * 4), flops), f"gated delta net, {form}", like, like_cost)
    sz, sw = rn(rows, M * dv), fl(M * dv)
    pair("output gate + norm of groups", lambda: ssd_ops.gated_out(o, sz, sw, dv, ssd.norm_groups, 1e-5), (rows * M * dv * 8, 0), "head norm, output gate", like_out,
         (rows * V * 128 * 8, 0))
    del cx, st, like, o, sz, gate, z, on
    # value norm + cache write, attention
    pg = _Paged(batch, ctx, G, d, dev)
    slots, pos = i32(torch.randperm(pg.k.shape[0] * 64, device=dev)[:rows]), i32(torch.arange(rows, device=dev)) % ctx
    qkv = rn(rows, (H + 2 * G) * d)
    pair("value norm + cache write", lambda: ops.head_norm_kv(qkv, slots, pg.k, pg.v, H, G, d, d, 1e-5, norm_qk=False, norm_v=True), (2 * rows * d * 4 * G, 0),
         "rotation + cache write", lambda: ops.rope_kv_paged(qkv, pos, slots, pg.k, pg.v, H, G, d, 1e4), (2 * rows * d * (2 * H + 4 * G), 0))
    talk, sinks, out = fl(H, H), fl(H), torch.empty(rows, H * d, dtype=bf, device=dev)
    mine, plain = H * (4 * d + 2 * H), H * 4 * d
    args = (H, G, both.scale, both.window, talk, True)
    if decode:
        byts, seen = 2 * rows * (2 * both.keys_seen(ctx) * G * d + 2 * H * d), rows * both.keys_seen(ctx)
        pair("attention, window, mixed heads", lambda: talk_ops.talk_decode(qkv, pg.k, pg.v, pg.table, pg.ctx, ctx, *args, out=out), (byts, seen * mine),
             "attention, window + sinks", lambda: ops.attn_decode(qkv, pg.k, pg.v, pg.table, pg.ctx, H, G, d, both.scale, max_ctx=ctx, window=both.window,
             sinks=sinks), (byts, seen * plain))
    else:
        qs, ql = i32(torch.arange(batch, device=dev) * ctx), torch.full((batch,), ctx, dtype=torch.int32, device=dev)
        byts, seen = 2 * rows * (2 * H * d + 2 * G * d), batch * both.pairs_seen(ctx)
        pair("attention, window, mixed heads", lambda: talk_ops.talk_prefill(qkv, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, ctx, *args, out=out),
             (byts, seen * mine), "attention, window + sinks", lambda: ops.attn_prefill(qkv, pg.k, pg.v, pg.table, qs, ql, pg.ctx, ctx, H, G, d, both.scale,
             window=both.window, sinks=sinks), (byts, seen * plain))
    del pg, qkv, out
    # router, experts
    wr, bias = rn((e.num_experts + 15) // 16 * 16, W) * 0.02, fl(e.num_experts) * 0.01
    gu, down = rn(e.num_experts, 2 * f, W), rn(e.num_experts, W, f)
    weights, ids = moe_ops.route(x, wr, e.top_k, e.score, bias, exact=True, experts=e.num_experts)
    lw, lids = moe_ops.route(x, wr[: e.num_experts], e.top_k, "sigmoid")
    holder = {}

    def expert_cost(ids):
        touched = int(torch.unique(ids).numel())
        return (2 * (touched * 3 * f * W + ids.numel() * (2 * W + 3 * f)), 2 * ids.numel() * 3 * f * W)

    def like_routed():
        moe_ops.route(x, wr[: e.num_experts], e.top_k, "sigmoid")
        xs, p, so, ct, cap = moe_cuda.dispatch_local(x, lids, e.num_experts, 0, e.num_experts)
        rpe = rows * e.top_k / e.num_experts
        h = moe_cuda.grouped_gemm(xs, gu, so, ct, cap, epi=1, rows_per_expert=rpe)
        holder["y"], holder["pos"] = moe_cuda.grouped_gemm(h, down, so, ct, cap, epi=0, rows_per_expert=rpe), p
    add = lambda p, q: (p[0] + q[0], p[1] + q[1])
    pair("router, dispatch, two grouped GEMMs, clamped gate", lambda: moe_ops.routed_rows(x, wr, e.top_k, e.score, bias, e.num_experts, gu, down, e.limit),
         add(expert_cost(ids), pair.gemm(e.num_experts, W, out_bytes=8)), "router, dispatch, two grouped GEMMs", like_routed,
         add(expert_cost(lids), pair.gemm(e.num_experts, W, out_bytes=4)))
    er = moe_ops.expert_rows(x, weights, ids, gu, down, e.limit)
    like_routed()
    sg, sd = rn(2 * e.shared_ffn, W), rn(W, e.shared_ffn)
    cost = (2 * (3 * e.shared_ffn * W + rows * (2 * W + 2 * e.shared_ffn)), 6 * rows * e.shared_ffn * W)
    pair("shared expert, clamped gate", lambda: ops.linear(ops.linear_swiglu(x, sg, mode=5, limit=e.shared_limit), sd), cost, "shared expert",
         lambda: ops.linear(ops.silu_mul(ops.linear(x, sg)), sd), cost)
    # the layer's end and its begin
    xs, a, b, r, w1, w2, w3, w16, r16 = fl(rows, W), rn(rows, W), rn(rows, W), rn(rows, W), fl(W), fl(W), fl(W), rn(W), rn(rows, W)

    def like_end():
        y = moe_cuda.combine(holder["y"], holder["pos"], lids, lw, rows, W)
        ops.add_rmsnorm(a, r16, w16, 1e-5)
        ops.add_rmsnorm(moe_ops.add_shared(y, b), r16, w16, 1e-5)
    pair("residual step (all sums, three norms)", lambda: residual_ops.step(xs, a, b, er, w1, None, 1e-5, W, beside=residual_ops.Beside(r, w2, w3)),
         (rows * W * (8 + 2 + 6 + 2 * e.top_k), 0), "expert sum, shared sum, two add + norm", like_end, (rows * W * (2 * e.top_k + 2 * 6), 0))
    tok, tab = i32(torch.randint(0, 1024, (rows,), device=dev)), rn(1024, W)
    last = torch.full((batch,), -1, dtype=torch.int32, device=dev)
    big = lambda: residual_ops.bigram_rows(tok, last, starts, sl, buckets=1021, mul_prev=37, mul_cur=3)
    pair("bigram rows, embed of two tables + norms", lambda: residual_ops.embed(tok, tab, 1.0, w1, None, 1e-5, W, second=residual_ops.Second(tab, big(), w2)),
         (rows * W * 10, 0), "embed + norm", lambda: ops.embed_rmsnorm(tok, tab, w16, 1e-5), (rows * W * 6, 0))
    del gu, down, er, holder, xs
    if decode:
        wv = rn(spec.vocab, W)
        pair("logits, 32-bit", lambda: ops.linear(x, wv, out_dtype=f32), pair.gemm(spec.vocab, W, out_bytes=4), "logits", lambda: ops.linear(x, wv),
             pair.gemm(spec.vocab, W))
    ops.check_status()
    return pair.lines


def run(device, steps: int, warmup: int, design: str = "duponex", batches=(1, 8, 64), prompt: int = 1024, layers: int | None = None) -> dict:
    out: dict = {"design": design, "prompt": prompt, "peaks": peaks(), "sizes": {}}
    for name in SIZES[design]:
        spec = named_shape(name)
        if layers:
            spec = dataclasses.replace(spec, layer_specs=spec.layer_specs[:layers], loop=None)
            spec.layers = len(spec.runs)
        other = closest_spec(spec)
        out["sizes"][name] = {
            "closest": {"name": other.name, "ffn": other.ffn},
            design: model_throughput(spec, prompt, batches, steps, warmup, device),
            "closest_model": model_throughput(other, prompt, batches, steps, warmup, device),
            "kernels": {"decode rows 64, context 1024": kernel_table(spec, 64, 1024, 30, device),
                        "prefill 8 x 1024": kernel_table(spec, 8192, 1024, 15, device),
                        "prefill 1 x 8192": kernel_table(spec, 8192, 8192, 15, device)}}
    return out
