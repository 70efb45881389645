"""Duponex decoder against the plain restatement in ``duponex_oracle``: every mechanism alone, whole prompts, portions,
mixed batches, decoding, block edges, recycled cache blocks, sizes that need padding, and generation through the
scheduler. Every case runs on the CPU oracles of the operators and, on a GPU, through the kernels in BF16 and FP32."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import duponex_oracle as O
from _design import GPU, TORCH, close, each_form, feed_in_cuts, ids, load, paged, write
from flyingfish_b200 import ops
from flyingfish_b200.api import Model, generate_plain
from flyingfish_b200.config import ConfigError, Settings, named_shape, read_model_spec, spec_from_hf_config
from flyingfish_b200.engine.engine import Span
from flyingfish_b200.engine.scheduler import Request, Scheduler
from flyingfish_b200.loaders.checkpoint import CheckpointError
from flyingfish_b200.loaders.safetensors_io import save_safetensors
from flyingfish_b200.ops import stream_ops


# unequal layers: sizes, masks, a layer without value mixing in front of the mixing ones, one without a feed-forward
LAYERS = [O.layer(v_mix=False, kv_heads=1, vdim=16), O.layer(), O.layer(size=37, dim=48, heads=6, kv_heads=2, scale=0.25), O.layer(ff=None, size=64)]
CFG = O.config(LAYERS, streams=3)


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    w = O.tensors(CFG)
    return write(tmp_path_factory.mktemp("duponex"), CFG, w), w


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@each_form
@pytest.mark.parametrize("streams,width,true_width", [(1, 64, 64), (2, 104, 100), (3, 256, 256), (4, 1024, 1024), (5, 40, 40), (11, 64, 61)])
def test_stream_embed_and_step(device, dtype, streams, width, true_width):
    g = torch.Generator().manual_seed(streams)
    dt, rows, eps = TORCH[dtype], 7, 1e-3
    rn = lambda *s: torch.randn(*s, generator=g)
    mask = (torch.arange(width) < true_width).float()
    table, norm, chan = (rn(30, width) * mask).to(dt), ((1 + 0.3 * rn(width)) * mask).to(dt), ((1 + 0.5 * rn(width)) * mask).to(dt)
    read, nxt, out, mix = rn(streams), rn(streams), rn(streams), rn(streams, streams)
    tok = torch.randint(0, 30, (rows,), generator=g).to(torch.int32)
    y = (rn(rows, width) * mask).to(dt)
    x, n = stream_ops.embed(tok.to(device), table.to(device), 1.7, read.to(device), norm.to(device), eps, true_width)
    e = table.double()[tok.long()] * 1.7
    xs = e[None].repeat(streams, 1, 1)
    lim = 1e-5 if dtype == "fp32" else 8e-3
    close(x.transpose(0, 1), xs, dtype, "streams", 1e-6)
    t = slice(0, true_width)
    want = O.rms(O.stream_read(xs, read.double())[:, t], eps) * norm.double()[t]
    close(n[:, t], want, dtype, "embed norm", lim)
    coef = torch.cat([nxt, 0.6 * out, mix.reshape(-1)]).to(device)
    n = stream_ops.step(x, y.to(device), chan.to(device), coef, norm.to(device), eps, true_width)
    xs = O.stream_write(xs, y.double() * chan.double(), mix.double(), out.double(), 0.6)
    close(x.transpose(0, 1), xs, dtype, "written streams", 1e-5)
    close(n[:, t], O.rms(O.stream_read(xs, nxt.double())[:, t], eps) * norm.double()[t], dtype, "step norm", lim)
    assert (n[:, true_width:] == 0).all()
    before = x.clone()
    stream_ops.step(x, y.to(device), chan.to(device), coef, norm.to(device), eps, true_width, write=False)
    assert torch.equal(before, x)


@each_form
@pytest.mark.parametrize("m", [1, 5, 130])
@pytest.mark.parametrize("n,k", [(200, 104), (72, 40), (264, 512)])
def test_linear_bias_and_squared_relu(device, dtype, m, n, k):
    g = torch.Generator().manual_seed(m)
    dt = TORCH[dtype]
    x, w, b = (torch.randn(*s, generator=g).to(dt) for s in ((m, k), (n, k), (n,)))
    ref = x.double() @ w.double().T
    dev = lambda t: t.to(device)
    lim = 1e-5 if dtype == "fp32" else 8e-3
    close(ops.linear(dev(x), dev(w), bias=dev(b)), ref + b.double(), dtype, "bias", lim)
    close(ops.linear(dev(x), dev(w), act="relu2"), O.relu_squared(ref), dtype, "relu2", lim)
    close(ops.linear(dev(x), dev(w), bias=dev(b), act="relu2"), O.relu_squared(ref + b.double()), dtype, "both", lim)


@each_form
@pytest.mark.parametrize("dim,vdim,hq,hkv", [(32, 24, 4, 2), (20, 40, 3, 3), (128, 128, 8, 2), (136, 264, 2, 1)])
def test_head_norm_value_mixing_and_cache_write(device, dtype, dim, vdim, hq, hkv):
    g = torch.Generator().manual_seed(dim)
    dt, rows, eps = TORCH[dtype], 9, 0.05
    dk, dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16

    def packed(heads, d, p):
        t = torch.zeros(rows, heads, p)
        t[..., :d] = torch.randn(rows, heads, d, generator=g)
        return t.reshape(rows, heads * p)
    row = torch.cat([packed(hq, dim, dk), packed(hkv, dim, dk), packed(hkv, vdim, dv), packed(hq, vdim, dv)], 1).to(dt)
    first = torch.cat([torch.zeros(rows, 16), packed(hkv, vdim, dv)], 1).to(dt).to(device)[:, 16:]
    slots = torch.tensor([5, 64, 127, 0, 191, -1, 70, 33, 1], dtype=torch.int32)
    kc, vc = (torch.zeros(3, hkv, 64, d, dtype=dt, device=device) for d in (dk, dv))
    qkv = row.clone().to(device)
    ops.head_norm_kv(qkv, slots.to(device), kc, vc, hq, hkv, dim, vdim, eps, first_v=first, mix=0.3)
    q = row[:, : hq * dk].double().view(rows, hq, dk)[..., :dim]
    k = row[:, hq * dk: (hq + hkv) * dk].double().view(rows, hkv, dk)[..., :dim]
    v = row[:, (hq + hkv) * dk: (hq + hkv) * dk + hkv * dv].double().view(rows, hkv, dv)[..., :vdim]
    v = O.mix_values(v, first.double().cpu().view(rows, hkv, dv)[..., :vdim], 0.3)
    lim = 1e-5 if dtype == "fp32" else 6e-3
    close(qkv[:, : hq * dk].view(rows, hq, dk)[..., :dim], O.rms(q, eps), dtype, "q", lim)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kc[s // 64, :, s % 64, :dim], O.rms(k, eps)[r], dtype, "k", lim)
            close(vc[s // 64, :, s % 64, :vdim], v[r], dtype, "v", lim)
    assert int((kc != 0).any(-1).sum()) == 8 * hkv and torch.equal(qkv.cpu()[:, hq * dk:], row[:, hq * dk:])


def _attention_reference(q, k, v, scale, chunk, gate):
    """q [n, H, dk] at the last n positions of k [G, ctx, dk]."""
    n, H, _ = q.shape
    G, ctx, _ = k.shape
    see = O.chunk_visible(ctx, chunk)[ctx - n:] if chunk else torch.tril(torch.ones(ctx, ctx, dtype=torch.bool))[ctx - n:]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[g].T) * scale
        out.append(torch.softmax(s.masked_fill(~see, float("-inf")), -1) @ v[g])
    return torch.cat(out, -1) * (torch.sigmoid(gate) if gate is not None else 1.0)


@each_form
@pytest.mark.parametrize("dk,dv,hq,hkv", [(128, 128, 8, 2), (64, 32, 6, 2), (16, 16, 2, 2), (80, 112, 6, 1), (144, 160, 2, 1)])
@pytest.mark.parametrize("chunk,gated", [(0, True), (64, False), (50, True), (300, True), (1000, True)])
def test_block_local_attention(device, dtype, dk, dv, hq, hkv, chunk, gated):
    """Prefill portions that start inside a block and decode rows on both sides of block and page edges; one key is made to
    stand out for one query so that leaving it out (or letting it in) shows."""
    dt = TORCH[dtype]
    scale = dk ** -0.5
    ctx, qlen = [300, 65, 128, 201, 51, 7], [300, 2, 70, 150, 1, 7]
    kc, vc, bt, ks, vs = paged(device, dt, hkv, dk, dv, ctx, seed=chunk + dk)
    g = torch.Generator().manual_seed(3)
    width = hq * dk + 16
    q = torch.randn(sum(qlen), width, generator=g)
    at = 0
    for b, (c, n) in enumerate(zip(ctx, qlen)):
        for pos, key in ((c - 1, (c - 1) // chunk * chunk if chunk else 0), (c - 1, (c - 1) // chunk * chunk - 1 if chunk else 0)):
            if key >= 0 and pos - (c - n) >= 0:      # the last query looks like the first key of its block, then like the one before it
                r = at + pos - (c - n)
                q[r, : hq * dk] += (ks[b][:, key].float() * 2.0).repeat_interleave(hq // hkv, 0).reshape(-1)
        at += n
    q = q.to(dt)
    gate = torch.randn(sum(qlen), hq * dv, generator=g).to(dt) if gated else None
    q0 = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    i32 = lambda t: torch.as_tensor(t, dtype=torch.int32).to(device)
    to = lambda t: None if t is None else t.to(device)
    args = (to(kc), to(vc), to(bt))
    got = ops.attn_prefill(to(q), *args, to(q0), i32(qlen), i32(ctx), max(qlen), hq, hkv, dk, scale, chunk=chunk, vdim=dv, gate=to(gate))
    lim = 2e-5 if dtype == "fp32" else 1.5e-2
    want, last = [], []
    for b, (c, n) in enumerate(zip(ctx, qlen)):
        r = slice(int(q0[b]), int(q0[b]) + n)
        qb = q[r, : hq * dk].double().view(n, hq, dk)
        want.append(_attention_reference(qb, ks[b], vs[b], scale, chunk, None if gate is None else gate[r].double()))
        last.append(int(q0[b]) + n - 1)
    want = torch.cat(want)
    close(got, want, dtype, "prefill", lim)
    for split in (max(ctx), 64):
        got = ops.attn_decode(to(q[last].contiguous()), *args, i32(ctx), hq, hkv, dk, scale, chunk=chunk, vdim=dv, max_ctx=split,
                              gate=None if gate is None else to(gate[last].contiguous()))
        close(got, want[last], dtype, f"decode {split}", lim)
    if device == "cuda":
        ops.check_status()


def test_block_mask_restatement():
    see = O.chunk_visible(7, 3)
    assert [torch.nonzero(r).flatten().tolist() for r in see] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


# ------------------------------------------------------------------------------------------
# the model: whole prompts, portions, decoding, batches
# ------------------------------------------------------------------------------------------
@each_form
def test_whole_prompt_and_layers(base, device, dtype):
    from flyingfish_b200.utils.trace import Trace
    path, w = base
    m = load(path, device, dtype)
    toks = ids(150)
    want, after = O.forward(CFG, w, toks)
    got, seq = feed_in_cuts(m.engine, toks, [150])
    close(got, want, dtype, "logits")
    m.engine.free_sequence(seq.seq_id)
    m.engine.model.trace = Trace(device=device)
    feed_in_cuts(m.engine, toks, [150])
    for i in range(len(LAYERS)):
        close(m.engine.model.trace.tensors[f"step.0.layer.{i}"], after[i], dtype, f"residual after layer {i}", 2e-5 if dtype == "fp32" else 3e-2)


@each_form
@pytest.mark.parametrize("cuts", [[1], [40, 1], [2], [5, 2, 3, 37, 64, 1], [64], [37], [50, 14, 1]])
def test_portions_and_decoding_equal_the_whole_prompt(base, device, dtype, cuts):
    """Token by token, portions down to two tokens, cuts on and beside page (64) and block (37, 50, 64) edges."""
    path, w = base
    m = load(path, device, dtype)
    toks = ids(140, seed=2)
    want, _ = O.forward(CFG, w, toks)
    got, _ = feed_in_cuts(m.engine, toks, cuts)
    close(got, want, dtype, str(cuts))
    if device == "cuda" and 1 in cuts:
        assert m.engine.stats["graph_replays"] > 0


@each_form
def test_mixed_batches_equal_each_request_alone(base, device, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, rows wanted here and there, in an
    order the engine has to sort."""
    path, w = base
    e = load(path, device, dtype).engine
    toks = {n: ids(k, seed=10 + i) for i, (n, k) in enumerate((("a", 130), ("b", 40), ("c", 70), ("d", 9)))}
    want = {n: O.forward(CFG, w, t)[0] for n, t in toks.items()}
    seqs, at, got = {}, dict.fromkeys(toks, 0), {n: {} for n in toks}
    steps = [[("b", 1), ("a", 60)], [("a", 1), ("b", 2), ("c", 33)], [("b", 1), ("c", 1), ("a", 1)], [("d", 9), ("c", 1), ("a", 31), ("b", 1)],
             [("a", 37), ("b", 30), ("c", 35)], [("b", 1)], [("b", 4)]]
    for step in steps:
        spans = []
        for n, k in step:
            part = toks[n][at[n]: at[n] + k]
            seqs[n] = seqs.get(n) or e.add_sequence(part)
            spans.append(Span(seqs[n], part, [j for j in range(k) if (at[n] + j) % 3 != 1]))
        out = e.feed(spans)
        r = 0
        for (n, k), sp in zip(step, spans):
            for j in sp.want:
                got[n][at[n] + j] = out[r].float().cpu()
                r += 1
            at[n] += k
        assert (0 if out is None else out.shape[0]) == r
    assert at == {n: len(t) for n, t in toks.items()}
    for n in toks:
        rows = sorted(got[n])
        close(torch.stack([got[n][i] for i in rows]), want[n][rows], dtype, n)
    # nothing wanted: nothing computed for the head, the tokens are committed all the same
    assert e.feed([Span(e.add_sequence([1, 2]), [1, 2])]) is None


@each_form
def test_blocks_are_reused_and_the_pool_is_tight(base, device, dtype):
    """Three blocks' worth of pool; requests come and go, the last over blocks in another order and full of old rows."""
    path, w = base
    e = load(path, device, dtype, capacity=192, kv_tokens=192).engine
    assert e.kv.num_blocks == 3
    for k in e.kv.k + e.kv.v:
        k.fill_(37.0)                                     # stale rows must not be seen
    a, sa = feed_in_cuts(e, ids(64, seed=20), [30, 34])
    b, sb = feed_in_cuts(e, ids(70, seed=21), [70])
    assert e.kv.alloc.free_blocks == 0
    e.free_sequence(sa.seq_id)
    c, sc = feed_in_cuts(e, ids(50, seed=22), [1, 20, 1])
    e.free_sequence(sb.seq_id)
    d, _ = feed_in_cuts(e, ids(128, seed=23), [7, 64, 50, 1])
    for n, (got, toks) in {"a": (a, ids(64, seed=20)), "b": (b, ids(70, seed=21)), "c": (c, ids(50, seed=22)), "d": (d, ids(128, seed=23))}.items():
        close(got, O.forward(CFG, w, toks)[0], dtype, n)


def needle_model(size, heads=2, kv_heads=1):
    """Two layers in which token 7 is the key every query looks for: the queries are one constant direction, token 7's key
    points there and no other's does; its value is large."""
    dim, width = 32, 48
    cfg = O.config([O.layer(size=size, dim=dim, vdim=24, heads=heads, kv_heads=kv_heads, scale=0.6) for _ in range(2)], width=width, vocab=64, streams=2)
    w = O.tensors(cfg, seed=4)
    w["embed"][:, 0] = 0.0
    w["embed"][7, 0] = 12.0
    for i in range(2):
        p = f"l{i}.mix."
        w[p + "q"] = w[p + "q"] * 0.02
        w[p + "q.b"] = torch.zeros_like(w[p + "q.b"])
        w[p + "q.b"].view(heads, dim)[:, 0] = 5.0
        w[p + "k.b"] = w[p + "k.b"] * 0.0
        w[p + "k"].view(kv_heads, dim, width)[:, 0] = 0.0
        w[p + "k"].view(kv_heads, dim, width)[:, 0, 0] = 40.0
        w[p + "v"] = w[p + "v"] * 3.0
        w[p + "o"][0], w[p + "o.b"][0], w[f"l{i}.mlp.down"][0] = 0.0, 0.0, 0.0        # channel 0 stays the token's own
        for q in (1, 2):
            w[f"l{i}.norm{q}"] = torch.ones_like(w[f"l{i}.norm{q}"])
    return cfg, w


@each_form
@pytest.mark.parametrize("size", [48, 64, 100])
def test_far_keys_and_block_edges(tmp_path, device, dtype, size):
    """A key that takes nearly all the weight of its block: at the block's first and last position, at page edges, far
    away; queries just inside and just outside the block, in a prompt and decoded."""
    cfg, w = needle_model(size)
    path = write(tmp_path, cfg, w)
    plain = [t if t != 7 else 8 for t in ids(2 * size + 20, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    e = load(path, device, dtype).engine
    for at in sorted({0, 1, size - 1, size, 2 * size - 1, 63, 64}):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved = ((want - without) ** 2).mean(-1).sqrt() / (without ** 2).mean(-1).sqrt()
        end = (at // size + 1) * size
        assert moved[at: end].min() > 0.2 and (moved[end:] == 0).all() and (moved[:at] == 0).all()
        for cuts in ([len(toks)], [max(end - 3, 1), 1]):          # the block's end in the prompt, and decoded
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            close(got, want, dtype, f"needle at {at}, cuts {cuts}", None if dtype == "fp32" else 8e-2)
            # rows of later blocks do not know the needle at all
            other, seq = feed_in_cuts(e, plain, cuts)
            e.free_sequence(seq.seq_id)
            assert torch.equal(other[end:], got[end:])


SIZES = {
    "one stream, factor one": O.config([O.layer(ff=40), O.layer(ff=None)], streams=1, residual_mult=1.0, scale=1.0),
    "tensor-core widths": O.config([O.layer(heads=4, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, size=96, ff=256)] * 2, width=256, vocab=512, streams=4),
    "odd sizes": O.config([O.layer(heads=3, kv_heads=3, dim=20, vdim=28, ff=51, size=29), O.layer(heads=9, kv_heads=3, dim=12, vdim=28, ff=33, size=7)], width=75, vocab=131, streams=5),
    "wide heads": O.config([O.layer(heads=2, kv_heads=1, dim=144, vdim=200, size=70, scale=0.1)] * 2, streams=2),
    "one head, a block per token": O.config([O.layer(heads=1, kv_heads=1, dim=16, vdim=16, size=1), O.layer(heads=1, kv_heads=1, dim=16, vdim=16, size=100000)], streams=3),
    "no mixing": O.config([O.layer(v_mix=False), O.layer(v_mix=False, heads=12, kv_heads=4)], streams=9),
    "one mixing layer": O.config([O.layer(v_mix=False), O.layer(v_mix=True)], eps=0.02),
    "large epsilon": O.config([O.layer()] * 3, eps=0.3),
}


@each_form
@pytest.mark.parametrize("name", sorted(SIZES))
def test_other_sizes(tmp_path, device, dtype, name):
    cfg = SIZES[name]
    w = O.tensors(cfg, seed=5)
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    toks = ids(135, vocab=cfg["vocab"], seed=8)
    want, _ = O.forward(cfg, w, toks)
    for cuts in ([135], [70, 1, 1, 2, 50, 1]):
        got, seq = feed_in_cuts(e, toks, cuts)
        e.free_sequence(seq.seq_id)
        close(got, want, dtype, f"{name} {cuts}")


@each_form
def test_a_batch_larger_than_a_forward(base, device, dtype):
    path, w = base
    e = load(path, device, dtype, chunk=64).engine
    a, b = ids(150, seed=30), ids(90, seed=31)
    sa, sb = e.add_sequence(a), e.add_sequence(b)
    wa, wb = [149, 3, 64, 63], [0, 89, 50]
    got = e.feed([Span(sa, a, wa), Span(sb, b, wb)])
    want = torch.cat([O.forward(CFG, w, a)[0][wa], O.forward(CFG, w, b)[0][wb]])
    assert e.max_prefill_rows == 64
    close(got, want, dtype, "split batch")


# ------------------------------------------------------------------------------------------
# generation through the framework's entry points
# ------------------------------------------------------------------------------------------
def greedy_agrees(w, prompt, got, dtype, cfg=CFG):
    """Every generated token is the oracle's first choice, or within rounding of it."""
    lg, _ = O.forward(cfg, w, prompt + got)
    for j, t in enumerate(got):
        row = lg[len(prompt) - 1 + j]
        assert row.max() - row[t] <= (1e-4 if dtype == "fp32" else 0.12) * row.std(), f"token {j}"


@each_form
def test_generation(base, device, dtype):
    path, w = base
    m = load(path, device, dtype, capacity=512)
    prompts = [ids(n, seed=40 + n) for n in (100, 3, 65)]
    outs = m.generate_batch(prompts, 40)
    for p, o in zip(prompts, outs):
        assert len(o) == 40
        greedy_agrees(w, p, o, dtype)
    m.reset()
    one = generate_plain(m, prompts[1], 150, ignore_eos=True)        # long decoding over pages and blocks
    greedy_agrees(w, prompts[1], one.ids, dtype)


@each_form
def test_scheduler_batches_portions_with_decoding(base, device, dtype):
    path, w = base
    m = load(path, device, dtype, capacity=256, kv_tokens=640)
    sch = Scheduler(m.engine, token_budget=40)
    lens = (150, 20, 90, 5, 61, 33)
    reqs = [sch.submit(Request(prompt=ids(n, seed=50 + n), max_tokens=30, ignore_eos=True)) for n in lens]
    sch.run_until_idle()
    assert m.engine.stats["mixed_steps"] > 3 and all(r.state == "finished" and len(r.output) == 30 for r in reqs)
    for r in reqs:
        greedy_agrees(w, r.prompt, r.output, dtype)
    assert m.engine.kv.alloc.free_blocks == m.engine.kv.num_blocks


@each_form
def test_preempted_requests_are_recomputed(base, device, dtype):
    path, w = base
    m = load(path, device, dtype, capacity=192, kv_tokens=320)
    sch = Scheduler(m.engine, token_budget=64)
    reqs = [sch.submit(Request(prompt=ids(60, seed=60 + n), max_tokens=12, ignore_eos=True)) for n in range(4)]
    sch.run_until_idle(max_iters=200)
    assert sch.stats["preempted"] > 0 and all(len(r.output) == 12 for r in reqs)
    for r in reqs:
        greedy_agrees(w, r.prompt, r.output, dtype)


def test_prefix_cache_restores_unequal_layers(base, tmp_path):
    path, w = base
    m = load(path, "cpu", "fp32", prefix_cache=True, runtime_dir=str(tmp_path))
    p = ids(90, seed=70)
    m.prefill(p[:70])
    assert m.prefill(p) == int(O.forward(CFG, w, p)[0][-1].argmax()) and m.prefix_store().hits == 1


@each_form
def test_verification_rows_and_draft_chain(base, device, dtype):
    """Several rows per sequence in one decode-style step, across page and block edges; drafts of another model accepted or
    refused give the tokens of plain decoding."""
    from flyingfish_b200.spec.chain import ChainSpeculator
    path, w = base
    m = load(path, device, dtype)
    for n in (48, 62, 99, 73):
        toks = ids(n + 4, seed=100 + n)
        s = m.engine.add_sequence(toks[:n])
        m.engine.prefill([s])
        s.pending = toks[n]
        got = m.engine.verify([s], [toks[n + 1:]])[0]
        lg = O.forward(CFG, w, toks)[0][n:]
        assert all(row.max() - row[t] <= (1e-4 if dtype == "fp32" else 0.12) * row.std() for row, t in zip(lg, got)), n
        m.engine.free_sequence(s.seq_id)
    out = ChainSpeculator(m, load(path, device, dtype), k=3).generate(ids(40, seed=7), 30, ignore_eos=True)
    greedy_agrees(w, ids(40, seed=7), out.ids[:30], dtype)


# ------------------------------------------------------------------------------------------
# configuration, checkpoint, command line, runner
# ------------------------------------------------------------------------------------------
def test_configuration_is_read_and_checked(base):
    path, _ = base
    s = read_model_spec(path)
    assert (s.arch, s.layers, s.hidden, s.vocab) == ("duponex", 4, 104, 198)
    assert s.kv_geometry() == [(1, 32, 16), (2, 32, 32), (2, 48, 32), (2, 32, 32)]
    assert [l.chunk for l in s.layer_specs] == [50, 50, 37, 64] and s.layer_specs[3].ffn == 0 and not s.layer_specs[0].v_mix
    n = 130
    l = s.layer_specs[2]
    assert l.pairs_seen(n) == int(O.chunk_visible(n, 37).sum()) and l.keys_seen(n) == int(O.chunk_visible(n, 37)[-1].sum())
    for change in ({"type": "recurrence"}, {"mlp": {"kind": "experts", "ff": 8}}, {"mixer": O.mixer(heads=3)}, {"mixer": O.mixer(scale=0.0)}):
        with pytest.raises(ConfigError):
            spec_from_hf_config(dict(CFG, layers=[dict(LAYERS[1], **change)]))
    with pytest.raises(ConfigError):
        spec_from_hf_config(dict(CFG, layers=[O.layer(), O.layer(vdim=16)]))
    with pytest.raises(ConfigError):
        spec_from_hf_config(dict(CFG, streams=17))


def test_checkpoint_is_audited(tmp_path):
    w = O.tensors(CFG)
    for i, (drop, put) in enumerate((("l1.mix.vmix", None), (None, ("l3.mlp.gate", torch.zeros(2, 2))), ("l0.hc1.in", ("l0.hc1.in", torch.zeros(4))))):
        t = {n: x for n, x in w.items() if n != drop}
        if put:
            t[put[0]] = put[1].to(torch.bfloat16)
        with pytest.raises(CheckpointError):
            load(write(tmp_path, CFG, t, f"m{i}"), "cpu", "bf16")
    # tensors of a part the configuration switches off may be there
    load(write(tmp_path, CFG, dict(w, **{"l0.mix.vmix": torch.tensor(0.5).to(torch.bfloat16), "l3.norm2": w["l3.norm1"].clone()}), "more"), "cpu", "bf16")


def test_planner_counts_unequal_layers():
    from flyingfish_b200.planner.plan import DeviceInfo, plan_memory
    s = named_shape("duponex-tiny")
    info = DeviceInfo(name="x", total_bytes=1 << 30, free_bytes=1 << 30)
    p = plan_memory(s, Settings(capacity=256, max_batch=2, kv_tokens=1000), info, 0)
    assert p.kv_blocks == 16 and p.kv_bytes == 16 * 64 * 2 * sum(h * (a + b) for h, a, b in s.kv_geometry())


def test_other_models_refuse_fed_batches_and_32_bit(base):
    m = Model.load("tiny-llama", Settings(capacity=128, max_batch=2), device="cpu")
    with pytest.raises(ValueError):
        m.engine.feed([Span(m.engine.add_sequence([1]), [1])])
    with pytest.raises(ValueError):
        load(base[0], "cpu", "bf16", kv_format="affine8")


def test_command_line_generates(base, capsys):
    from flyingfish_b200.cli import main
    path, w = base
    p = ids(12, seed=80)
    assert main(["--model", path, "--cpu", "--dtype", "fp32", "--kv-tokens", "256", "--capacity", "128", "generate", "--tokens",
                 ",".join(map(str, p)), "--max-new-tokens", "6", "--ignore-eos"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    greedy_agrees(w, p, out["generated_ids"], "fp32")
    assert main(["--model", path, "inspect"]) == 0
    assert json.loads(capsys.readouterr().out)["spec"]["arch"] == "duponex"


def _trace(vocab=198):
    a, b, c = ids(90, vocab, 90), ids(20, vocab, 91), ids(30, vocab, 92)
    return {"a": a, "b": b, "c": c}, [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [0, 59]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[1:20], "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "c", "tokens": c[:29], "want": [28]}, {"id": "a", "tokens": a[60:61], "want": [0]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[61:62], "want": [0]}, {"id": "c", "tokens": c[29:], "want": [0]}], "end": ["c"]},
        {"step": 4, "entries": [{"id": "a", "tokens": a[62:90], "want": [27, 0]}], "end": ["a"]}]


def _trace_wants(w, toks):
    lg = {n: O.forward(CFG, w, t)[0] for n, t in toks.items()}
    return {0: torch.stack([lg["a"][0], lg["a"][59], lg["b"][0]]), 2: torch.stack([lg["c"][28], lg["a"][60]]),
            3: torch.stack([lg["a"][61], lg["c"][29]]), 4: torch.stack([lg["a"][89], lg["a"][62]])}


@each_form
def test_trace_runner_steps(base, device, dtype):
    from flyingfish_b200.serve.trace_runner import TraceError, TraceRunner, load_engine
    path, w = base
    m, e = load_engine(path, dtype, 192, device)
    assert e.kv.num_blocks == 3
    r = TraceRunner(e, m.spec.vocab)
    toks, steps = _trace()
    want = _trace_wants(w, toks)
    for s in steps:
        out = r.step(s["entries"], s["end"])
        if s["step"] in want:
            close(out, want[s["step"]], dtype, f"step {s['step']}")
        else:
            assert out is None
    assert not r.live and e.kv.alloc.free_blocks == 3
    for entries, end in (([{"id": "x", "tokens": [198], "want": []}], []), ([{"id": "x", "tokens": [1], "want": [1]}], []), ([], ["x"])):
        with pytest.raises(TraceError):
            r.step(entries, end)


@GPU
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(base, tmp_path, dtype):
    import numpy as np
    path, w = base
    toks, steps = _trace()
    exe = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    p = subprocess.run([sys.executable, str(exe), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "192"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=500)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    for i, want in _trace_wants(w, toks).items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").copy()).view(want.shape)
        close(got, want, "bf16" if dtype == "bfloat16" else "fp32", f"step {i}")
    assert not (tmp_path / "1.f32").exists()


def test_random_shape_generates():
    m = Model.load("duponex-tiny", Settings(capacity=128, max_batch=2), device="cpu", seed=3)
    out = m.generate_batch([[1, 2, 3], [4] * 50], 5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 512 for o in out for t in o)


@GPU
def test_random_shape_gpu_matches_cpu():
    from _oracle import assert_tokens_equal_up_to_ties
    st = Settings(capacity=256, max_batch=2)
    cpu, gpu = (Model.load("duponex-tiny", st, device=d, seed=3) for d in ("cpu", "cuda"))
    prompts = [ids(80, 512, 1), ids(9, 512, 2)]
    for p, a, b in zip(prompts, cpu.generate_batch(prompts, 12), gpu.generate_batch(prompts, 12)):
        assert_tokens_equal_up_to_ties(cpu, p, a, b)
    ops.check_status()
