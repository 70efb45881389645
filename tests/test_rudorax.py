"""Rudorax decoder against the plain restatement in ``rudorax_oracle``: every mechanism alone, whole prompts, portions, mixed
batches, decoding, window edges, far keys, states and blocks that are used again, sizes that need padding, and generation through
the scheduler. Every case runs on the CPU oracles of the operators and, on a GPU, through the kernels in BF16 and FP32."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import rudorax_oracle as O
from _design import GPU, TORCH, close, each_form, feed_in_cuts, ids, load, paged, write
from flyingfish_b200 import ops
from flyingfish_b200.api import Model, generate_plain
from flyingfish_b200.config import ConfigError, RopeSpec, Settings, named_shape, read_model_spec, spec_from_hf_config
from flyingfish_b200.engine.engine import Span
from flyingfish_b200.engine.scheduler import Request, Scheduler
from flyingfish_b200.loaders.checkpoint import CheckpointError
from flyingfish_b200.ops import mlstm_ops, moe_ops, ref, residual_ops

# a memory's outputs are divided by their root mean square: where its first keys and queries nearly cancel, rounding is magnified
MODEL_LIMIT = {"fp32": 2e-4, "bf16": 0.1}


def agree(got, want, dtype, what):
    close(got, want, dtype, what, MODEL_LIMIT[dtype])


# unequal layers, a layer of each kind without a feed-forward, two layers run twice
LAYERS = [O.attn_layer(kv_heads=1, vdim=16), O.mlstm_layer(), O.attn_layer(size=37, dim=48, heads=6, kv_heads=2, scale=0.25, turn=O.rot(dims=40, base=900.0)),
          O.mlstm_layer(heads=2, dim=40, vdim=72, gate_cap=4.0, mlp=None), O.attn_layer(size=64, mlp=None)]
CFG = O.config(LAYERS, loop=(1, 3, 2))


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    w = O.tensors(CFG)
    return write(tmp_path_factory.mktemp("rudorax"), CFG, w), w


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@each_form
@pytest.mark.parametrize("width,true_width,two", [(64, 64, True), (104, 100, True), (1024, 1024, False), (40, 37, True)])
def test_residual_embed_and_step(device, dtype, width, true_width, two):
    g = torch.Generator().manual_seed(width)
    dt, rows, eps, t = TORCH[dtype], 7, 1e-3, slice(0, true_width)
    mask = (torch.arange(width) < true_width).float()
    rn = lambda *s: torch.randn(*s, generator=g) * mask
    dev = lambda x: None if x is None else x.to(device)
    table, w1, w2 = rn(30, width).to(dt), 1 + rn(width), 1 + rn(width) if two else None
    tok = torch.randint(0, 30, (rows,), generator=g).to(torch.int32)
    lim = 1e-5 if dtype == "fp32" else 8e-3
    x, n1, n2 = residual_ops.embed(dev(tok), dev(table), 1.7, dev(w1), dev(w2), eps, true_width)
    want = table.double()[tok.long()] * 1.7
    close(x, want, dtype, "stream", 1e-6)
    a, b = rn(rows, width).to(dt), rn(rows, width).to(dt)
    # three experts of which a row chose two, or one and an identity output; one choice was not served
    y, h = rn(20, width).to(dt), rn(rows, width).to(dt)
    eids = torch.tensor([[0, 1], [2, 3], [1, 2], [4, 0], [2, 1], [0, 3], [1, 0]], dtype=torch.int32)
    pos = torch.tensor([3, 7, 0, -1, 19, 4, -1, 5, 6, 8, -1, -1, 9, 10], dtype=torch.int32)
    ew = torch.rand(rows, 2, generator=g)
    for k in range(2):
        for r in range(rows):
            if eids[r, k] < 3 and pos[2 * r + k] < 0:
                ew[r, k] = 0.0 if device == "cpu" else ew[r, k]
    for extra in (False, True):
        rows_of = moe_ops.ExpertRows(dev(y), dev(pos), dev(eids), dev(ew), dev(h), 3) if extra else None
        want = want + a.double()
        if extra:
            want = want + b.double()
            for r in range(rows):
                for k in range(2):
                    p = int(pos[2 * r + k])
                    if eids[r, k] >= 3 or p >= 0:
                        want[r] += ew[r, k].double() * (h[r] if eids[r, k] >= 3 else y[p]).double()
        n1, n2 = residual_ops.step(x, dev(a), dev(b) if extra else None, rows_of, dev(w1), dev(w2), eps, true_width)
        close(x, want, dtype, "sum", 1e-5)
        close(n1[:, t], O.rms(want[:, t], eps) * w1.double()[t], dtype, "first norm", lim)
        assert (n2 is None) == (not two)
        if two:
            close(n2[:, t], O.rms(want[:, t], eps) * w2.double()[t], dtype, "second norm", lim)


def test_scaled_rotation_frequencies():
    for turn in (O.rot(), O.rot(dims=64, base=1e6, factor=8.0, original=4096, fast=32.0, slow=1.0), O.rot(dims=2, factor=1.5),
                 O.rot(dims=10, original=8), dict(O.rot(), scaling=None)):
        s = turn["scaling"] or {}
        freqs, amp = RopeSpec(base=turn["base"], dims=turn["dims"], **s).frequencies()
        want, wamp = O.yarn_frequencies(turn)
        assert torch.allclose(torch.tensor(freqs, dtype=torch.float64), want, rtol=1e-12) and amp == wamp
    plain, _ = O.yarn_frequencies(dict(O.rot(), scaling=None))
    scaled, _ = O.yarn_frequencies(O.rot())
    assert not torch.allclose(plain, scaled) and float(scaled[0]) == 1.0


@each_form
@pytest.mark.parametrize("dim,vdim,hq,hkv,dims", [(32, 24, 4, 2, 16), (20, 40, 3, 3, 20), (128, 128, 8, 2, 128), (136, 264, 2, 1, 6)])
def test_head_norm_rotation_and_cache_write(device, dtype, dim, vdim, hq, hkv, dims):
    g = torch.Generator().manual_seed(dim)
    dt, rows, eps, first = TORCH[dtype], 9, 0.05, 4990
    dk, dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16

    def packed(heads, d, p):
        t = torch.zeros(rows, heads, p)
        t[..., :d] = torch.randn(rows, heads, d, generator=g)
        return t.reshape(rows, heads * p)
    row = torch.cat([packed(hq, dim, dk), packed(hkv, dim, dk), packed(hkv, vdim, dv)], 1).to(dt)
    wq, wk = 1 + 0.4 * torch.randn(dim, generator=g), 1 + 0.4 * torch.randn(dim, generator=g)
    pad = lambda w: torch.cat([w, torch.zeros(dk - dim)]).to(device)
    slots = torch.tensor([5, 64, 127, 0, 191, -1, 70, 33, 1], dtype=torch.int32)
    kc, vc = (torch.zeros(3, hkv, 64, d, dtype=dt, device=device) for d in (dk, dv))
    turn = O.rot(dims=dims, base=300.0)
    freqs, amp = RopeSpec(base=300.0, dims=dims, **turn["scaling"]).frequencies()
    positions = torch.arange(first, first + rows, dtype=torch.int32, device=device)
    table = ops.rope_angles(positions, ops.rope_frequencies(freqs, device), amp)
    qkv = row.clone().to(device)
    ops.head_norm_kv(qkv, slots.to(device), kc, vc, hq, hkv, dim, vdim, eps, q_weight=pad(wq), k_weight=pad(wk), cos_sin=table)
    heads = lambda lo, n, d, p: row[:, lo: lo + n * p].double().view(rows, n, p)[..., :d]
    q = O.rotate_pairs(O.rms(heads(0, hq, dim, dk), eps) * wq.double(), turn, first)
    k = O.rotate_pairs(O.rms(heads(hq * dk, hkv, dim, dk), eps) * wk.double(), turn, first)
    v = heads((hq + hkv) * dk, hkv, vdim, dv)
    lim = 2e-6 if dtype == "fp32" else 6e-3
    close(qkv[:, : hq * dk].view(rows, hq, dk)[..., :dim], q, dtype, "q", lim)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kc[s // 64, :, s % 64, :dim], k[r], dtype, "k", lim)
            close(vc[s // 64, :, s % 64, :vdim], v[r], dtype, "v", lim)
    assert int((kc != 0).any(-1).sum()) == 8 * hkv


def _attention_reference(q, k, v, scale, size, sink):
    """q [n, H, dk] at the last n positions of k [G, ctx, dk]."""
    n, H, _ = q.shape
    G, ctx, _ = k.shape
    see = O.window_visible(ctx, size)[ctx - n:]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[h // (H // G)].T) * scale
        out.append(O.softmax_with_sink(s.masked_fill(~see, float("-inf")), sink[h]) @ v[h // (H // G)])
    return torch.cat(out, -1)


@each_form
@pytest.mark.parametrize("dk,dv,hq,hkv", [(128, 128, 8, 2), (64, 32, 6, 2), (16, 16, 2, 2), (80, 112, 20, 1), (144, 160, 2, 1)])
@pytest.mark.parametrize("size", [1, 50, 64, 65, 1000])
def test_windowed_attention_with_sinks(device, dtype, dk, dv, hq, hkv, size):
    """Prefill portions and decode rows; the last query of a sequence looks like the first key of its window in one case and like
    the key before it in the other, so that leaving the one out or letting the other in shows. One sink takes most of the weight."""
    dt, scale = TORCH[dtype], dk ** -0.5
    ctx, qlen = [300, 65, 128, 201, 51, 7, 1], [300, 2, 70, 150, 1, 7, 1]
    kc, vc, bt, ks, vs = paged(device, dt, hkv, dk, dv, ctx, seed=size + dk)
    g = torch.Generator().manual_seed(3)
    q0 = torch.randn(sum(qlen), hq * dk + 16, generator=g)
    sink = torch.randn(hq, generator=g)
    sink[0] = 4.0
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    i32 = lambda t: torch.as_tensor(t, dtype=torch.int32).to(device)
    args = tuple(t.to(device) for t in (kc, vc, bt))
    lim = 2e-5 if dtype == "fp32" else 1.5e-2
    for back in (0, 1):
        q = q0.clone()
        for b, c in enumerate(ctx):
            key = c - size - back
            if key >= 0:
                r = int(starts[b]) + qlen[b] - 1
                q[r, : hq * dk] += (ks[b][:, key].float() * 2.0).repeat_interleave(hq // hkv, 0).reshape(-1)
        q = q.to(dt)
        want, last = [], []
        for b, n in enumerate(qlen):
            r = slice(int(starts[b]), int(starts[b]) + n)
            want.append(_attention_reference(q[r, : hq * dk].double().view(n, hq, dk), ks[b], vs[b], scale, size, sink.double()))
            last.append(int(starts[b]) + n - 1)
        want = torch.cat(want)
        kw = dict(window=size, sinks=sink.to(device), vdim=dv)
        got = ops.attn_prefill(q.to(device), *args, starts.to(device), i32(qlen), i32(ctx), max(qlen), hq, hkv, dk, scale, **kw)
        close(got, want, dtype, "prefill", lim)
        for split in (max(ctx), 64):
            got = ops.attn_decode(q[last].contiguous().to(device), *args, i32(ctx), hq, hkv, dk, scale, max_ctx=split, **kw)
            close(got, want[last], dtype, f"decode {split}", lim)
    if device == "cuda":
        ops.check_status()


def test_window_mask_restatement():
    assert [torch.nonzero(r).flatten().tolist() for r in O.window_visible(5, 3)] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4]]


@each_form
@pytest.mark.parametrize("dim,vdim,heads,cap", [(24, 40, 3, 7.0), (64, 64, 2, 15.0), (128, 200, 2, 3.0), (16, 16, 1, 1.0), (144, 72, 1, 30.0), (272, 24, 1, 8.0)])
def test_matrix_memory(device, dtype, monkeypatch, dim, vdim, heads, cap):
    """Several sequences at once in slots out of order, their rows cut into calls of very different lengths (one token, two, a
    chunk and its neighbours, segments of a long portion); gates at both ends of their caps; stale slots reset."""
    monkeypatch.setattr(mlstm_ops, "SEGMENT_ROWS", 128)
    monkeypatch.setattr(mlstm_ops, "FILL_CTAS", 1 << 30)
    g = torch.Generator().manual_seed(dim)
    dt = TORCH[dtype]
    dk, dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    lens = [390, 131]
    cuts = [(1, 64), (63, 2), (2, 65), (324, 0)]

    def packed(n, d, p):
        t = torch.zeros(n, heads, p)
        t[..., :d] = torch.randn(n, heads, d, generator=g)
        return t.reshape(n, heads * p)
    seqs = []
    for n in lens:
        x = torch.cat([packed(n, dim, dk), packed(n, dim, dk), packed(n, vdim, dv), packed(n, vdim, dv)], 1).to(dt)
        z = torch.randn(n, 2 * heads, generator=g) * 3.0
        z[:, heads:] += 4.0
        z[5], z[70, :heads], z[100, heads:] = 100.0, 60.0, -100.0       # everything at its cap; a token that counts; a forgetting one
        seqs.append((x, z))
    bias = torch.randn(2 * heads, generator=g)
    want = []
    for x, z in seqs:
        part = lambda lo, d, p: x[:, lo: lo + heads * p].double().view(-1, heads, p)[..., :d]
        zi, zf = (O.capped(t, cap) for t in (z + bias).double().split(heads, 1))
        want.append(O.matrix_memory(part(0, dim, dk) * dim ** -0.5, part(heads * dk, dim, dk), part(2 * heads * dk, vdim, dv), zi,
                                    torch.nn.functional.logsigmoid(zf)))
    st = mlstm_ops.MemoryState(5, heads, dk, dv, device)
    for t in (st.S, st.n, st.m):
        t.fill_(3.0)
    slots = [3, 1]
    for s in slots:
        st.reset(s)
    at = [0, 0]
    lim = 3e-3                                    # the outputs before their norm: a denominator near zero magnifies rounding
    for cut in cuts:
        live = [i for i in (0, 1) if cut[i]]
        x = torch.cat([seqs[i][0][at[i]: at[i] + cut[i]] for i in live]).to(device)
        z = torch.cat([seqs[i][1][at[i]: at[i] + cut[i]] for i in live]).to(device)
        start = torch.tensor([0] + [cut[i] for i in live]).cumsum(0).to(torch.int32).to(device)
        out = torch.full((x.shape[0], heads, dv), 9.0, device=device)
        mlstm_ops.memory(x, z, bias.to(device), cap, st, start, torch.tensor([slots[i] for i in live], dtype=torch.int32, device=device),
                         dim ** -0.5, out, max(cut))
        w = torch.cat([want[i][at[i]: at[i] + cut[i]] for i in live])
        close(out[..., :vdim].reshape(-1, vdim), w.reshape(-1, vdim), dtype, f"portion {cut} at {at}", lim)
        got = out[..., :vdim].double().cpu()
        assert ((got - w).norm(dim=-1) / w.norm(dim=-1)).median() < 1e-5
        assert (out[..., vdim:] == 0).all()
        at = [a + c for a, c in zip(at, cut)]
    assert at == lens and (st.S[[0, 2, 4]] == 3.0).all() and (st.m[[0, 2, 4]] == 3.0).all()
    gate = seqs[1][0][-2:, heads * (2 * dk + dv):]
    o = torch.zeros(2, heads, dv)
    o[..., :vdim] = want[1][-2:].float()
    wn = torch.zeros(heads, dv)
    wn[:, :vdim] = 1 + 0.3 * torch.randn(heads, vdim, generator=g)
    y = mlstm_ops.head_out(o.to(device), gate.to(device), wn.reshape(-1).to(device), vdim, 0.01)
    ref_y = O.rms(o[..., :vdim].double(), 0.01) * wn[:, :vdim].double() * torch.sigmoid(gate.double().view(2, heads, dv)[..., :vdim])
    close(y.view(2, heads, dv)[..., :vdim].reshape(-1, vdim), ref_y.reshape(-1, vdim), dtype, "out", 1e-5 if dtype == "fp32" else 8e-3)


@each_form
@pytest.mark.parametrize("m", [1, 5, 130])
@pytest.mark.parametrize("n,k", [(16, 104), (200, 72), (264, 512)])
def test_linear_with_32_bit_result(device, dtype, m, n, k):
    g = torch.Generator().manual_seed(m)
    x, w = (torch.randn(*s, generator=g).to(TORCH[dtype]) for s in ((m, k), (n, k)))
    y = ops.linear(x.to(device), w.to(device), out_dtype=torch.float32)
    assert y.dtype == torch.float32
    close(y, x.double() @ w.double().T, dtype, "logits", 1e-5)
    z = y.clone()
    close(ops.softcap(z, 5.0), O.capped(y.double(), 5.0), dtype, "cap", 1e-5)


@each_form
@pytest.mark.parametrize("experts,identity,top,ff,width,rows", [(6, 2, 3, 40, 104, 37), (5, 0, 1, 64, 64, 3), (9, 3, 12, 72, 40, 20), (4, 4, 2, 128, 256, 600), (70, 30, 6, 24, 64, 64)])
def test_experts(device, dtype, experts, identity, top, ff, width, rows):
    """Choice with the bias, weights without it; identity outputs; experts nobody chose, and every output chosen."""
    g = torch.Generator().manual_seed(experts)
    dt = TORCH[dtype]
    n = experts + identity
    lin = lambda o, i: (torch.randn(o, i, generator=g) / i ** 0.5).to(dt)
    t = {"router": 2 * lin(n, width), "correction": 0.2 * torch.randn(n, generator=g)}
    for e in range(experts):
        t.update({f"e{e}.gate": lin(ff, width), f"e{e}.up": lin(ff, width), f"e{e}.down": lin(width, ff)})
    x = torch.randn(rows, width, generator=g).to(dt)
    get = lambda name: t[name].double()
    fp = (ff + 63) // 64 * 64
    grow = lambda w, r: torch.cat([w, w.new_zeros(r - w.shape[0], w.shape[1])])
    gu = torch.stack([ref.interleave_gate_up(grow(t[f"e{e}.gate"], fp), grow(t[f"e{e}.up"], fp)) for e in range(experts)])
    down = torch.stack([grow(t[f"e{e}.down"].T, fp).T for e in range(experts)]).contiguous()
    pad = grow(t["router"], (n + 15) // 16 * 16)
    dev = lambda v: v.to(device)
    w, chosen = moe_ops.route(dev(x), dev(pad), top, "softmax", dev(t["correction"]), exact=True, experts=n)
    want_ids, want_w = O.choose_experts(x.double(), get, "", top)
    assert torch.equal(chosen.cpu().long(), want_ids)
    close(w, want_w, dtype, "weights", 1e-5)
    assert (want_ids != O.choose_experts(x.double(), lambda k: get(k) * (k != "correction"), "", top)[0]).any() or top == n
    cfg = {"router": {"experts": experts, "identity": identity, "top": top}}
    want = O.mixture(x.double(), get, "", cfg)
    for er in (moe_ops.expert_rows(dev(x), w, chosen, dev(gu), dev(down)),
               moe_ops.routed_rows(dev(x), dev(pad), top, "softmax", dev(t["correction"]), n, dev(gu), dev(down))):
        assert torch.equal(er.ids.cpu().long(), want_ids)
        s = torch.zeros(rows, width, device=device)
        residual_ops.step(s, dev(torch.zeros_like(x)), None, er, torch.ones(width, device=device), None, 1e-5, width)
        close(s, want, dtype, "sum", 1e-5 if dtype == "fp32" else 2e-2)


# ------------------------------------------------------------------------------------------
# the model: whole prompts, portions, decoding, batches
# ------------------------------------------------------------------------------------------
@each_form
def test_whole_prompt_and_layer_runs(base, device, dtype):
    from flyingfish_b200.utils.trace import Trace
    path, w = base
    m = load(path, device, dtype)
    toks = ids(150)
    want, after = O.forward(CFG, w, toks)
    got, seq = feed_in_cuts(m.engine, toks, [150])
    agree(got, want, dtype, "logits")
    m.engine.free_sequence(seq.seq_id)
    m.engine.model.trace = Trace(device=device)
    feed_in_cuts(m.engine, toks, [150])
    assert after.shape[0] == len(m.engine.model.runs) == 7
    for i in range(after.shape[0]):
        agree(m.engine.model.trace.tensors[f"step.0.run.{i}"], after[i], dtype, f"residual after run {i}")


@each_form
@pytest.mark.parametrize("cuts", [[1], [40, 1], [2], [5, 2, 3, 37, 64, 1], [64], [37], [50, 14, 1]])
def test_portions_and_decoding_equal_the_whole_prompt(base, device, dtype, cuts):
    """Token by token, portions down to two tokens, cuts on and beside page, chunk (64) and window (37, 50, 64) edges."""
    path, w = base
    m = load(path, device, dtype)
    toks = ids(140, seed=2)
    want, _ = O.forward(CFG, w, toks)
    got, _ = feed_in_cuts(m.engine, toks, cuts)
    agree(got, want, dtype, str(cuts))
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
        agree(torch.stack([got[n][i] for i in rows]), want[n][rows], dtype, n)


@each_form
def test_blocks_and_states_are_used_again(base, device, dtype):
    """Three blocks and two state slots; requests come and go, the last over blocks and slots full of old rows."""
    path, w = base
    e = load(path, device, dtype, capacity=192, kv_tokens=192, max_batch=2).engine
    assert e.kv.num_blocks == 3 and len(e.state_slots) == 2
    for k in e.kv.k + e.kv.v:
        if k is not None:
            k.fill_(37.0)                                 # stale rows must not be seen
    for st in e.model.states.values():
        for t in (st.S, st.n, st.m):
            t.fill_(5.0)
    a, sa = feed_in_cuts(e, ids(64, seed=20), [30, 34])
    b, sb = feed_in_cuts(e, ids(70, seed=21), [70])
    assert e.kv.alloc.free_blocks == 0 and not e.state_slots
    with pytest.raises(ValueError):
        e.add_sequence([1])
    e.free_sequence(sa.seq_id)
    c, sc = feed_in_cuts(e, ids(50, seed=22), [1, 20, 1])
    e.free_sequence(sb.seq_id)
    d, _ = feed_in_cuts(e, ids(128, seed=23), [7, 64, 50, 1])
    for n, (got, toks) in {"a": (a, ids(64, seed=20)), "b": (b, ids(70, seed=21)), "c": (c, ids(50, seed=22)), "d": (d, ids(128, seed=23))}.items():
        agree(got, O.forward(CFG, w, toks)[0], dtype, n)


def needle_attention(size):
    """One attention layer in which token 7 is the key every query looks for. Channel 0 of every token is the direction of the
    queries, channel 1 of token 7 alone that of its key, both on an element that does not turn."""
    dim, width = 32, 48
    cfg = O.config([O.attn_layer(size=size, dim=dim, vdim=24, heads=2, kv_heads=1, scale=0.5, turn=O.rot(dims=4), mlp=None)], width=width, vocab=64, scale=1.0)
    w = O.tensors(cfg, seed=4)
    w["embed"][:, 0], w["embed"][:, 1] = 3.0, 0.0
    w["embed"][7, 1] = 9.0
    for name, heads, channel in (("q", 2, 0), ("k", 1, 1)):
        m = w["l0.mix." + name].view(heads, dim, width)
        m *= 0.3
        m[:, 31] = 0.0
        m[:, 31, channel] = 3.0
        w[f"l0.mix.{name}.norm"] = torch.ones_like(w[f"l0.mix.{name}.norm"])
    w["l0.mix.v"] = w["l0.mix.v"] * 4.0
    return cfg, w


def needle_memory():
    """One memory layer that takes in token 7 and next to nothing of the others, and forgets slowly. Channel 0 of every token puts
    queries and keys on one side, so that what is read does not hang on a cancellation."""
    cfg = O.config([O.mlstm_layer(heads=2, dim=24, vdim=32, gate_cap=9.0, mlp=None)], width=48, vocab=64, scale=1.0)
    w = O.tensors(cfg, seed=6)
    w["embed"][:, 0], w["embed"][:, 1] = 3.0, 0.0
    w["embed"][7, 1] = 9.0
    for name in ("q", "k"):
        w["l0.mix." + name].view(2, 24, 48)[:, 23, 0] = 5.0
    w["l0.mix.i"] = w["l0.mix.i"] * 0.0
    w["l0.mix.i"][:, 1] = 3.0
    w["l0.mix.i.b"] = w["l0.mix.i.b"] * 0.0 - 4.0
    w["l0.mix.f"] = w["l0.mix.f"] * 0.1
    w["l0.mix.f.b"] = w["l0.mix.f.b"] * 0.0 + 7.0
    return cfg, w


def relative_change(a, b):
    return ((a - b) ** 2).mean(-1).sqrt() / (b ** 2).mean(-1).sqrt()


@each_form
@pytest.mark.parametrize("size", [1, 2, 48, 64, 100])
def test_far_keys_and_window_edges(tmp_path, device, dtype, size):
    """A key that takes nearly all the weight while it is in the window: at the first positions, at page edges, far away;
    queries just inside and just outside the window, in a prompt and decoded."""
    cfg, w = needle_attention(size)
    path = write(tmp_path, cfg, w)
    n = 2 * size + 20 if size > 2 else 70
    plain = [t if t != 7 else 8 for t in ids(n, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    e = load(path, device, dtype).engine
    other = {}
    for at in sorted({0, 1, min(size, n - 1), 63, 64}):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved, end = relative_change(want, without), at + size
        assert moved[at: end].min() > 0.15 and (moved[end:] == 0).all() and (moved[:at] == 0).all()
        for cuts in ([n], [max(end - 3, 1), 1]):                  # the window's end in the prompt, and decoded
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")
            # rows that do not see the needle do not know of it at all
            if tuple(cuts) not in other:
                other[tuple(cuts)], seq = feed_in_cuts(e, plain, cuts)
                e.free_sequence(seq.seq_id)
            assert torch.equal(other[tuple(cuts)][end:], got[end:])


@each_form
def test_the_memory_keeps_a_far_token(tmp_path, device, dtype):
    cfg, w = needle_memory()
    e = load(write(tmp_path, cfg, w), device, dtype, capacity=512).engine
    n = 300
    plain = [t if t != 7 else 8 for t in ids(n, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    for at in (0, 1, 63, 64, 127):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved = relative_change(want, without)
        assert moved[at:].min() > 0.15 and (moved[:at] == 0).all()
        for cuts in ([n], [at + 1, 2, 64, 65, 1], [100, 100, 60, 1]):
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")


@each_form
def test_a_sink_that_matters(tmp_path, device, dtype):
    """Sinks that take most of the weight in one head and none in another."""
    cfg = O.config([O.attn_layer(heads=4, kv_heads=2, size=20)] * 2)
    w = O.tensors(cfg, seed=9)
    for i in range(2):
        w[f"l{i}.mix.sink"] = torch.tensor([6.0, -8.0, 3.0, 0.0]).to(torch.bfloat16)
    toks = ids(60, seed=9)
    want, _ = O.forward(cfg, w, toks)
    off, _ = O.forward(cfg, {n: (t * 0 - 60 if n.endswith("sink") else t) for n, t in w.items()}, toks)
    assert relative_change(off, want).min() > 0.1
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    for cuts in ([60], [3, 40, 1]):
        got, seq = feed_in_cuts(e, toks, cuts)
        e.free_sequence(seq.seq_id)
        agree(got, want, dtype, str(cuts))


A, M = O.attn_layer, O.mlstm_layer
SIZES = {
    "every constant one": O.config([A(heads=2, kv_heads=2, scale=1.0, size=9), M(heads=1, gate_cap=1.0)], scale=1.0, loop=(0, 2, 1)),
    "tensor-core widths": O.config([A(heads=4, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, size=96, turn=O.rot(dims=128), mlp=O.moe(ff=128, shared=256)),
                                    M(heads=2, dim=128, vdim=128, mlp=O.moe(ff=128, shared=256))], width=256, vocab=512),
    "odd sizes": O.config([A(heads=3, kv_heads=3, dim=20, vdim=28, size=29, turn=O.rot(dims=6)), M(heads=5, dim=12, vdim=28, mlp=O.moe(ff=33, shared=17)),
                           A(heads=9, kv_heads=3, dim=12, vdim=28, size=7, turn=O.rot(dims=12))], width=75, vocab=131, loop=(1, 3, 3)),
    "wide heads": O.config([A(heads=2, kv_heads=1, dim=144, vdim=200, size=70, scale=0.1), M(heads=1, dim=264, vdim=136)]),
    "one token windows": O.config([A(heads=1, kv_heads=1, dim=16, vdim=16, size=1), A(heads=1, kv_heads=1, dim=16, vdim=16, size=100000)]),
    "memories only": O.config([M(), M(mlp=None), M(heads=2, dim=64, vdim=64)], loop=(0, 3, 2)),
    "attention only, no loop": O.config([A(), A(heads=12, kv_heads=4)], softcap=2.0),
    "no cap on the logits": O.config([A(), M()], softcap=None),
    "one expert, no identity": O.config([A(mlp=O.moe(experts=1, identity=0, top=1)), M(mlp=O.moe(experts=3, identity=0, top=3))]),
    "identities alone or most": O.config([A(mlp=O.moe(experts=2, identity=9, top=5)), M(mlp=O.moe(experts=1, identity=40, top=2))]),
    "no shared expert": O.config([A(mlp=dict(O.moe(), shared=None)), M()]),
    "plain rotation": O.config([A(turn=dict(O.rot(dims=24, base=700.0), scaling=None)), A(turn=O.rot(dims=2, factor=40.0))], eps=0.2),
    "long loop": O.config([A(), M(), A(mlp=None)], loop=(0, 2, 5)),
}


@each_form
@pytest.mark.parametrize("name", sorted(SIZES))
def test_other_sizes(tmp_path, device, dtype, name):
    cfg = SIZES[name]
    w = O.tensors(cfg, seed=5)
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    toks = ids(135, vocab=cfg["vocab"], seed=8)
    O.MARGINS.clear()
    want, _ = O.forward(cfg, w, toks)
    assert not O.MARGINS or min(O.MARGINS) > 0.02                 # no choice that rounding could turn
    for cuts in ([135], [70, 1, 1, 2, 50, 1]):
        got, seq = feed_in_cuts(e, toks, cuts)
        e.free_sequence(seq.seq_id)
        agree(got, want, dtype, f"{name} {cuts}")


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
    agree(got, want, dtype, "split batch")


@GPU
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_prompt_in_segments(base, dtype):
    """A prompt long enough for the memory's segments, then decoded on."""
    path, w = base
    e = load(path, "cuda", dtype, capacity=1600).engine
    toks = ids(1300, seed=33)
    want, _ = O.forward(CFG, w, toks)
    got, _ = feed_in_cuts(e, toks, [1260, 30, 1])
    agree(got, want, dtype, "long")
    ops.check_status()


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
    one = generate_plain(m, prompts[1], 150, ignore_eos=True)        # long decoding over pages and windows
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
    assert m.engine.kv.alloc.free_blocks == m.engine.kv.num_blocks and len(m.engine.state_slots) == 4


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


def test_what_a_state_cannot_do_is_refused(base, tmp_path):
    path, _ = base
    with pytest.raises(ValueError):
        load(path, "cpu", "fp32", prefix_cache=True, runtime_dir=str(tmp_path))
    m = load(path, "cpu", "fp32")
    s = m.engine.add_sequence(ids(5))
    m.engine.prefill([s])
    with pytest.raises(ValueError):
        m.engine.verify([s], [[1, 2]])
    assert not m.engine.poisoned and len(m.engine.decode([s])) == 1
    with pytest.raises(ValueError):
        load(path, "cpu", "bf16", kv_format="affine8")


def test_prefix_cache_and_verification_without_states(tmp_path):
    """A model of attention layers alone keeps both."""
    cfg = SIZES["attention only, no loop"]
    w = O.tensors(cfg, seed=5)
    path = write(tmp_path, cfg, w)
    m = load(path, "cpu", "fp32", prefix_cache=True, runtime_dir=str(tmp_path))
    p = ids(90, seed=70)
    m.prefill(p[:70])
    assert m.prefill(p) == int(O.forward(cfg, w, p)[0][-1].argmax()) and m.prefix_store().hits == 1
    m.reset()
    s = m.engine.add_sequence(p[:60])
    m.engine.prefill([s])
    s.pending = p[60]
    got = m.engine.verify([s], [p[61:64]])[0]
    assert got == O.forward(cfg, w, p[:64])[0][60:].argmax(-1).tolist()


# ------------------------------------------------------------------------------------------
# configuration, checkpoint, command line, runner
# ------------------------------------------------------------------------------------------
def test_configuration_is_read_and_checked(base):
    path, _ = base
    s = read_model_spec(path)
    assert (s.arch, s.layers, s.hidden, s.vocab, s.loop) == ("rudorax", 7, 104, 198, (1, 3, 2)) and s.runs == [0, 1, 2, 1, 2, 3, 4] == O.run_order(CFG)
    assert s.kv_geometry() == [(1, 32, 16), (0, 0, 0), (2, 48, 32), (0, 0, 0), (2, 48, 32), (0, 0, 0), (2, 32, 32)]
    assert [l.window for l in s.layer_specs] == [50, 0, 37, 0, 64] and s.layer_specs[3].moe is None and s.layer_specs[1].gate_cap == 7.0
    l = s.layer_specs[2]
    n = 130
    assert l.pairs_seen(n) == int(O.window_visible(n, 37).sum()) and l.keys_seen(n) == int(O.window_visible(n, 37)[-1].sum())
    assert l.rope == RopeSpec(base=900.0, dims=40, factor=3.0, original=300, fast=20.0, slow=2.0)
    weights = {n: t for n, t in O.tensors(CFG).items() if t.dim() == 2 and n not in ("embed", "head")}
    assert sum(t.numel() for t in weights.values()) == s.dense_param_count() - 2 * s.vocab * s.hidden
    for change in ({"type": "recurrence"}, {"mlp": {"kind": "dense", "ff": 8}}, {"mixer": A(heads=3)["mixer"]}, {"mixer": A(scale=0.0)["mixer"]},
                   {"mixer": A(turn=O.rot(dims=7))["mixer"]}, {"mixer": A(turn=O.rot(dims=34))["mixer"]}, {"mlp": O.moe(top=9)}):
        with pytest.raises(ConfigError):
            spec_from_hf_config(dict(CFG, loop=None, layers=[dict(A(), **change)]))
    with pytest.raises(ConfigError):
        spec_from_hf_config(dict(CFG, layers=[M(gate_cap=0.0)], loop=None))
    for loop in ((3, 6, 2), (2, 1, 2), (0, 2, 0)):
        with pytest.raises(ConfigError):
            spec_from_hf_config(O.config(LAYERS, loop=loop))


def test_checkpoint_is_audited(tmp_path):
    w = O.tensors(CFG)
    changes = (("l1.mix.f.b", None), (None, ("l3.mlp.e0.gate", torch.zeros(2, 2))), ("l0.mlp.router", ("l0.mlp.router", torch.zeros(6, 104))),
               ("l2.mlp.e5.down", None), ("l0.mix.sink", None))
    for i, (drop, put) in enumerate(changes):
        t = {n: x for n, x in w.items() if n != drop}
        if put:
            t[put[0]] = put[1].to(torch.bfloat16)
        with pytest.raises(CheckpointError):
            load(write(tmp_path, CFG, t, f"m{i}"), "cpu", "bf16")
    # tensors of a part the configuration switches off may be there
    load(write(tmp_path, CFG, dict(w, **{"l3.norm2": w["l3.norm1"].clone()}), "more"), "cpu", "bf16")


def test_planner_counts_what_a_run_keeps():
    from flyingfish_b200.planner.plan import DeviceInfo, plan_memory
    s = named_shape("rudorax-tiny")
    info = DeviceInfo(name="x", total_bytes=1 << 30, free_bytes=1 << 30)
    p = plan_memory(s, Settings(capacity=256, max_batch=2, kv_tokens=1000), info, 0)
    assert p.kv_blocks == 16 and p.kv_bytes == 16 * 64 * 2 * sum(h * (a + b) for h, a, b in s.kv_geometry())
    none = spec_from_hf_config(SIZES["memories only"])
    assert plan_memory(none, Settings(capacity=256, max_batch=2), info, 0).kv_blocks == 9


def test_command_line_generates(base, capsys):
    from flyingfish_b200.cli import main
    path, w = base
    p = ids(12, seed=80)
    assert main(["--model", path, "--cpu", "--dtype", "fp32", "--kv-tokens", "256", "--capacity", "128", "generate", "--tokens",
                 ",".join(map(str, p)), "--max-new-tokens", "6", "--ignore-eos"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    greedy_agrees(w, p, out["generated_ids"], "fp32")
    assert main(["--model", path, "inspect"]) == 0
    assert json.loads(capsys.readouterr().out)["spec"]["arch"] == "rudorax"


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
    from flyingfish_b200.serve.trace_runner import LIVE_REQUESTS, TraceRunner, load_engine
    path, w = base
    m, e = load_engine(path, dtype, 192, device)
    assert e.kv.num_blocks == 3 and len(e.state_slots) == LIVE_REQUESTS
    r = TraceRunner(e, m.spec.vocab)
    toks, steps = _trace()
    want = _trace_wants(w, toks)
    for s in steps:
        out = r.step(s["entries"], s["end"])
        if s["step"] in want:
            agree(out, want[s["step"]], dtype, f"step {s['step']}")
        else:
            assert out is None
    assert not r.live and e.kv.alloc.free_blocks == 3 and len(e.state_slots) == LIVE_REQUESTS


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
        agree(got, want, "bf16" if dtype == "bfloat16" else "fp32", f"step {i}")
    assert not (tmp_path / "1.f32").exists()


def test_random_shape_generates():
    m = Model.load("rudorax-tiny", Settings(capacity=128, max_batch=2), device="cpu", seed=3)
    out = m.generate_batch([[1, 2, 3], [4] * 50], 5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 512 for o in out for t in o)


@GPU
def test_random_shape_gpu_matches_cpu():
    from _oracle import assert_tokens_equal_up_to_ties
    st = Settings(capacity=256, max_batch=2)
    cpu, gpu = (Model.load("rudorax-tiny", st, device=d, seed=3) for d in ("cpu", "cuda"))
    prompts = [ids(80, 512, 1), ids(9, 512, 2)]
    for p, a, b in zip(prompts, cpu.generate_batch(prompts, 12), gpu.generate_batch(prompts, 12)):
        assert_tokens_equal_up_to_ties(cpu, p, a, b)
    ops.check_status()
