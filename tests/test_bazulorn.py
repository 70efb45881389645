"""Bazulorn decoder against the plain restatement in ``bazulorn_oracle``: every mechanism alone, whole prompts, portions, mixed
batches, decoding, window edges, far keys, states and blocks that are used again, sizes that need padding, and generation through
the scheduler. Every case runs on the CPU oracles of the operators and, on a GPU, through the kernels in BF16 and FP32."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import bazulorn_oracle as O
from _design import GPU, TORCH, close, each_form, feed_in_cuts, ids, load, paged
from _design import write as write_dir
from flyingfish_b200 import ops
from flyingfish_b200.api import Model, generate_plain
from flyingfish_b200.config import ConfigError, Settings, named_shape, read_model_spec, spec_from_hf_config
from flyingfish_b200.engine.engine import Span
from flyingfish_b200.engine.scheduler import Request, Scheduler
from flyingfish_b200.loaders.checkpoint import CheckpointError
from flyingfish_b200.ops import delta_ops, moe_ops, ref, residual_ops, ssd_ops, talk_ops

# heads' outputs are divided by their root mean square: where they nearly cancel, rounding is magnified
MODEL_LIMIT = {"fp32": 2e-4, "bf16": 0.1}
A, D = O.pair_layer, O.delta_layer


def agree(got, want, dtype, what):
    close(got, want, dtype, what, MODEL_LIMIT[dtype])


def write(tmp_path, cfg, tensors, name="m"):
    return write_dir(tmp_path, O.public(cfg), tensors, name)


# unequal layers, a layer of each kind without a feed-forward, a dense one
LAYERS = [D(mlp=O.dense()), A(kv_heads=1, vdim=16), D(heads=3, kv_heads=3, dim=40, vdim=24, conv=2, ranks=(7, 30)),
          A(size=37, dim=48, heads=6, kv_heads=2, scale=0.25, ssd=dict(heads=4, groups=1, conv=5, norm_groups=1, state=33), mlp=O.moe(top=1, shared=0)),
          D(kv_heads=4, mlp=None), A(size=64, mlp=None)]
CFG = O.config(LAYERS)


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    w = O.tensors(CFG)
    return write(tmp_path_factory.mktemp("bazulorn"), CFG, w), w


def packed(g, n, heads, d, p):
    t = torch.zeros(n, heads, p)
    t[..., :d] = torch.randn(n, heads, d, generator=g)
    return t.reshape(n, heads * p)


def starts_of(lens, device):
    return torch.tensor([0] + list(lens)).cumsum(0).to(torch.int32).to(device)


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(61, 13, 5), (1, 1, 1), (65537, 40961, 70001), (521, 0, 3)])
def test_bigram_rows(device, buckets, mul_prev, mul_cur):
    """Sequences cut into calls, one paused, two that never meet; the first token has the row behind the last bucket."""
    cfg = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    toks = {0: ids(300, 50000, 1), 1: ids(7, 50000, 2), 2: ids(40, 50000, 3)}
    last = torch.full((5,), -1, dtype=torch.int32, device=device)
    slot, at, got = {0: 3, 1: 0, 2: 4}, dict.fromkeys(toks, 0), {s: [] for s in toks}
    for step in ([(0, 1), (2, 38)], [(1, 2), (0, 270)], [(0, 1), (1, 5), (2, 1)], [(2, 1), (0, 28)]):
        part = [toks[s][at[s]: at[s] + n] for s, n in step]
        rows = residual_ops.bigram_rows(torch.tensor(sum(part, []), dtype=torch.int32, device=device), last, starts_of([n for _, n in step], device),
                                        torch.tensor([slot[s] for s, _ in step], dtype=torch.int32, device=device), **cfg).tolist()
        for s, n in step:
            got[s] += rows[:n]
            rows, at[s] = rows[n:], at[s] + n
    for s, t in toks.items():
        assert got[s] == O.bigram_rows(t, cfg) and got[s][0] == buckets and all(0 <= r < buckets for r in got[s][1:])
    assert last.tolist() == [toks[1][-1], -1, -1, toks[0][-1], toks[2][-1]]


@each_form
@pytest.mark.parametrize("width,true_width", [(64, 64), (104, 100), (1024, 1024), (40, 37)])
def test_embedding_pair_and_sum_of_two_mixers(device, dtype, width, true_width):
    g = torch.Generator().manual_seed(width)
    dt, rows, eps, t = TORCH[dtype], 7, 1e-2, slice(0, true_width)
    mask = (torch.arange(width) < true_width).float()
    rn = lambda *s: torch.randn(*s, generator=g) * mask
    dev = lambda x: x.to(device)
    table, second, w0, w1 = rn(30, width).to(dt), rn(12, width).to(dt), (1 + rn(width)) * mask, 1 + rn(width)
    tok, row = (torch.randint(0, n, (rows,), generator=g).to(torch.int32) for n in (30, 12))
    lim = 1e-5 if dtype == "fp32" else 8e-3
    x, n1, n2 = residual_ops.embed(dev(tok), dev(table), 1.0, dev(w1), None, eps, true_width, second=residual_ops.Second(dev(second), dev(row), dev(w0)))
    want = O.rms((table.double()[tok.long()] + second.double()[row.long()])[:, t], eps) * w0.double()[t]
    assert n2 is None
    close(x[:, t], want, dtype, "stream", 1e-5)
    close(n1[:, t], O.rms(want, eps) * w1.double()[t], dtype, "norm", lim)
    a, r, b = (3.0 * rn(rows, width).to(dt) for _ in range(3))
    r[2] *= 1e-3                                     # the norm's eps counts
    wa, wr = (rn(width) for _ in range(2))
    for extra in (None, b):
        want = want + O.rms(a.double()[:, t], eps) * wa.double()[t] + O.rms(r.double()[:, t], eps) * wr.double()[t]
        want = want if extra is None else want + b.double()[:, t]
        n1, _ = residual_ops.step(x, dev(a), None if extra is None else dev(b), None, dev(w1), None, eps, true_width,
                                  beside=residual_ops.Beside(dev(r), dev(wa), dev(wr)))
        close(x[:, t], want, dtype, "sum", 1e-5)
        close(n1[:, t], O.rms(want, eps) * w1.double()[t], dtype, "norm", lim)


@each_form
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 8])
@pytest.mark.parametrize("nh,dn,vh,dv,bias", [(4, 24, 3, 40, False), (2, 128, 2, 200, True), (6, 16, 1, 16, True), (2, 264, 4, 8, False)])
def test_short_convolution(device, dtype, taps, nh, dn, vh, dv, bias):
    """Portions from one row on (shorter than the convolution's reach), sequences beside each other, slots out of order."""
    g = torch.Generator().manual_seed(taps * dn)
    dt, lens = TORCH[dtype], [70, 23]
    pad = lambda d: (d + 7) // 8 * 8
    ch = nh * pad(dn) + vh * pad(dv)
    x = [torch.cat([packed(g, n, nh, dn, pad(dn)), packed(g, n, vh, dv, pad(dv)), torch.randn(n, 8, generator=g)], 1).to(dt) for n in lens]
    w, b = torch.randn(taps, ch, generator=g), torch.randn(ch, generator=g) if bias else None
    conv = delta_ops.ConvWeights(w.to(device), None if b is None else b.to(device), nh, pad(dn), vh, pad(dv))
    want = [O.silu(O.causal_conv(t[:, :ch].double(), w.t().double(), None if b is None else b.double())) for t in x]
    st = delta_ops.ConvState(4, conv, device)
    st.x.fill_(7.0)
    slots = [2, 0]
    for s in slots:
        st.reset(s)
    at, lim = [0, 0], 2e-5 if dtype == "fp32" else 8e-3
    for cut in ((1, 2), (1, 0), (2, 20), (40, 1), (26, 0)):
        live = [i for i in (0, 1) if cut[i]]
        part = torch.cat([x[i][at[i]: at[i] + cut[i]] for i in live]).to(device)
        y, unit = delta_ops.short_conv(part, conv, st, starts_of([cut[i] for i in live], device),
                                       torch.tensor([slots[i] for i in live], dtype=torch.int32, device=device), max(cut), unit_scale=0.3)
        ref_y = torch.cat([want[i][at[i]: at[i] + cut[i]] for i in live])
        close(y, ref_y, dtype, f"rows {cut}", lim)
        h = y[:, : nh * pad(dn)].double().cpu().view(-1, nh, pad(dn))
        f = torch.tensor([0.3] * (nh // 2) + [1.0] * (nh - nh // 2), dtype=torch.float64)
        close(unit, f / torch.sqrt((h * h).sum(-1) + 1e-6), "fp32", "unit factors", 1e-5)
        at = [a + c for a, c in zip(at, cut)]
    assert at == lens and (st.x[[1, 3]] == 7.0).all()
    for s, t in zip(slots, x):
        if taps > 1:
            assert torch.equal(st.x[s].cpu(), t[-(taps - 1):, :ch].float())


@each_form
@pytest.mark.parametrize("dim,vdim,heads,groups,strength", [(24, 40, 4, 2, -1.5), (64, 64, 2, 2, 0.0), (128, 128, 2, 1, -3.0), (16, 200, 1, 1, 2.5),
                                                             (96, 72, 3, 3, 5.0), (144, 24, 2, 1, -1.0)])
def test_channel_delta_rule(device, dtype, monkeypatch, dim, vdim, heads, groups, strength):
    """Several sequences in slots out of order, their rows cut into calls from one token to several chunks; decays from nearly none to
    all of the state at once; the chunked form in one round and in several; stale slots reset."""
    g = torch.Generator().manual_seed(dim)
    dt, dk, dv = TORCH[dtype], (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    lens, cuts = [390, 131], [(1, 64), (63, 2), (2, 65), (324, 0)]
    rate = -torch.exp(torch.randn(heads, generator=g) + strength)
    bias = torch.randn(heads * dk, generator=g) - 1.0
    seqs, want = [], []
    for n in lens:
        x = torch.cat([packed(g, n, 2 * groups, dim, dk), packed(g, n, heads, vdim, dv)], 1).to(dt)
        z = torch.randn(n, heads * dk, generator=g) * 2.0
        z[5], z[90], z[91:95] = -40.0, 30.0, 8.0                     # nothing forgotten, everything, most of it
        b = (torch.randn(n, heads, generator=g) * 2.0).to(dt)
        qk = x[:, : 2 * groups * dk].double().view(n, 2 * groups, dk)[..., :dim]
        unit = torch.rsqrt((qk * qk).sum(-1) + 1e-6)
        unit[:, :groups] *= dim ** -0.5
        seqs.append((x, unit.float(), z, b))
        qk = (qk * unit[..., None]).repeat_interleave(heads // groups, 1)
        decay = torch.exp(rate.double()[:, None] * O.softplus((z + bias).double()).view(n, heads, dk)[..., :dim])
        v = x[:, 2 * groups * dk:].double().view(n, heads, dv)[..., :vdim]
        want.append(O.delta_rule(qk[:, :heads], qk[:, heads:], v, torch.sigmoid(b.double()), decay))
    for budget in (delta_ops.SCRATCH_BYTES, 1):
        monkeypatch.setattr(delta_ops, "SCRATCH_BYTES", budget)
        st = delta_ops.DeltaState(5, heads, groups, dk, dv, device)
        st.S.fill_(3.0)
        slots, at = [3, 1], [0, 0]
        for s in slots:
            st.reset(s)
        for cut in cuts:
            live = [i for i in (0, 1) if cut[i]]
            x, unit, z, b = (torch.cat([seqs[i][k][at[i]: at[i] + cut[i]] for i in live]).to(device) for k in range(4))
            out = torch.full((x.shape[0], heads, dv), 9.0, device=device)
            delta_ops.delta_rule(x, unit, z, b, rate.to(device), bias.to(device), st, starts_of([cut[i] for i in live], device),
                                 torch.tensor([slots[i] for i in live], dtype=torch.int32, device=device), out, max(cut))
            w = torch.cat([want[i][at[i]: at[i] + cut[i]] for i in live])
            scale = w.abs().max()
            assert (out[..., :vdim].double().cpu() - w).abs().max() <= 5e-5 * scale, f"portion {cut} at {at}"
            assert (out[..., vdim:] == 0).all()
            at = [a + c for a, c in zip(at, cut)]
        assert at == lens and (st.S[[0, 2, 4]] == 3.0).all() and (st.S[slots][:, :, dim:] == 0).all()
    gate = torch.randn(4, heads * dv, generator=g).to(dt)
    o, wn = torch.zeros(4, heads, dv), torch.zeros(dv)
    o[..., :vdim], wn[:vdim] = want[1][-4:].float(), 1 + 0.3 * torch.randn(vdim, generator=g)
    y = delta_ops.head_out(o.to(device), gate.to(device), wn.to(device), vdim, 0.01)
    ref_y = O.rms(o[..., :vdim].double(), 0.01) * wn[:vdim].double() * torch.sigmoid(gate.double().view(4, heads, dv)[..., :vdim])
    close(y.view(4, heads, dv)[..., :vdim].reshape(-1, vdim), ref_y.reshape(-1, vdim), dtype, "out", 1e-5 if dtype == "fp32" else 8e-3)


@each_form
@pytest.mark.parametrize("state,vdim,heads,groups,parts", [(20, 28, 6, 3, 4), (64, 64, 4, 1, 1), (128, 64, 4, 4, 8), (16, 200, 2, 2, 5), (144, 24, 3, 1, 9), (272, 16, 1, 1, 2)])
def test_state_space(device, dtype, monkeypatch, state, vdim, heads, groups, parts):
    """As the delta rule's test, with segments of long prompts; then the gate and the norm in parts that do not follow the heads."""
    monkeypatch.setattr(ssd_ops, "SEGMENT_ROWS", 128)
    monkeypatch.setattr(ssd_ops, "FILL_CTAS", 1 << 30)
    g = torch.Generator().manual_seed(state)
    dt, dk, dv = TORCH[dtype], (state + 15) // 16 * 16, (vdim + 15) // 16 * 16
    lens, cuts = [390, 131], [(1, 64), (63, 2), (2, 65), (324, 0)]
    rate, skip, bias = -torch.exp(torch.randn(heads, generator=g)), torch.randn(heads, generator=g), torch.randn(heads, generator=g) - 2.0
    seqs, want = [], []
    for n in lens:
        x = torch.cat([packed(g, n, 2 * groups, state, dk), packed(g, n, heads, vdim, dv)], 1).to(dt)
        z = (torch.randn(n, heads, generator=g) * 2.0).to(dt)
        z[5], z[90] = 30.0, -60.0                                    # a token that wipes the state, one that is not taken in
        seqs.append((x, z))
        m = x[:, : 2 * groups * dk].double().view(n, 2 * groups, dk)[..., :state].repeat_interleave(heads // groups, 1)
        v = x[:, 2 * groups * dk:].double().view(n, heads, dv)[..., :vdim]
        want.append(O.state_space(v, m[:, heads:], m[:, :heads], O.softplus(z.double() + bias.double()), rate.double(), skip.double()))
    st = ssd_ops.SsdState(5, heads, groups, dk, dv, device)
    st.S.fill_(3.0)
    slots, at = [3, 1], [0, 0]
    for s in slots:
        st.reset(s)
    for cut in cuts:
        live = [i for i in (0, 1) if cut[i]]
        x, z = (torch.cat([seqs[i][k][at[i]: at[i] + cut[i]] for i in live]).to(device) for k in range(2))
        out = torch.full((x.shape[0], heads, dv), 9.0, device=device)
        ssd_ops.state_space(x, z, bias.to(device), rate.to(device), skip.to(device), st, starts_of([cut[i] for i in live], device),
                            torch.tensor([slots[i] for i in live], dtype=torch.int32, device=device), out, max(cut))
        w = torch.cat([want[i][at[i]: at[i] + cut[i]] for i in live])
        close(out[..., :vdim].reshape(-1, vdim), w.reshape(-1, vdim), dtype, f"portion {cut} at {at}", 2e-3)
        assert ((out[..., :vdim].double().cpu() - w).norm(dim=-1) / w.norm(dim=-1)).median() < 1e-5
        assert (out[..., vdim:] == 0).all()
        at = [a + c for a, c in zip(at, cut)]
    assert at == lens and (st.S[[0, 2, 4]] == 3.0).all()
    rows = 5
    o, wn, z = torch.zeros(rows, heads, dv), torch.zeros(heads, dv), torch.randn(rows, heads * dv, generator=g).to(dt)
    o[..., :vdim], wn[:, :vdim] = torch.randn(rows, heads, vdim, generator=g), 1 + 0.3 * torch.randn(heads, vdim, generator=g)
    if heads * vdim % parts == 0:
        y = ssd_ops.gated_out(o.to(device), z.to(device), wn.reshape(-1).to(device), vdim, parts, 0.01).view(rows, heads, dv)
        own = lambda t: t.double().reshape(rows, heads, dv)[..., :vdim].reshape(rows, -1)
        ref_y = O.gated_group_norm(own(o), own(z), parts, wn[:, :vdim].double().reshape(-1), 0.01)
        close(y[..., :vdim].reshape(rows, -1), ref_y, dtype, "gated norm", 1e-5 if dtype == "fp32" else 8e-3)
        assert (y[..., vdim:] == 0).all()


@each_form
@pytest.mark.parametrize("dk,dv,hq,hkv", [(128, 128, 8, 2), (64, 32, 6, 2), (16, 16, 1, 1), (80, 112, 20, 2), (48, 16, 5, 5), (144, 160, 2, 1), (32, 48, 40, 4)])
@pytest.mark.parametrize("size", [1, 50, 64, 65, 1000])
def test_windowed_attention_with_mixed_heads(device, dtype, monkeypatch, dk, dv, hq, hkv, size):
    """Prompt portions and decoded rows; the last query of a sequence looks like the first key of its window in one case and like the
    key before it in the other, so that leaving the one out or letting the other in shows. Scores around zero: the soft-max's extra
    term takes a good part of the weight where few keys are seen."""
    dt, scale = TORCH[dtype], dk ** -0.5
    ctx, qlen = [300, 65, 128, 201, 51, 7, 1], [300, 2, 70, 150, 1, 7, 1]
    kc, vc, bt, ks, vs = paged(device, dt, hkv, dk, dv, ctx, seed=size + dk)
    g = torch.Generator().manual_seed(3)
    q0 = torch.randn(sum(qlen), hq * dk + 16, generator=g)
    talk = (torch.eye(hq) + 0.5 * torch.randn(hq, hq, generator=g)).to(torch.bfloat16).float()
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    i32 = lambda t: torch.as_tensor(t, dtype=torch.int32).to(device)
    caches = tuple(t.to(device) for t in (kc, vc, bt))
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
            full = torch.zeros(ctx[b], hq, dk, dtype=torch.float64)
            full[ctx[b] - n:] = q[r, : hq * dk].double().view(n, hq, dk)
            o = O.talking_attention(full, ks[b].transpose(0, 1), vs[b].transpose(0, 1), scale, size, talk.double())
            want.append(o[ctx[b] - n:].reshape(n, hq * dv))
            last.append(int(starts[b]) + n - 1)
        want = torch.cat(want)
        args = (hq, hkv, scale, size, talk.to(device), True)
        for budget in (talk_ops.ROUND_BYTES, 1):                     # one round of tiles, and one tile of every sequence a round
            monkeypatch.setattr(talk_ops, "ROUND_BYTES", budget)
            out = torch.full((q.shape[0], hq * dv), 9.0, dtype=dt, device=device)
            talk_ops.talk_prefill(q.to(device), *caches, starts.to(device), i32(qlen), i32(ctx), max(qlen), max(ctx), *args, out=out)
            close(out, want, dtype, "prompt", lim)
        for ctas in (1, 10000):                                      # one CTA per key head, and a split for every page
            monkeypatch.setattr(talk_ops, "DECODE_CTAS", ctas)
            out = torch.full((len(ctx), hq * dv), 9.0, dtype=dt, device=device)
            talk_ops.talk_decode(q[last].contiguous().to(device), *caches, i32(ctx), max(ctx), *args, out=out)
            close(out, want[last], dtype, "decode", lim)
    if device == "cuda":
        ops.check_status()


@each_form
def test_attention_without_the_extra_term_and_padding_rows(device, dtype):
    """``one`` off; and a decoded row without a sequence (no keys) gives zeros."""
    dt, hq, hkv, d = TORCH[dtype], 4, 2, 32
    kc, vc, bt, ks, vs = paged(device, dt, hkv, d, d, [100, 70], seed=1)
    g = torch.Generator().manual_seed(3)
    q, talk = torch.randn(2, hq * d, generator=g).to(dt), torch.randn(hq, hq, generator=g).to(torch.bfloat16).float()
    ctx = torch.tensor([100, 0], dtype=torch.int32, device=device)
    out = torch.full((2, hq * d), 9.0, dtype=dt, device=device)
    talk_ops.talk_decode(q.to(device), kc.to(device), vc.to(device), bt.to(device), ctx, 100, hq, hkv, 0.3, 60, talk.to(device), False, out=out)
    k, v = ks[0][:, 40:100], vs[0][:, 40:100]
    w = torch.stack([torch.softmax(q[0].double().view(hq, d)[h] @ k[h // 2].T * 0.3, -1) for h in range(hq)])
    m = talk.double() @ w
    close(out[:1], torch.cat([m[h] @ v[h // 2] for h in range(hq)])[None], dtype, "row", 2e-5 if dtype == "fp32" else 1.5e-2)
    assert (out[1] == 0).all()


def test_window_mask_restatement():
    assert [torch.nonzero(r).flatten().tolist() for r in O.window_visible(5, 3)] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4]]


@each_form
@pytest.mark.parametrize("dim,vdim,hq,hkv", [(32, 24, 4, 2), (20, 40, 3, 3), (128, 128, 8, 2), (136, 264, 2, 1)])
def test_value_norm_and_cache_write(device, dtype, dim, vdim, hq, hkv):
    g = torch.Generator().manual_seed(dim)
    dt, rows, eps = TORCH[dtype], 9, 0.05
    dk, dv = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    row = torch.cat([packed(g, rows, hq, dim, dk), packed(g, rows, hkv, dim, dk), packed(g, rows, hkv, vdim, dv), torch.randn(rows, 8, generator=g)], 1).to(dt)
    slots = torch.tensor([5, 64, 127, 0, 191, -1, 70, 33, 1], dtype=torch.int32)
    kc, vc = (torch.zeros(3, hkv, 64, d, dtype=dt, device=device) for d in (dk, dv))
    qkv = row.clone().to(device)
    ops.head_norm_kv(qkv, slots.to(device), kc, vc, hq, hkv, dim, vdim, eps, norm_qk=False, norm_v=True)
    assert torch.equal(qkv.cpu(), row)
    k = row[:, hq * dk: (hq + hkv) * dk].view(rows, hkv, dk)
    v = O.rms(row[:, (hq + hkv) * dk: -8].double().view(rows, hkv, dv)[..., :vdim], eps)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(kc[s // 64, :, s % 64].cpu(), k[r])
            close(vc[s // 64, :, s % 64, :vdim], v[r], dtype, "v", 2e-6 if dtype == "fp32" else 6e-3)
    assert int((kc != 0).any(-1).sum()) == 8 * hkv


@each_form
@pytest.mark.parametrize("rows,f,width", [(3, 128, 104), (40, 256, 72), (130, 128, 64), (300, 384, 256)])
def test_clamped_gate_in_the_projection(device, dtype, rows, f, width):
    """Gates and inputs on both sides of the limit; the limit is a parameter."""
    g = torch.Generator().manual_seed(rows)
    dt = TORCH[dtype]
    x = torch.randn(rows, width, generator=g).to(dt)
    gate, up = (3.0 * torch.randn(f, width, generator=g) / width ** 0.5 for _ in range(2))
    gate, up = gate.to(dt), up.to(dt)
    for limit in (0.5, 7.0):
        y = ops.linear_swiglu(x.to(device), ref.interleave_gate_up(gate, up).to(device), mode=5, limit=limit)
        a, u = (x.double() @ gate.double().T).clamp(max=limit), (x.double() @ up.double().T).clamp(-limit, limit)
        close(y, a * torch.sigmoid(1.702 * a) * (u + 1.0), dtype, f"limit {limit}", 2e-5 if dtype == "fp32" else 8e-3)


@each_form
@pytest.mark.parametrize("experts,top,ff,width,rows,limit", [(6, 3, 40, 104, 37, 1.5), (5, 1, 64, 64, 3, 0.3), (12, 12, 72, 40, 20, 2.0), (4, 2, 128, 256, 600, 7.0), (70, 6, 24, 64, 64, 1.0)])
def test_experts(device, dtype, experts, top, ff, width, rows, limit):
    """The bias is part of the logits, of the choice and of the weights; weights over the chosen logits alone."""
    g = torch.Generator().manual_seed(experts)
    dt = TORCH[dtype]
    lin = lambda o, i: (torch.randn(o, i, generator=g) / i ** 0.5).to(dt)
    t = {"router": 2 * lin(experts, width), "router.b": 2.0 * torch.randn(experts, generator=g)}
    for e in range(experts):
        t.update({f"e{e}.gate": 2 * lin(ff, width), f"e{e}.up": 2 * lin(ff, width), f"e{e}.down": lin(width, ff)})
    x = torch.randn(rows, width, generator=g).to(dt)
    get = lambda name: t[name].double()
    fp = (ff + 63) // 64 * 64
    grow = lambda w, r: torch.cat([w, w.new_zeros(r - w.shape[0], w.shape[1])])
    gu = torch.stack([ref.interleave_gate_up(grow(t[f"e{e}.gate"], fp), grow(t[f"e{e}.up"], fp)) for e in range(experts)])
    down = torch.stack([grow(t[f"e{e}.down"].T, fp).T for e in range(experts)]).contiguous()
    pad = grow(t["router"], (experts + 15) // 16 * 16)
    dev = lambda v: v.to(device)
    want_ids, want_w = O.choose_experts(x.double(), get, "", top)
    w, chosen = moe_ops.route(dev(x), dev(pad), top, "biased_softmax", dev(t["router.b"]), exact=True, experts=experts)
    assert torch.equal(chosen.cpu().long(), want_ids)
    close(w, want_w, dtype, "weights", 1e-5)
    assert (want_ids != O.choose_experts(x.double(), lambda k: get(k) * (k != "router.b"), "", top)[0]).any() or top == experts
    want = O.experts(x.double(), get, "", {"router": {"experts": experts, "top": top}, "expert": {"limit": limit}})
    for er in (moe_ops.expert_rows(dev(x), w, chosen, dev(gu), dev(down), limit),
               moe_ops.routed_rows(dev(x), dev(pad), top, "biased_softmax", dev(t["router.b"]), experts, dev(gu), dev(down), limit)):
        assert torch.equal(er.ids.cpu().long(), want_ids)
        s = torch.zeros(rows, width, device=device)
        residual_ops.step(s, dev(torch.zeros_like(x)), None, er, torch.ones(width, device=device), None, 1e-5, width)
        close(s, want, dtype, "sum", 1e-5 if dtype == "fp32" else 2e-2)


# ------------------------------------------------------------------------------------------
# the model: whole prompts, portions, decoding, batches
# ------------------------------------------------------------------------------------------
@each_form
def test_whole_prompt_and_layers(base, device, dtype):
    from flyingfish_b200.utils.trace import Trace
    path, w = base
    m = load(path, device, dtype)
    toks = ids(150)
    O.MARGINS.clear()
    want, after = O.forward(CFG, w, toks)
    assert min(O.MARGINS) > 0.1
    got, seq = feed_in_cuts(m.engine, toks, [150])
    agree(got, want, dtype, "logits")
    m.engine.free_sequence(seq.seq_id)
    m.engine.model.trace = Trace(device=device)
    feed_in_cuts(m.engine, toks, [150])
    for i in range(len(LAYERS)):
        agree(m.engine.model.trace.tensors[f"step.0.layer.{i}"], after[i], dtype, f"residual after layer {i}")


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
    for st in e.model.states:
        st.S.fill_(5.0)
    for st in e.model.convs:
        st.x.fill_(5.0)
    e.model.last_token.fill_(11)
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


def plain_start(cfg, seed):
    """Weights whose bigram table is empty and whose channels 0 and 1 are signs: 0 the same for every token, 1 only of token 7."""
    w = O.tensors(cfg, seed=seed)
    w["bigram"].zero_()
    w["embed.norm"].fill_(1.0)
    w["embed"][:, :4] = 0.0
    w["embed"][:, 0] = 3.0
    w["embed"][7, 1] = 9.0
    return w


def needle_attention(size):
    """One layer of which the attention alone counts, and in which token 7 is the key every query looks for: channel 0 of every token
    is the direction of the queries, channel 1 of token 7 alone that of its key."""
    dim, width = 32, 48
    cfg = O.config([A(size=size, dim=dim, vdim=24, heads=2, kv_heads=1, scale=0.5, mlp=None)], width=width, vocab=64)
    w = plain_start(cfg, 4)
    w["l0.mix.right.out"].zero_()
    w["l0.mix.left.out"].fill_(3.0)
    for name, heads, channel in (("q", 2, 0), ("k", 1, 1)):
        m = w["l0.mix.left." + name].view(heads, dim, width)
        m *= 0.2
        m[:, 31] = 0.0
        m[:, 31, channel] = 3.0
        w[f"l0.mix.left.{name}.b"] *= 0.1
    return cfg, w


def needle_delta():
    """One delta layer that takes in token 7 and next to nothing of the others, and forgets slowly. Channel 0 of every token puts
    queries and keys on one side."""
    cfg = O.config([D(heads=2, kv_heads=1, dim=24, vdim=32, mlp=None)], width=48, vocab=64)
    w = plain_start(cfg, 6)
    w["l0.mix.b"] = w["l0.mix.b"] * 0.0
    w["l0.mix.b"][:, 0], w["l0.mix.b"][:, 1] = -2.0, 4.0
    w["l0.mix.A_log"].fill_(-7.0)
    for name in ("q", "k"):
        w[f"l0.mix.{name}"] *= 0.2
        w[f"l0.mix.{name}"][:, 0] = 1.0
        w[f"l0.mix.{name}.conv"] *= 0.2
        w[f"l0.mix.{name}.conv"][:, -1] = 1.0
    return cfg, w


def needle_state_space():
    """One layer of which the state space alone counts: token 7 takes a large step, the others none to speak of, and nothing is
    forgotten. The input maps of every token look alike, so do the output maps."""
    cfg = O.config([A(ssd=dict(heads=2, groups=1, state=24, vdim=32, norm_groups=2), mlp=None)], width=48, vocab=64)
    w = plain_start(cfg, 6)
    w["l0.mix.left.out"].zero_()
    rows = w["l0.mix.right.in"]
    inner = 64
    rows[2 * inner: 2 * inner + 48] *= 0.2
    rows[2 * inner: 2 * inner + 48, 0] = 1.0
    rows[-2:] = 0.0
    rows[-2:, 1] = 2.0
    for name, v in (("dt_bias", -6.0), ("A_log", -9.0), ("D", 0.0)):
        w["l0.mix.right." + name].fill_(v)
    conv = w["l0.mix.right.conv"]
    conv[inner:] *= 0.2
    conv[inner:, -1] = 1.0
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
    for at in sorted({0, 1, min(size, n - 1), 63, 64}):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved, end = relative_change(want, without), at + size
        assert moved[at: end].min() > 0.15 and (moved[end:] < 1e-9).all() and (moved[:at] == 0).all()
        for cuts in ([n], [max(end - 3, 1), 1]):                  # the window's end in the prompt, and decoded
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")


@each_form
@pytest.mark.parametrize("make", [needle_delta, needle_state_space])
def test_the_state_keeps_a_far_token(tmp_path, device, dtype, make):
    cfg, w = make()
    e = load(write(tmp_path, cfg, w), device, dtype, capacity=512).engine
    n = 300
    plain = [t if t != 7 else 8 for t in ids(n, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    for at in (0, 1, 63, 64, 127):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved = relative_change(want, without)
        assert moved[at:].min() > 0.03 and moved[at:].median() > 0.12 and (moved[:at] == 0).all()
        for cuts in ([n], [at + 1, 2, 64, 65, 1], [100, 100, 60, 1]):
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")


@each_form
def test_previous_token_convolution_and_first_tokens(tmp_path, device, dtype):
    """What only the last few tokens carry: the bigram of a portion's first token, the convolution's inputs, the row of a sequence's
    first token. Each is made to count in the oracle, then portions are cut around it."""
    cfg = O.config([D(mlp=None), A(mlp=None)])
    w = O.tensors(cfg, seed=9)
    toks = ids(40, seed=9)
    want, _ = O.forward(cfg, w, toks)
    other, _ = O.forward(cfg, w, [toks[0] + 1 if toks[0] < 100 else toks[0] - 1] + toks[1:])
    assert relative_change(other, want)[1] > 0.3                   # the second token's row depends on the first
    last = dict(w, bigram=torch.cat([w["bigram"][:-1], -w["bigram"][-1:]]))
    assert relative_change(O.forward(cfg, last, toks)[0], want)[0] > 0.3
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    for cuts in ([1], [2], [3, 2, 1, 2], [1, 2, 36, 1], [39, 1]):
        got, seq = feed_in_cuts(e, toks, cuts)
        e.free_sequence(seq.seq_id)
        agree(got, want, dtype, str(cuts))


@each_form
def test_the_extra_term_and_the_mixing_matter(tmp_path, device, dtype, monkeypatch):
    cfg = O.config([A(heads=4, kv_heads=2, size=5, mlp=None)] * 2)
    w = O.tensors(cfg, seed=9)
    for i in range(2):
        w[f"l{i}.mix.right.out"].zero_()
    toks = ids(60, seed=9)
    want, _ = O.forward(cfg, w, toks)
    with monkeypatch.context() as m:
        m.setattr(O, "softmax_with_one", lambda s: torch.softmax(s, -1))
        assert relative_change(O.forward(cfg, w, toks)[0], want).median() > 0.02
    plain = {n: (torch.eye(4).to(torch.bfloat16) if n.endswith("talk") else t) for n, t in w.items()}
    assert relative_change(O.forward(cfg, plain, toks)[0], want).median() > 0.1
    turned = {n: (t.t().contiguous() if n.endswith("talk") else t) for n, t in w.items()}
    assert relative_change(O.forward(cfg, turned, toks)[0], want).median() > 0.1
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    for cuts in ([60], [3, 40, 1]):
        got, seq = feed_in_cuts(e, toks, cuts)
        e.free_sequence(seq.seq_id)
        agree(got, want, dtype, str(cuts))


SIZES = {
    "every number one": O.config([A(heads=1, kv_heads=1, dim=1, vdim=1, size=1, scale=1.0, ssd=dict(heads=1, groups=1, state=1, vdim=2, conv=1, norm_groups=1),
                                    mlp=O.moe(experts=1, top=1, ff=1, limit=1.0, shared=1, shared_limit=1.0)),
                                  D(heads=1, kv_heads=1, dim=2, vdim=1, conv=1, ranks=(1, 1), mlp=O.dense(1))], width=16, vocab=40, buckets=1, mul_prev=1, mul_cur=1),
    "tensor-core widths": O.config([A(heads=8, kv_heads=2, dim=128, vdim=128, scale=128 ** -0.5, size=96, ssd=dict(heads=4, groups=2, state=128, vdim=64, conv=4, norm_groups=2),
                                      mlp=O.moe(ff=128, shared=256)), D(heads=2, kv_heads=2, dim=128, vdim=128, ranks=(128, 128), mlp=O.dense(512))], width=256, vocab=512),
    "odd sizes": O.config([A(heads=3, kv_heads=3, dim=20, vdim=28, size=29, ssd=dict(heads=5, groups=5, state=13, vdim=9, conv=2, norm_groups=3), mlp=O.moe(ff=33, shared=17)),
                           D(heads=5, kv_heads=1, dim=12, vdim=28, conv=7, ranks=(3, 5), mlp=O.dense(35)), A(heads=9, kv_heads=3, dim=12, vdim=28, size=7)], width=75, vocab=131),
    "wide heads": O.config([A(heads=2, kv_heads=1, dim=144, vdim=200, size=70, scale=0.1, ssd=dict(heads=1, groups=1, state=264, vdim=136, norm_groups=1)),
                            D(heads=1, kv_heads=1, dim=144, vdim=136)]),
    "many heads": O.config([A(heads=33, kv_heads=11, dim=16, vdim=16, size=40, ssd=dict(heads=24, groups=8, state=16, vdim=16, norm_groups=8)), D(heads=20, kv_heads=4, dim=16, vdim=16)]),
    "windows of one and of all": O.config([A(heads=1, kv_heads=1, dim=16, vdim=16, size=1), A(heads=2, kv_heads=1, dim=16, vdim=16, size=100000)], buckets=4096, mul_prev=1, mul_cur=0),
    "delta layers only": O.config([D(), D(mlp=None), D(heads=2, kv_heads=1, dim=64, vdim=64, conv=8)], eps=0.2),
    "pairs only": O.config([A(), A(heads=12, kv_heads=4)]),
    "one expert, all experts": O.config([A(mlp=O.moe(experts=1, top=1)), D(mlp=O.moe(experts=3, top=3))]),
    "no shared expert": O.config([A(mlp=O.moe(shared=0)), D(mlp=O.moe(shared=0, limit=100.0))]),
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
    assert not O.MARGINS or min(O.MARGINS) > 0.1                  # no choice that rounding could turn
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
def test_long_prompt(base, dtype):
    """A prompt long enough for the state space's segments, then decoded on."""
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


# ------------------------------------------------------------------------------------------
# configuration, checkpoint, command line, runner
# ------------------------------------------------------------------------------------------
def test_configuration_is_read_and_checked(base):
    path, _ = base
    s = read_model_spec(path)
    assert (s.arch, s.layers, s.hidden, s.vocab, s.tie_embeddings) == ("bazulorn", 6, 104, 198, True)
    assert s.extra["bazulorn"] == {"buckets": 61, "mul_prev": 13, "mul_cur": 5}
    assert s.kv_geometry() == [(0, 0, 0), (1, 32, 16), (0, 0, 0), (2, 48, 32), (0, 0, 0), (2, 32, 32)]
    ls = s.layer_specs
    assert [l.window for l in ls] == [0, 50, 0, 37, 0, 64] and [(l.decay_rank, l.gate_rank) for l in ls if l.mixer == "channel_delta"] == [(20, 12), (7, 30), (20, 12)]
    assert ls[0].ffn == 88 and ls[4].moe is None and ls[3].moe.n_shared == 0 and ls[1].moe.shared_limit == 0.8 and ls[3].beside.norm_groups == 1
    l = ls[3]
    n = 130
    assert l.pairs_seen(n) == int(O.window_visible(n, 37).sum()) and l.keys_seen(n) == int(O.window_visible(n, 37)[-1].sum())
    small = ("embed", "bigram", "left.talk")
    weights = {k: t for k, t in O.tensors(CFG).items() if t.dim() == 2 and not k.endswith(small)}
    norms = sum(t.numel() for k, t in O.tensors(CFG).items() if k.endswith((".left.out", ".right.out")))
    assert sum(t.numel() for t in weights.values()) + norms == s.dense_param_count() - s.vocab * s.hidden
    right = lambda **kw: {"mixer": A(ssd=kw)["mixer"]}
    for change in ({"type": "recurrence"}, {"mlp": {"kind": "other", "ff": 8}}, {"mixer": A(heads=3)["mixer"]}, {"mixer": A(scale=0.0)["mixer"]},
                   {"mixer": A(size=0)["mixer"]}, right(groups=4), right(conv=0), right(conv=9), right(norm_groups=5), {"mlp": O.moe(top=9)},
                   {"mlp": O.moe(limit=0.0)}, {"mlp": O.moe(shared_limit=0.0)}):
        with pytest.raises(ConfigError):
            spec_from_hf_config(O.public(O.config([dict(A(), **change)])))
    for layers, kw in (([D(heads=3)], {}), ([D(conv=12)], {}), ([], {}), ([D()], {"buckets": 0}), ([D()], {"mul_prev": -1})):
        with pytest.raises(ConfigError):
            spec_from_hf_config(O.public(O.config(layers, **kw)))


def test_checkpoint_is_audited(tmp_path):
    w = O.tensors(CFG)
    changes = (("l0.mix.a2", None), (None, ("l3.mlp.e9.gate", torch.zeros(2, 2))), ("l1.mlp.router", ("l1.mlp.router", torch.zeros(5, 104))),
               ("l1.mlp.e5.down", None), ("l1.mix.left.talk", None), ("bigram", ("bigram", torch.zeros(61, 104))), (None, ("head", torch.zeros(198, 104))))
    for i, (drop, put) in enumerate(changes):
        t = {n: x for n, x in w.items() if n != drop}
        if put:
            t[put[0]] = put[1].to(torch.bfloat16)
        with pytest.raises(CheckpointError):
            load(write(tmp_path, CFG, t, f"m{i}"), "cpu", "bf16")
    with pytest.raises((ConfigError, CheckpointError)):
        load(write(tmp_path, CFG, {n: x for n, x in w.items() if n != "l0.mix.a1"}, "rank"), "cpu", "bf16")


def test_planner_counts_what_a_layer_keeps():
    from flyingfish_b200.planner.plan import DeviceInfo, plan_memory
    s = named_shape("bazulorn-tiny")
    info = DeviceInfo(name="x", total_bytes=1 << 30, free_bytes=1 << 30)
    p = plan_memory(s, Settings(capacity=256, max_batch=2, kv_tokens=1000), info, 0)
    assert p.kv_blocks == 16 and p.kv_bytes == 16 * 64 * 2 * sum(h * (a + b) for h, a, b in s.kv_geometry())
    none = spec_from_hf_config(O.public(SIZES["delta layers only"]))
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
    assert json.loads(capsys.readouterr().out)["spec"]["arch"] == "bazulorn"


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
    m = Model.load("bazulorn-tiny", Settings(capacity=128, max_batch=2), device="cpu", seed=3)
    out = m.generate_batch([[1, 2, 3], [4] * 50], 5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 512 for o in out for t in o)


@GPU
def test_random_shape_gpu_matches_cpu():
    from _oracle import assert_tokens_equal_up_to_ties
    st = Settings(capacity=256, max_batch=2)
    cpu, gpu = (Model.load("bazulorn-tiny", st, device=d, seed=3) for d in ("cpu", "cuda"))
    prompts = [ids(80, 512, 1), ids(9, 512, 2)]
    for p, a, b in zip(prompts, cpu.generate_batch(prompts, 12), gpu.generate_batch(prompts, 12)):
        assert_tokens_equal_up_to_ties(cpu, p, a, b)
    ops.check_status()
