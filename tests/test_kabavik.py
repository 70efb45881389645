"""Kabavik decoder against the plain restatement in ``kabavik_oracle``: every mechanism alone, whole prompts, portions, mixed batches,
decoding, window edges, kept first positions, far keys, blocks that are used again, sizes that need padding, and generation through
the scheduler. Every case runs on the CPU oracles of the operators and, on a GPU, through the kernels in BF16 and FP32."""
import dataclasses
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import kabavik_oracle as O
from _design import GPU, TORCH, close, each_form, feed_in_cuts, ids, load, paged, write
from flyingfish_b200 import ops
from flyingfish_b200.api import Model, generate_plain
from flyingfish_b200.config import ConfigError, RopeSpec, Settings, named_shape, read_model_spec, spec_from_hf_config
from flyingfish_b200.engine.engine import Span
from flyingfish_b200.engine.scheduler import Request, Scheduler
from flyingfish_b200.loaders.checkpoint import CheckpointError
from flyingfish_b200.ops import mla_ops, ref, residual_ops
from flyingfish_b200.ops.residual_ops import Norm

# the norms behind the sub-layers and the capped scores magnify rounding a little
MODEL_LIMIT = {"fp32": 1e-4, "bf16": 6e-2}


def agree(got, want, dtype, what):
    close(got, want, dtype, what, MODEL_LIMIT[dtype])


W, L, C = O.window_layer, O.latent_layer, O.capped_layer
# every mixer, a layer that shares keys and values across others, a layer without a feed-forward
LAYERS = [W(), C(), L(), W(size=37, keep=5, heads=2, kv_from=0), C(heads=6, kv_heads=3, dim=16, every=5, mlp=None), W(size=64, keep=0, kv_heads=6, vdim=40)]
CFG = O.config(LAYERS)


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    w = O.tensors(CFG)
    return write(tmp_path_factory.mktemp("kabavik"), CFG, w), w


def i32(t, device):
    return torch.as_tensor(t, dtype=torch.int32).to(device)


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@each_form
@pytest.mark.parametrize("width,true_width", [(64, 64), (104, 100), (1024, 1024), (40, 37), (2600, 2595)])
def test_residual_between_two_norms(device, dtype, width, true_width):
    g = torch.Generator().manual_seed(width)
    dt, rows, eps, t = TORCH[dtype], 7, 1e-3, slice(0, true_width)
    mask = (torch.arange(width) < true_width).float()
    rn = lambda *s: torch.randn(*s, generator=g) * mask
    dev = lambda x: x.to(device)
    table, tok = rn(30, width).to(dt), torch.randint(0, 30, (rows,), generator=g).to(torch.int32)
    vecs = {k: ((1 + rn(width)) * mask, rn(width)) for k in ("rms", "tanh")}
    made = {"rms": Norm("rms", dev(vecs["rms"][0])), "tanh": Norm("tanh", *map(dev, vecs["tanh"]), alpha=1.3), "copy": Norm()}

    def plain(kind, x):
        if kind == "copy":
            return x
        w, b = (v.double()[t] for v in vecs[kind])
        return O.rms(x, eps) * w if kind == "rms" else O.tanh_norm(x, 1.3, w, b)
    lim = 1e-5 if dtype == "fp32" else 8e-3
    for outer in made:
        x, n = residual_ops.embed_normed(dev(tok), dev(table), 1.7, made[outer], eps, true_width)
        want = table.double()[tok.long()] * 1.7
        close(x, want, dtype, "stream", 1e-6)
        close(n[:, t], plain(outer, want[:, t]), dtype, outer, lim)
        for inner in made:
            y = (2.0 * rn(rows, width)).to(dt)
            n = residual_ops.add_normed(x, dev(y), made[inner], made[outer], eps, true_width)
            want[:, t] += plain(inner, y.double()[:, t])
            close(x, want, dtype, f"sum of {inner}", 1e-5)
            close(n[:, t], plain(outer, want[:, t]), dtype, f"{outer} after {inner}", lim)
            assert (x[:, true_width:] == 0).all() and (n[:, true_width:] == 0).all()


@each_form
@pytest.mark.parametrize("m,n,k,ffn", [(1, 24, 104, 128), (9, 88, 256, 256), (64, 256, 2048, 128), (150, 40, 72, 384), (300, 264, 512, 128)])
def test_gelu_and_factors_in_the_epilogues(device, dtype, m, n, k, ffn):
    g = torch.Generator().manual_seed(m + n)
    dt = TORCH[dtype]
    rn = lambda *s: torch.randn(*s, generator=g)
    x, w, b = rn(m, k).to(dt), (rn(n, k) / k ** 0.5 * 2).to(dt), rn(n).to(dt)
    table, rows = rn(13, 3 * n).to(dt), torch.randint(0, 13, (m,), generator=g).to(torch.int32)
    part = table[:, n: 2 * n]
    dev = lambda t: t.to(device)
    lim = 2e-6 if dtype == "fp32" else 6e-3
    z = x.double() @ w.double().T
    got = ops.linear(dev(x), dev(w), act="gelu_tanh", mul=(dev(table)[:, n: 2 * n], dev(rows)))
    close(got, O.gelu_tanh(z) * part.double()[rows.long()], dtype, "gate times factors", lim)
    got = ops.linear(dev(x), dev(w), bias=dev(b), mul=(dev(table)[:, n: 2 * n], dev(rows)))
    close(got, (z + b.double()) * part.double()[rows.long()], dtype, "bias, factors", lim)
    close(ops.linear(dev(x), dev(w), bias=dev(b), act="gelu_tanh"), O.gelu_tanh(z + b.double()), dtype, "bias, gelu", lim)
    gate, up = ((rn(ffn, k) / k ** 0.5 * 2).to(dt) for _ in range(2))
    got = ops.linear_swiglu(dev(x), dev(ref.interleave_gate_up(gate, up)), mode=3)
    close(got, O.gelu_tanh(x.double() @ gate.double().T) * (x.double() @ up.double().T), dtype, "gated", lim)


@each_form
@pytest.mark.parametrize("rows,heads,n,k,x_cols,out_cols", [(1, 3, 64, 32, None, None), (70, 4, 48, 16, 32, 80), (200, 2, 512, 128, None, 576), (130, 5, 40, 72, None, None)])
def test_head_linear(device, dtype, rows, heads, n, k, x_cols, out_cols):
    """The columns of the rows between and behind the heads are neither read nor written."""
    g = torch.Generator().manual_seed(n)
    dt = TORCH[dtype]
    xc, oc = x_cols or k, out_cols or n
    x = torch.full((rows, (heads - 1) * xc + k + 24), float("nan"))
    w = (torch.randn(heads, n, k, generator=g) / k ** 0.5).to(dt)
    want = torch.empty(rows, heads, n, dtype=torch.float64)
    for h in range(heads):
        x[:, h * xc: h * xc + k] = torch.randn(rows, k, generator=g)
    if xc > k:                                   # what a tile reads past a head meets zeros: it must be finite
        x = torch.where(torch.isnan(x), torch.tensor(3.0), x)
    x = x.to(dt)
    for h in range(heads):
        want[:, h] = x.double()[:, h * xc: h * xc + k] @ w[h].double().T
    out = torch.full((rows, heads * oc + 8), 7.0, dtype=dt, device=device)
    got = ops.head_linear(x.to(device)[:, : (heads - 1) * xc + k], w.to(device), out=out, x_cols=x_cols, out_cols=out_cols)
    for h in range(heads):
        close(got[:, h * oc: h * oc + n], want[:, h], dtype, f"head {h}", 2e-6 if dtype == "fp32" else 6e-3)
        assert (got[:, h * oc + n: (h + 1) * oc] == 7.0).all()
    assert (got[:, heads * oc:] == 7.0).all()


def test_scaled_rotation_frequencies():
    for turn in (O.linear_rot(), O.linear_rot(64, 1e6, 8.0), dict(O.linear_rot(), scaling=None)):
        freqs, amp = RopeSpec(base=turn["base"], dims=turn["dims"], halves=True, factor=(turn["scaling"] or {"factor": 1.0})["factor"]).frequencies()
        want, _ = O.linear_frequencies(turn)
        assert torch.allclose(torch.tensor(freqs, dtype=torch.float64), want, rtol=1e-12) and amp == 1.0
    for turn in (O.yarn_rot(), O.yarn_rot(64, 1e6, 8.0, 4096, 32.0, 1.0), O.yarn_rot(2, factor=1.5), O.yarn_rot(10, original=8)):
        freqs, amp = RopeSpec(base=turn["base"], dims=turn["dims"], **turn["scaling"]).frequencies()
        want, wamp = O.yarn_frequencies(turn)
        assert torch.allclose(torch.tensor(freqs, dtype=torch.float64), want, rtol=1e-12) and amp == wamp


def _packed(g, rows, heads, d, p):
    t = torch.zeros(rows, heads, p)
    t[..., :d] = torch.randn(rows, heads, d, generator=g)
    return t.reshape(rows, heads * p)


@each_form
@pytest.mark.parametrize("dim,vdim,hq,hkv,dims", [(32, 24, 4, 2, 16), (20, 40, 3, 3, 12), (128, 128, 8, 2, 128), (136, 264, 2, 1, 6), (40, 16, 12, 0, 22)])
@pytest.mark.parametrize("whole", [True, False])
def test_norms_rotated_halves_temperature_and_cache_write(device, dtype, dim, vdim, hq, hkv, dims, whole):
    g = torch.Generator().manual_seed(dim)
    dt, rows, eps, first, pad = TORCH[dtype], 9, 0.05, 4990, lambda n: (n + 15) // 16 * 16
    dk, dv = pad(dim), pad(vdim)
    row = torch.cat([_packed(g, rows, hq, dim, dk)] + ([_packed(g, rows, hkv, dim, dk), _packed(g, rows, hkv, vdim, dv)] if hkv else []), 1).to(dt)
    many = lambda heads: heads if whole else 1
    wq, wk = 1 + 0.4 * torch.randn(many(hq), dim, generator=g), 1 + 0.4 * torch.randn(many(max(hkv, 1)), dim, generator=g)
    padded = lambda w: torch.cat([w, torch.zeros(w.shape[0], dk - dim)], 1).reshape(-1).to(device)
    slots = torch.tensor([5, 64, 127, 0, 191, -1, 70, 33, 1], dtype=torch.int32)
    kc, vc = (torch.zeros(3, hkv, 64, d, dtype=dt, device=device) for d in (dk, dv)) if hkv else (None, None)
    turn = O.linear_rot(dims=dims, base=300.0)
    freqs, amp = RopeSpec(base=300.0, dims=dims, factor=3.0, halves=True).frequencies()
    positions = torch.arange(first, first + rows, dtype=torch.int32, device=device)
    table = ops.rope_angles(positions, ops.rope_frequencies(freqs, device), amp)
    qkv = row.clone().to(device)
    ops.head_norm_kv(qkv, slots.to(device), kc, vc, hq, hkv, dim, vdim, eps, q_weight=padded(wq), k_weight=padded(wk) if hkv else None, cos_sin=table, whole=whole,
                     halves=True, temp=(positions, 0.7, 999))
    heads = lambda lo, n, d, p: row[:, lo: lo + n * p].double().view(rows, n, p)[..., :d]

    def normed(x, w):
        n = O.rms(x.reshape(rows, -1), eps).view(x.shape) if whole else O.rms(x, eps)
        return O.rotate_halves(n * w.double(), turn, first)
    lim = 2e-6 if dtype == "fp32" else 6e-3
    q = normed(heads(0, hq, dim, dk), wq) * O.query_temperature(rows, {"coef": 0.7, "every": 999}, first)[:, None, None]
    close(qkv[:, : hq * dk].view(rows, hq, dk)[..., :dim], q, dtype, "q", lim)
    if hkv:
        k, v = normed(heads(hq * dk, hkv, dim, dk), wk), heads((hq + hkv) * dk, hkv, vdim, dv)
        for r, s in enumerate(slots.tolist()):
            if s >= 0:
                close(kc[s // 64, :, s % 64, :dim], k[r], dtype, "k", lim)
                close(vc[s // 64, :, s % 64, :vdim], v[r], dtype, "v", lim)
        assert int((kc != 0).any(-1).sum()) == 8 * hkv


@each_form
@pytest.mark.parametrize("hkv", [2, 0])
def test_head_norm_with_a_temperature(device, dtype, hkv):
    """The per-head form without rotation; the factor changes at multiples of ``every``."""
    g = torch.Generator().manual_seed(3)
    dt, rows, dim, dk, hq = TORCH[dtype], 12, 40, 48, 4
    row = torch.cat([_packed(g, rows, hq, dim, dk)] + ([_packed(g, rows, hkv, dim, dk), _packed(g, rows, hkv, 16, 16)] if hkv else []), 1).to(dt)
    positions, slots = torch.arange(rows, dtype=torch.int32, device=device), i32(list(range(rows)), device)
    kc, vc = (torch.zeros(1, hkv, 64, d, dtype=dt, device=device) for d in (dk, 16)) if hkv else (None, None)
    wn = torch.cat([1 + 0.4 * torch.randn(dim, generator=g), torch.zeros(dk - dim)]).to(device)
    got = row.clone().to(device)
    ops.head_norm_kv(got, slots, kc, vc, hq, hkv, dim, 16, 1e-5, q_weight=wn, k_weight=wn, temp=(positions, 0.9, 4))
    f = O.query_temperature(rows, {"coef": 0.9, "every": 4})
    assert f[:3].eq(1.0).all() and f[3:7].eq(f[3]).all() and f[3] > 1.5 and f[7] > f[3]
    part = lambda lo, n: O.rms(row[:, lo: lo + n * dk].double().view(rows, n, dk)[..., :dim], 1e-5) * wn[:dim].double().cpu()
    lim = 2e-6 if dtype == "fp32" else 6e-3
    close(got[:, : hq * dk].view(rows, hq, dk)[..., :dim], part(0, hq) * f[:, None, None], dtype, "q", lim)
    if hkv:
        close(kc[0, :, :rows, :dim].transpose(0, 1), part(hq * dk, hkv), dtype, "k", lim)


@each_form
@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 24, 8, 56), (8, 128, 64, 512), (1, 16, 2, 16), (5, 40, 20, 136)])
def test_latent_norm_and_cache_write(device, dtype, heads, dim, rot, rank):
    g = torch.Generator().manual_seed(rank)
    dt, rows, eps, first, pad = TORCH[dtype], 9, 0.05, 771, lambda n: (n + 15) // 16 * 16
    dk, rp, tp = pad(dim), pad(rank), pad(rot)
    p = torch.cat([_packed(g, rows, heads, dim, dk), _packed(g, rows, heads, rot, tp), _packed(g, rows, 1, rank, rp), _packed(g, rows, 1, rot, tp),
                   torch.randn(rows, 8, generator=g)], 1).to(dt)
    w = torch.cat([1 + 0.4 * torch.randn(rank, generator=g), torch.zeros(rp - rank)])
    slots = torch.tensor([5, 64, 127, 0, 191, -1, 70, 33, 1], dtype=torch.int32)
    cache = torch.zeros(3, 1, 64, rp + tp, dtype=dt, device=device)
    q = torch.full((rows, heads, rp + tp), 5.0, dtype=dt, device=device)
    turn = O.yarn_rot(dims=rot)
    freqs, amp = RopeSpec(base=turn["base"], dims=rot, **turn["scaling"]).frequencies()
    positions = torch.arange(first, first + rows, dtype=torch.int32, device=device)
    table = ops.rope_angles(positions, ops.rope_frequencies(freqs, device), amp)
    at = heads * (dk + tp)
    mla_ops.latent_norm_kv(p.to(device), slots.to(device), cache, q, heads * dk, at, rank, rp, w.to(device), table, eps)
    lim = 2e-6 if dtype == "fp32" else 6e-3
    want = O.rotate_pairs(p[:, heads * dk: at].double().view(rows, heads, tp)[..., :rot], turn, first)
    close(q[..., rp: rp + rot], want, dtype, "rotated queries", lim)
    assert (q[..., :rp] == 5.0).all() and (q[..., rp + rot:] == 0).all()
    c = O.rms(p[:, at: at + rank].double(), eps) * w[:rank].double()
    k = O.rotate_pairs(p[:, None, at + rp: at + rp + rot].double(), turn, first)[:, 0]
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            close(cache[s // 64, :, s % 64, :rank], c[r: r + 1], dtype, "latent", lim)
            close(cache[s // 64, :, s % 64, rp: rp + rot], k[r: r + 1], dtype, "key", lim)
    assert int((cache != 0).any(-1).sum()) == 8 and (cache[..., rank:rp] == 0).all()


def _pointed(q0, ks, starts, qlen, ctx, key_of, group, width, gain):
    """Queries whose last row per sequence looks like the key at ``key_of(ctx)`` (where there is one)."""
    q = q0.clone()
    for b, c in enumerate(ctx):
        key = key_of(c)
        if 0 <= key < c:
            q[int(starts[b]) + qlen[b] - 1, :width] += (ks[b][:, key].float() * gain).repeat_interleave(group, 0).reshape(-1)
    return q


def _attend_rows(q, ks, vs, starts, qlen, hq, dk, scale, mask, cap=None, head_gate=None):
    want = []
    for b, n in enumerate(qlen):
        r = slice(int(starts[b]), int(starts[b]) + n)
        k, v = ks[b].transpose(0, 1), vs[b].transpose(0, 1)
        o = O.attend(q[r, : hq * dk].double().view(n, hq, dk), k, v, scale, O.visible(n, mask, k.shape[0] - n), cap)
        if head_gate is not None:
            o = o * torch.sigmoid(head_gate[r].double())[..., None]
        want.append(o.reshape(n, -1))
    return torch.cat(want)


@each_form
@pytest.mark.parametrize("dk,dv,hq,hkv", [(128, 128, 8, 2), (64, 32, 6, 2), (80, 112, 20, 1), (144, 160, 2, 1)])
@pytest.mark.parametrize("size,keep", [(1, 1), (50, 4), (64, 64), (65, 70), (33, 130), (1000, 3)])
def test_window_that_keeps_the_first_positions(device, dtype, dk, dv, hq, hkv, size, keep):
    """Prefill portions and decode rows; the last query of a sequence looks like the first key of its window, the key before it, the
    last kept position or the one after it in turn, so that leaving one out or letting one in shows."""
    dt, scale = TORCH[dtype], dk ** -0.5
    ctx, qlen = [300, 65, 128, 201, 51, 7, 1], [300, 2, 70, 150, 1, 7, 1]
    kc, vc, bt, ks, vs = paged(device, dt, hkv, dk, dv, ctx, seed=size + dk)
    q0 = torch.randn(sum(qlen), hq * dk + 16, generator=torch.Generator().manual_seed(3))
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    args = tuple(t.to(device) for t in (kc, vc, bt))
    last = [int(starts[b]) + n - 1 for b, n in enumerate(qlen)]
    lim = 2e-5 if dtype == "fp32" else 1.5e-2
    kw = dict(window=size, vdim=dv, keep=keep)
    for name, key_of in (("first inside", lambda c: c - size), ("last outside", lambda c: c - size - 1), ("last kept", lambda c: keep - 1),
                         ("first not kept", lambda c: keep)):
        q = _pointed(q0, ks, starts, qlen, ctx, key_of, hq // hkv, hq * dk, 2.0).to(dt)
        want = _attend_rows(q, ks, vs, starts, qlen, hq, dk, scale, {"size": size, "keep_first": keep})
        got = ops.attn_prefill(q.to(device), *args, starts.to(device), i32(qlen, device), i32(ctx, device), max(qlen), hq, hkv, dk, scale, **kw)
        close(got, want, dtype, f"prefill, {name}", lim)
        for split in (max(ctx), 64):
            got = ops.attn_decode(q[last].contiguous().to(device), *args, i32(ctx, device), hq, hkv, dk, scale, max_ctx=split, **kw)
            close(got, want[last], dtype, f"decode {split}, {name}", lim)
    if device == "cuda":
        ops.check_status()


@each_form
@pytest.mark.parametrize("dk,dv,hq,hkv", [(128, 128, 8, 2), (96, 48, 6, 3), (16, 112, 17, 1), (160, 144, 2, 1)])
@pytest.mark.parametrize("cap,gain", [(1.0, 4.0), (30.0, 4.0), (5.0, 60.0), (50.0, 0.01)])
def test_capped_scores(device, dtype, dk, dv, hq, hkv, cap, gain):
    """Scores far past the cap on both sides, around it, and so small that the cap does nothing."""
    dt, scale = TORCH[dtype], dk ** -0.5
    ctx, qlen = [200, 65, 128, 1], [200, 2, 70, 1]
    kc, vc, bt, ks, vs = paged(device, dt, hkv, dk, dv, ctx, seed=dk)
    q0 = gain * torch.randn(sum(qlen), hq * dk, generator=torch.Generator().manual_seed(3))
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    q = _pointed(q0, ks, starts, qlen, ctx, lambda c: c // 3, hq // hkv, hq * dk, 1.0).to(dt)
    want = _attend_rows(q, ks, vs, starts, qlen, hq, dk, scale, None, cap)
    args = tuple(t.to(device) for t in (kc, vc, bt))
    lim = 2e-5 if dtype == "fp32" else 1.5e-2
    kw = dict(vdim=dv, softcap=cap)
    got = ops.attn_prefill(q.to(device), *args, starts.to(device), i32(qlen, device), i32(ctx, device), max(qlen), hq, hkv, dk, scale, **kw)
    close(got, want, dtype, "prefill", lim)
    last = [int(starts[b]) + n - 1 for b, n in enumerate(qlen)]
    for split in (max(ctx), 64):
        got = ops.attn_decode(q[last].contiguous().to(device), *args, i32(ctx, device), hq, hkv, dk, scale, max_ctx=split, **kw)
        close(got, want[last], dtype, f"decode {split}", lim)
    # with a window that keeps first positions too
    mask = {"size": 40, "keep_first": 3}
    want = _attend_rows(q, ks, vs, starts, qlen, hq, dk, scale, mask, cap)
    kw.update(window=40, keep=3)
    got = ops.attn_prefill(q.to(device), *args, starts.to(device), i32(qlen, device), i32(ctx, device), max(qlen), hq, hkv, dk, scale, **kw)
    close(got, want, dtype, "prefill, window", lim)
    got = ops.attn_decode(q[last].contiguous().to(device), *args, i32(ctx, device), hq, hkv, dk, scale, **kw)
    close(got, want[last], dtype, "decode, window", lim)


@each_form
@pytest.mark.parametrize("rank,rot,heads", [(64, 16, 4), (16, 16, 1), (112, 16, 21), (128, 16, 3), (160, 48, 17), (512, 64, 16), (592, 32, 2)])
@pytest.mark.parametrize("size", [0, 1, 45, 64, 1000])
def test_latent_attention(device, dtype, rank, rot, heads, size):
    """Every kernel that serves a width: the value is the key row's first columns; a gate per head; the last query looks like the first
    key of its window or the key before it."""
    dt, width = TORCH[dtype], rank + rot
    scale = width ** -0.5
    ctx, qlen = [260, 65, 128, 201, 7, 1], [260, 2, 70, 1, 7, 1]
    kc, _, bt, ks, _ = paged(device, dt, 1, width, 16, ctx, seed=rank + size)
    vs = [k[..., :rank] for k in ks]
    g = torch.Generator().manual_seed(4)
    q0, gate = torch.randn(sum(qlen), heads * width, generator=g), (2 * torch.randn(sum(qlen), heads + 5, generator=g)).to(dt)
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    kc, bt = kc.to(device), bt.to(device)
    last = [int(starts[b]) + n - 1 for b, n in enumerate(qlen)]
    lim = 2e-5 if dtype == "fp32" else 1.5e-2
    hg = gate.to(device)[:, 3: 3 + heads]
    for back in (0, 1):
        q = _pointed(q0, ks, starts, qlen, ctx, lambda c: c - (size or c) - back, heads, heads * width, 2.0).to(dt)
        want = _attend_rows(q, ks, vs, starts, qlen, heads, width, scale, {"size": size} if size else None, None, gate[:, 3: 3 + heads])
        qd = q.to(device).view(-1, heads, width)
        got = mla_ops.latent_attention(qd, kc, bt, starts.to(device), i32(qlen, device), i32(ctx, device), max(qlen), max(ctx), scale, rank, size, hg)
        close(got, want, dtype, "prefill", lim)
        one = torch.ones(len(ctx), dtype=torch.int32, device=device)
        got = mla_ops.latent_attention(qd[last].contiguous(), kc, bt, i32(list(range(len(ctx))), device), one, i32(ctx, device), 1, max(ctx), scale, rank,
                                       size, hg[last], decode=True)
        close(got, want[last], dtype, "decode", lim)
    if device == "cuda":
        ops.check_status()


@GPU
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(4, 128, 64, 128, 512), (3, 32, 16, 48, 128), (17, 64, 32, 112, 160), (2, 80, 48, 16, 608)])
@pytest.mark.parametrize("size", [0, 1, 45, 64, 190])
def test_attention_over_expanded_latents(heads, dim, rot, vdim, rank, size):
    """Portions of several sequences at once, short ones beside long ones; the last query of a sequence looks like the first key of its window
    or the key before it."""
    bf, width, device = torch.bfloat16, rank + rot, "cuda"
    scale = (dim + rot) ** -0.5
    ctx, qlen = [260, 65, 128, 331, 7, 1], [260, 2, 70, 130, 7, 1]
    kc, _, bt, ks, _ = paged(device, bf, 1, width, 16, ctx, seed=rank + size)
    g = torch.Generator().manual_seed(4)
    n = sum(qlen)
    w_uk, w_uv = ((torch.randn(heads, d, rank, generator=g) / rank ** 0.5).to(bf) for d in (dim, vdim))
    p, q_full = torch.randn(n, heads * dim + 24, generator=g).to(bf), torch.randn(n, heads, width, generator=g).to(bf)
    q_full[..., :rank] = float("nan")                      # the absorbed queries are not there
    gate = (2 * torch.randn(n, heads + 5, generator=g)).to(bf)
    starts = torch.tensor([0] + qlen[:-1]).cumsum(0).to(torch.int32)
    keys, vals = [], []
    for k in ks:
        c, r = k[0, :, :rank], k[0, :, rank:]
        up = lambda w: torch.einsum("tr,hdr->htd", c, w.double()).to(bf).double()
        keys.append(torch.cat([up(w_uk), r.expand(heads, -1, -1)], -1))
        vals.append(up(w_uv))
    w_kv = torch.cat([w_uk.reshape(-1, rank), w_uv.reshape(-1, rank)]).to(device)
    pages = mla_ops.KeyPages.of(qlen, ctx, bt, size, 64, device)
    for back in (0, 1):
        q = torch.cat([p[:, : heads * dim].view(n, heads, dim), q_full[..., rank:]], -1).float()
        q = _pointed(q.view(n, -1), keys, starts, qlen, ctx, lambda c: c - (size or c) - back, 1, heads * (dim + rot), 1.0).to(bf).view(n, heads, -1)
        pd, qf = p.clone(), q_full.clone()
        pd[:, : heads * dim], qf[..., rank:] = q[..., :dim].reshape(n, -1), q[..., dim:]
        want = _attend_rows(q.reshape(n, -1), keys, vals, starts, qlen, heads, dim + rot, scale, {"size": size} if size else None, None, gate[:, 3: 3 + heads])
        out = torch.empty(n, heads * vdim, dtype=bf, device=device)
        mla_ops.expanded_attention(pd.to(device), qf.to(device), kc.to(device), w_kv, pages, bt.to(device), starts.to(device), i32(qlen, device),
                                   i32(ctx, device), max(qlen), dim, vdim, rank, scale, size, gate.to(device)[:, 3: 3 + heads], out)
        close(out, want, "bf16", f"back {back}", 2e-2)
    ops.check_status()


@GPU
def test_expanded_and_absorbed_forms_agree(tmp_path, monkeypatch):
    """The same prompt with its portions expanded and in the latent space; portions beside single tokens."""
    cfg = O.config([L(heads=4, kv_rank=200, rot_dim=32, dim=64, vdim=64, size=100), W(), L(heads=2, kv_rank=136, size=70), L(heads=3, kv_rank=136, rot_dim=20)])
    w = O.tensors(cfg, seed=15)
    e = load(write(tmp_path, cfg, w), "cuda", "bf16", capacity=512).engine
    a, b = ids(300, seed=90), ids(80, seed=91)
    wa, wb = O.forward(cfg, w, a)[0], O.forward(cfg, w, b)[0]
    asked = []
    real = mla_ops.expanded_attention
    monkeypatch.setattr(mla_ops, "expanded_attention", lambda *x, **k: (asked.append(1), real(*x, **k))[1])
    for least, limit in ((64, 1 << 16), (2, 1 << 16), (10 ** 6, 1 << 16), (64, 128)):
        monkeypatch.setattr(mla_ops, "EXPAND_MIN_ROWS", least)
        monkeypatch.setattr(mla_ops, "EXPAND_MAX_KEYS", limit)
        asked.clear()
        sa, sb, got = e.add_sequence(a[:130]), e.add_sequence(b[:79]), []
        got.append(e.feed([Span(sa, a[:130], list(range(130)))]))
        got.append(e.feed([Span(sb, b[:79], list(range(79))), Span(sa, a[130:131], [0])]))
        got.append(e.feed([Span(sa, a[131:290], list(range(159))), Span(sb, b[79:], [0])]))
        got.append(e.feed([Span(sa, a[290:], list(range(10)))]))
        agree(torch.cat([got[0], got[1][79:], got[2][:159], got[3]]), wa, "bf16", f"first request, {least}")
        agree(torch.cat([got[1][:79], got[2][159:]]), wb, "bf16", f"second request, {least}")
        assert len(asked) == {(64, 1 << 16): 9, (2, 1 << 16): 12, (10 ** 6, 1 << 16): 0, (64, 128): 3}[(least, limit)]
        for s in (sa, sb):
            e.free_sequence(s.seq_id)
    ops.check_status()


def test_key_pages_of_a_batch():
    table = torch.arange(40).view(4, 10)
    p = mla_ops.KeyPages.of([130, 1, 64, 10], [130, 300, 640, 70], table, 70, 64, "cpu")
    # the first query of the second sequence sits at 299 and sees from 230 on, that of the third at 576 from 507 on
    assert p.blocks.tolist() == [0, 1, 2, 13, 14, 27, 28, 29, 30, 31] and p.offsets.tolist() == [0, 0, -2, 8] and p.count == 10
    assert mla_ops.KeyPages.of([10], [640], table, 0, 64, "cpu").blocks.tolist() == list(range(10))


def test_mask_restatement():
    show = lambda m: [torch.nonzero(r).flatten().tolist() for r in m]
    assert show(O.visible(6, {"size": 2, "keep_first": 1})) == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5]]
    assert show(O.visible(2, {"size": 2}, 3)) == [[2, 3], [3, 4]] and show(O.visible(3, None)) == [[0], [0, 1], [0, 1, 2]]


# ------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------
class _Recorder:
    def __init__(self):
        self.got = {}

    def record(self, name, t):
        self.got[name] = t.detach().float().cpu()


@each_form
def test_whole_prompt_and_every_layer(base, device, dtype):
    path, w = base
    toks = ids(90, seed=2)
    want, after = O.forward(CFG, w, toks)
    m = load(path, device, dtype)
    m.engine.model.trace = rec = _Recorder()
    got, _ = feed_in_cuts(m.engine, toks, [90])
    agree(got, want, dtype, "logits")
    for i in range(len(LAYERS)):
        agree(rec.got[f"layer.{i}"], after[i], dtype, f"after layer {i}")


def test_every_mechanism_counts(base):
    """Each part, switched off in the restatement, changes what comes out."""
    _, w = base
    toks = ids(120, seed=2)
    want, _ = O.forward(CFG, w, toks)

    def without(layer, **mixer):
        l = dict(LAYERS[layer], mixer=dict(LAYERS[layer]["mixer"], **mixer))
        return O.forward(dict(CFG, layers=[l if i == layer else x for i, x in enumerate(LAYERS)]), w, toks)[0]
    other = [without(0, mask={"size": 50, "keep_first": 0}), without(0, mask={"size": 49, "keep_first": 3}), without(0, rot=dict(O.linear_rot(), scaling=None)),
             without(1, softcap=None), without(1, q_temp=None), without(2, mask={"size": 46}), without(2, rot=dict(O.yarn_rot(), scaling=None)),
             without(3, mask=None), O.forward(dict(CFG, token_side=None), w, toks)[0]]
    for i, o in enumerate(other):
        assert relative_change(o[60:], want[60:]).max() > 2e-3, i


def relative_change(a, b):
    return ((a - b) ** 2).mean(-1).sqrt() / (b ** 2).mean(-1).sqrt()


@each_form
@pytest.mark.parametrize("cuts", [[150, 1], [2], [64, 1], [63, 2, 64], [7, 50, 2, 1, 1, 80, 3], [1]])
def test_portions_and_decoding_equal_the_whole_prompt(base, device, dtype, cuts):
    path, w = base
    toks = ids(170, seed=3)
    want, _ = O.forward(CFG, w, toks)
    e = load(path, device, dtype).engine
    got, seq = feed_in_cuts(e, toks, cuts)
    agree(got, want, dtype, str(cuts))
    e.free_sequence(seq.seq_id)
    assert e.kv.alloc.free_blocks == e.kv.num_blocks


@each_form
def test_mixed_batches_equal_each_request_alone(base, device, dtype):
    path, w = base
    e = load(path, device, dtype, capacity=256, max_batch=4).engine
    lens = (150, 70, 40, 100)
    toks = [ids(n, seed=10 + i) for i, n in enumerate(lens)]
    want = [O.forward(CFG, w, t)[0] for t in toks]
    got = [[] for _ in lens]
    seqs, at = {}, [0] * 4
    plan = [(64, 2, 0, 0), (1, 30, 5, 0), (1, 0, 1, 63), (50, 1, 1, 1), (2, 1, 33, 2), (31, 36, 0, 33), (1, 0, 0, 1)]
    for sizes in plan:
        spans = []
        for i, n in enumerate(sizes):
            if n:
                part = toks[i][at[i]: at[i] + n]
                if i not in seqs:
                    seqs[i] = e.add_sequence(part)
                spans.append(Span(seqs[i], part, list(range(n))))
        out = e.feed(spans).float().cpu()
        row = 0
        for i, n in enumerate(sizes):
            got[i].append(out[row: row + n])
            row, at[i] = row + n, at[i] + n
    assert at == list(lens)
    for i in range(4):
        agree(torch.cat(got[i]), want[i], dtype, f"request {i}")


@each_form
def test_blocks_are_used_again(base, device, dtype):
    path, w = base
    e = load(path, device, dtype, capacity=128, max_batch=2, kv_tokens=256).engine
    kept, toks = e.add_sequence(ids(3, seed=20)), ids(100, seed=20)
    first, at = [], 0
    for turn in range(4):
        other = ids(70 + 11 * turn, seed=21 + turn)
        so = e.add_sequence(other)
        part = toks[at: at + 20]
        out = e.feed([Span(kept, part, list(range(len(part)))), Span(so, other, [len(other) - 1, 0])]).float().cpu()
        first.append(out[:20])
        want, _ = O.forward(CFG, w, other)
        agree(out[20:], want[[len(other) - 1, 0]], dtype, f"other {turn}")
        e.free_sequence(so.seq_id)
        at += 20
    agree(torch.cat(first), O.forward(CFG, w, toks[:80])[0], dtype, "kept")


def needle(kind, size=0, keep=0):
    """One layer in which token 7 is the key every query looks for. Channel 0 of every token is the direction of the queries, channel
    1 of token 7 alone that of its key, both on an element that does not turn."""
    dim, width = 32, 48
    layer = {"window": lambda: W(size=size, keep=keep, dim=dim, vdim=24, heads=2, kv_heads=1, scale=0.5, turn=O.linear_rot(dims=4), mlp=None),
             "latent": lambda: L(size=size, dim=dim, rot_dim=4, vdim=24, heads=2, kv_rank=40, scale=0.5, turn=O.yarn_rot(dims=4), mlp=None),
             "capped": lambda: C(dim=dim, vdim=24, heads=2, kv_heads=1, scale=0.5, softcap=12.0, coef=0.1, every=50, mlp=None)}[kind]()
    cfg = O.config([layer], width=width, vocab=64, scale=1.0, side=0)
    w = O.tensors(cfg, seed=4)
    w["embed"][:, 0], w["embed"][:, 1] = 3.0, 0.0
    w["embed"][7, 1] = 9.0
    n1, p = "l0.norm1", "l0.mix."
    w[n1], w[n1 + ".b"], w[n1 + ".alpha"] = torch.ones_like(w[n1]), torch.zeros_like(w[n1]), torch.full_like(w[n1 + ".alpha"], 0.5)
    w[p + "o"] = w[p + "o"] * 2.0
    if kind == "latent":
        q = w[p + "q"].view(2, dim + 4, width)
        q *= 0.2
        q[:, 31] = 0.0
        q[:, 31, 0] = 5.0
        w[p + "dkv"][39] = 0.0
        w[p + "dkv"][39, 1] = 12.0
        w[p + "dkv"][:39] *= 0.5
        w[p + "uk"] = w[p + "uk"] * 0.2
        uk = w[p + "uk"].view(2, dim, 40)
        uk[:, 31] = 0.0
        uk[:, 31, 39] = 3.0
        w[p + "dkv.norm"] = torch.ones_like(w[p + "dkv.norm"])
        return cfg, w
    for name, heads, channel in (("q", 2, 0), ("k", 1, 1)):
        m = w[p + name].view(heads, dim, width)
        m *= 0.2
        m[:, 31] = 0.0
        m[:, 31, channel] = 5.0
        w[p + name + ".b"] = w[p + name + ".b"] * 0.1
        w[p + name + ".b"].view(heads, dim)[:, 31] = 0.0
        w[p + name + ".norm"] = torch.ones_like(w[p + name + ".norm"])
    return cfg, w


@each_form
@pytest.mark.parametrize("kind,size,keep", [("window", 1, 0), ("window", 2, 1), ("window", 48, 2), ("window", 64, 64), ("window", 100, 5), ("window", 20, 70),
                                            ("latent", 1, 0), ("latent", 40, 0), ("latent", 64, 0)])
def test_far_keys_window_edges_and_first_positions(tmp_path, device, dtype, kind, size, keep):
    """A key that takes much of the weight while it is seen: at the first positions, the last kept one and the next, at page
    edges; queries just inside and just outside the window, in a prompt and decoded."""
    cfg, w = needle(kind, size, keep)
    path = write(tmp_path, cfg, w)
    n = max(2 * size + 20, keep + 40, 90)
    plain = [t if t != 7 else 8 for t in ids(n, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    e = load(path, device, dtype).engine
    other = {}
    for at in sorted({0, 1, keep, max(keep - 1, 0), min(size, n - 1), 63, 64}):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved, end = relative_change(want, without), n if at < keep else at + size
        assert moved[at: end].min() > 0.03 and (moved[end:] == 0).all() and (moved[:at] == 0).all()
        for cuts in ([n], [min(max(at + size - 3, 1), n - 1), 1]):                  # the window's end in the prompt, and decoded
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")
            # rows that do not see the needle do not know of it at all
            if tuple(cuts) not in other:
                other[tuple(cuts)], seq = feed_in_cuts(e, plain, cuts)
                e.free_sequence(seq.seq_id)
            assert torch.equal(other[tuple(cuts)][end:], got[end:])


@each_form
def test_full_attention_sees_a_far_key(tmp_path, device, dtype):
    cfg, w = needle("capped")
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    n = 260
    plain = [t if t != 7 else 8 for t in ids(n, vocab=64, seed=6)]
    without, _ = O.forward(cfg, w, plain)
    for at in (0, 63, 64, 130):
        toks = list(plain)
        toks[at] = 7
        want, _ = O.forward(cfg, w, toks)
        moved = relative_change(want, without)
        assert moved[at:].min() > 0.03 and (moved[:at] == 0).all()
        for cuts in ([n], [at + 1, 2, 64, 65, 1], [100, 100, 30, 1]):
            got, seq = feed_in_cuts(e, toks, cuts)
            e.free_sequence(seq.seq_id)
            agree(got, want, dtype, f"needle at {at}, cuts {cuts}")


SIZES = {
    "every constant one": O.config([W(heads=2, kv_heads=2, scale=1.0, size=9, turn=O.linear_rot(factor=1.0)), C(heads=1, kv_heads=1, scale=1.0, softcap=1.0, coef=1.0, every=1),
                                    L(heads=1, scale=1.0, turn=O.yarn_rot(factor=1.0))], scale=1.0, mult=1.0, logit_scale=1.0),
    "tensor-core widths": O.config([W(heads=4, kv_heads=1, dim=128, vdim=128, scale=128 ** -0.5, size=96, keep=70, turn=O.linear_rot(dims=128)),
                                    C(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.1, mlp={"kind": "dense", "ff": 256}),
                                    L(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=96, size=70)], width=256, vocab=512, side=64),
    "odd sizes": O.config([W(heads=3, kv_heads=3, dim=20, vdim=28, size=29, keep=1, turn=O.linear_rot(dims=6), mlp={"kind": "dense", "ff": 33}),
                           C(heads=9, kv_heads=3, dim=12, vdim=28, every=7), L(heads=5, dim=12, rot_dim=6, vdim=20, kv_rank=36, size=31)],
                          width=75, vocab=131, side=5),
    "wide heads": O.config([W(heads=2, kv_heads=1, dim=144, vdim=200, size=70, scale=0.1), C(heads=2, kv_heads=2, dim=136, vdim=32, scale=0.1)]),
    "wide latents": O.config([L(heads=3, kv_rank=120, rot_dim=24), L(heads=2, kv_rank=512, rot_dim=64, dim=16, vdim=16, size=90), L(heads=1, kv_rank=600)]),
    "one token windows": O.config([W(heads=1, kv_heads=1, dim=16, vdim=16, size=1, keep=0), L(size=1), W(size=1, keep=1), W(size=100000, keep=9)]),
    "kept positions fill pages": O.config([W(size=5, keep=64), W(size=40, keep=129), W(size=20, keep=65, kv_from=1)]),
    "shared keys of both kinds": O.config([C(), W(), dict(C(heads=6), mixer=dict(C(heads=6)["mixer"], kv_from=0)), W(kv_from=1, heads=2, keep=0),
                                           W(kv_from=1, size=9, heads=8, scale=0.4)]),
    "no cap, no temperature, no scaling": O.config([dict(C(), mixer={k: v for k, v in C()["mixer"].items() if k not in ("softcap", "q_temp")}),
                                                    W(turn=dict(O.linear_rot(), scaling=None)), L(turn=dict(O.yarn_rot(), scaling=None))], eps=0.2),
    "no masks": O.config([dict(W(), mixer={k: v for k, v in W()["mixer"].items() if k != "mask"}), dict(L(), mixer={k: v for k, v in L()["mixer"].items() if k != "mask"})]),
    "no token input": O.config([W(), L(mlp=None), C(mlp=None)], side=0),
    "latents only": O.config([L(), L(heads=20, dim=16, rot_dim=2, kv_rank=8), L(mlp=None)], side=300),
    "no feed-forward": O.config([W(mlp=None), C(mlp=None), L(mlp=None)]),
}


@each_form
@pytest.mark.parametrize("name", sorted(SIZES))
def test_other_sizes(tmp_path, device, dtype, name):
    cfg = SIZES[name]
    w = O.tensors(cfg, seed=5)
    e = load(write(tmp_path, cfg, w), device, dtype).engine
    toks = ids(155, vocab=cfg["vocab"], seed=8)
    want, _ = O.forward(cfg, w, toks)
    for cuts in ([155], [70, 1, 1, 2, 70, 1]):
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


@each_form
def test_prefix_cache_and_verification(base, tmp_path, device, dtype):
    path, w = base
    m = load(path, device, dtype, prefix_cache=True, runtime_dir=str(tmp_path))
    p = ids(90, seed=70)
    m.prefill(p[:70])
    first = m.prefill(p)
    assert m.prefix_store().hits == 1
    greedy_agrees(w, p, [first], dtype)
    m.reset()
    s = m.engine.add_sequence(p[:60])
    m.engine.prefill([s])
    s.pending = p[60]
    got = m.engine.verify([s], [p[61:64]])[0]
    lg = O.forward(CFG, w, p[:64])[0][60:]
    for row, t in zip(lg, got):
        assert row.max() - row[t] <= 0.12 * row.std()
    with pytest.raises(ValueError):
        load(path, device, dtype, kv_format="affine8")


# ------------------------------------------------------------------------------------------
# configuration, checkpoint, command line, runner
# ------------------------------------------------------------------------------------------
def test_configuration_is_read_and_checked(base):
    path, _ = base
    s = read_model_spec(path)
    assert (s.arch, s.layers, s.hidden, s.vocab, s.side_dim) == ("kabavik", 6, 104, 198, 20) and s.runs == list(range(6))
    assert s.kv_geometry() == [(2, 48, 32), (2, 48, 32), (1, 64 + 16, 0), (0, 0, 0), (3, 16, 32), (6, 48, 48)]
    assert [l.window for l in s.layer_specs] == [50, 0, 45, 37, 0, 64] and [l.keep_first for l in s.layer_specs] == [3, 0, 0, 5, 0, 0]
    assert [l.kv_from for l in s.layer_specs] == [-1, -1, -1, 0, -1, -1] and s.layer_specs[4].ffn == 0 and s.layer_specs[1].q_temp == (0.4, 37)
    assert s.layer_specs[1].softcap == 5.0 and s.layer_specs[1].rope is None and s.layer_specs[0].qk_norm == "row"
    for i, n in ((0, 130), (3, 40), (3, 43), (2, 60), (1, 20), (3, 3)):
        l = s.layer_specs[i]
        see = O.visible(n, LAYERS[i]["mixer"].get("mask"))
        assert l.pairs_seen(n) == int(see.sum()) and l.keys_seen(n) == int(see[-1].sum())
    assert s.layer_specs[0].rope == RopeSpec(base=4000.0, dims=12, factor=3.0, halves=True)
    assert s.layer_specs[2].rope == RopeSpec(base=700.0, dims=8, factor=6.0, original=200, fast=24.0, slow=1.5)
    weights = {n: t for n, t in O.tensors(CFG).items() if t.dim() == 2 and n not in ("embed", "head")}
    assert sum(t.numel() for t in weights.values()) == s.dense_param_count() - 2 * s.vocab * s.hidden
    bad = lambda l: spec_from_hf_config(dict(CFG, layers=[W(), l]))
    bad(W(kv_from=0))
    for l in (dict(W(), type="recurrence"), W(mlp={"kind": "moe"}), W(heads=3), W(scale=0.0), W(turn=O.linear_rot(dims=7)), W(turn=O.linear_rot(dims=42)),
              C(every=0), L(turn=O.yarn_rot(dims=12)), W(kv_from=1), W(kv_from=0, dim=32), W(kv_from=0, kv_heads=3), W(kv_from=5),
              dict(C(), mixer=dict(C()["mixer"], kv_from=0))):
        with pytest.raises(ConfigError):
            bad(l)
    with pytest.raises(ConfigError):
        spec_from_hf_config(dict(CFG, layers=[W(), W(kv_from=0), W(kv_from=1)]))
    with pytest.raises(ConfigError):
        spec_from_hf_config(dict(CFG, layers=[]))


def test_checkpoint_is_audited(tmp_path):
    w = O.tensors(CFG)
    changes = (("l1.mix.q.b", None), (None, ("l3.mlp.e0.gate", torch.zeros(2, 2))), ("l0.mix.q.norm", ("l0.mix.q.norm", torch.zeros(40))),
               ("l5.norm2b.alpha", None), ("side.embed", None), ("l2.mix.uk", None), ("l4.side.norm", None))
    for i, (drop, put) in enumerate(changes):
        t = {n: x for n, x in w.items() if n != drop}
        if put:
            t[put[0]] = put[1].to(torch.bfloat16)
        with pytest.raises(CheckpointError):
            load(write(tmp_path, CFG, t, f"m{i}"), "cpu", "bf16")
    # tensors of a part the configuration switches off may be there
    more = {"l4.norm2": w["l4.norm1"].clone(), "l4.norm2b.alpha": w["l4.norm1.alpha"].clone(), "l3.mix.k.b": w["l0.mix.k.b"].clone(),
            "l3.mix.v": w["l0.mix.v"].clone()}
    load(write(tmp_path, CFG, dict(w, **more), "more"), "cpu", "bf16")


def test_planner_counts_what_a_layer_caches():
    from flyingfish_b200.planner.plan import DeviceInfo, plan_memory
    s = named_shape("kabavik-tiny")
    info = DeviceInfo(name="x", total_bytes=1 << 30, free_bytes=1 << 30)
    p = plan_memory(s, Settings(capacity=256, max_batch=2, kv_tokens=1000), info, 0)
    assert s.kv_geometry()[1] == (1, 64, 0) and s.kv_geometry()[3] == (0, 0, 0)
    assert p.kv_blocks == 16 and p.kv_bytes == 16 * 64 * 2 * sum(h * (a + b) for h, a, b in s.kv_geometry())


def test_calibration_lists_every_projection():
    from flyingfish_b200.planner.calibrate import decode_linear_shapes
    shapes = {(n, k, epi) for _, n, k, epi in decode_linear_shapes(spec_from_hf_config(CFG))}
    assert (256, 104, 1) in shapes and (104, 128, 0) in shapes and (2 * 48, 104, 0) in shapes


def test_command_line_generates(base, capsys):
    from flyingfish_b200.cli import main
    path, w = base
    p = ids(12, seed=80)
    assert main(["--model", path, "--cpu", "--dtype", "fp32", "--kv-tokens", "256", "--capacity", "128", "generate", "--tokens",
                 ",".join(map(str, p)), "--max-new-tokens", "6", "--ignore-eos"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    greedy_agrees(w, p, out["generated_ids"], "fp32")
    assert main(["--model", path, "inspect"]) == 0
    assert json.loads(capsys.readouterr().out)["spec"]["arch"] == "kabavik"


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
    from flyingfish_b200.serve.trace_runner import TraceRunner, load_engine
    path, w = base
    m, e = load_engine(path, dtype, 192, device)
    assert e.kv.num_blocks == 3
    r = TraceRunner(e, m.spec.vocab)
    toks, steps = _trace()
    want = _trace_wants(w, toks)
    for s in steps:
        out = r.step(s["entries"], s["end"])
        if s["step"] in want:
            agree(out, want[s["step"]], dtype, f"step {s['step']}")
        else:
            assert out is None
    assert not r.live and e.kv.alloc.free_blocks == 3


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
    m = Model.load("kabavik-tiny", Settings(capacity=128, max_batch=2), device="cpu", seed=3)
    out = m.generate_batch([[1, 2, 3], [4] * 50], 5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 512 for o in out for t in o)
    assert dataclasses.asdict(m.spec)["layer_specs"][3]["kv_from"] == 0


@GPU
def test_random_shape_gpu_matches_cpu():
    from _oracle import assert_tokens_equal_up_to_ties
    st = Settings(capacity=256, max_batch=2)
    cpu, gpu = (Model.load("kabavik-tiny", st, device=d, seed=3) for d in ("cpu", "cuda"))
    prompts = [ids(80, 512, 1), ids(9, 512, 2)]
    for p, a, b in zip(prompts, cpu.generate_batch(prompts, 12), gpu.generate_batch(prompts, 12)):
        assert_tokens_equal_up_to_ties(cpu, p, a, b)
    ops.check_status()
