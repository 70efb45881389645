"""Kabavik decoder: sub-layers normed on both sides by a hyperbolic tangent, three kinds of attention, gated feed-forwards and a
token input per layer, all on an FP32 residual.

    x <- x + m after1(mixer(before1(x)))         before / after: tanh(alpha x) w + b
    x <- x + m after2(ff(before2(x)))
    x <- x + m rms(P (gelu(G x) * e)) w          e: the layer's part of the token's row in a table of its own

* Windowed attention: q and k are normed over their whole projections and the first elements of every head rotate (elements i and
  i + half); a query sees its last ``window`` positions and the first ``keep_first`` of the sequence. A layer may read the keys and
  values another layer cached; it then projects queries alone.
* Full attention: q and k are normed per head, nothing rotates, the query grows with the logarithm of its position, scores are capped.
* Latent attention: a token caches its normed latent and one rotated key part. Decoded tokens and narrow latents take the absorbed form:
  a head's query goes through its key matrix into the latent space (``ops.head_linear``), all heads attend to the one cached row, and
  the result leaves through the head's value matrix. Portions over wide latents expand the visible rows to keys and values first
  (``mla_ops.expanded_attention``). A head's result is multiplied by a gate that the attention kernels apply.
* The norm behind a sub-layer, the sum and the norm in front of the next one are one kernel (``ops.residual_ops.add_normed``); the residual
  factor is part of the weights of the norms behind, the logits' factor of the final norm. The feed-forward's activation and the
  token input's activation and product are GEMM epilogues.

A batch may hold portions of prompts and single decoded tokens together (``mixed_batches``): the single tokens stand behind the
portions and take the decode kernels. Sizes that are not multiples of the kernels' vectors are padded here, once, with zeros.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import LayerSpec, ModelSpec, pad_to
from ..ops import mla_ops, ref, residual_ops
from ..ops.residual_ops import Norm
from .decoder import DecoderModel
from .weights import DTYPES, LayerWeights, ModelWeights, TensorSource, TPInfo, pad_cols, pad_heads, pad_rows, random_tensor


# ------------------------------------------------------------------------------------------
# weights
# ------------------------------------------------------------------------------------------
def _norm_names(l: LayerSpec) -> tuple[str, ...]:
    return ("norm1", "norm1b") + (("norm2", "norm2b") if l.ffn else ())


def _mixer_tensors(l: LayerSpec, p: str, h: int, every: bool = False) -> dict[str, tuple[int, ...]]:
    """``every``: with the keys and values of a layer that takes another layer's."""
    o = l.heads * l.vdim
    if l.mixer == "latent":
        return {p + "q": (l.heads * (l.dim + l.rot_dim), h), p + "dkv": (l.kv_rank + l.rot_dim, h), p + "dkv.norm": (l.kv_rank,),
                p + "uk": (l.heads * l.dim, l.kv_rank), p + "uv": (o, l.kv_rank), p + "g": (l.heads, h), p + "o": (h, o)}
    q, k, v = l.heads * l.dim, l.kv_heads * l.dim, l.kv_heads * l.vdim
    whole = l.qk_norm == "row"
    m = {p + "q": (q, h), p + "q.b": (q,), p + "q.norm": (q if whole else l.dim,), p + "o": (h, o), p + "o.b": (h,)}
    if l.kv_from < 0 or every:
        m.update({p + "k": (k, h), p + "k.b": (k,), p + "k.norm": (k if whole else l.dim,), p + "v": (v, h), p + "v.b": (v,)})
    return m


def expected_tensors(spec: ModelSpec) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor names and shapes. Layer i's tensors start with ``l<i>.``; a norm has a weight, a vector ``.b`` and a scalar
    ``.alpha``."""
    h, side = spec.hidden, spec.side_dim
    m: dict[str, tuple[int, ...]] = {"embed": (spec.vocab, h), "head": (spec.vocab, h)}
    if side:
        m["side.embed"] = (spec.vocab, len(spec.layer_specs) * side)
    norms = ["final.norm"]
    for i, l in enumerate(spec.layer_specs):
        p = f"l{i}."
        norms += [p + n for n in _norm_names(l)]
        m.update(_mixer_tensors(l, p + "mix.", h))
        if l.ffn:
            m.update({p + "mlp.gate": (l.ffn, h), p + "mlp.up": (l.ffn, h), p + "mlp.down": (h, l.ffn)})
        if side:
            m.update({p + "side.gate": (side, h), p + "side.proj": (h, side), p + "side.norm": (h,)})
    for n in norms:
        m.update({n: (h,), n + ".b": (h,), n + ".alpha": ()})
    return m


def unused_tensors(spec: ModelSpec) -> tuple[str, ...]:
    """Tensors of parts a layer's configuration switches off: a checkpoint may carry them, nothing reads them."""
    names: list[str] = []
    for i, l in enumerate(spec.layer_specs):
        if not l.ffn:
            names += [f"l{i}.{n}{leaf}" for n in ("norm2", "norm2b") for leaf in ("", ".b", ".alpha")]
        if l.kv_from >= 0:
            own = _mixer_tensors(l, f"l{i}.mix.", spec.hidden)
            names += [n for n in _mixer_tensors(l, f"l{i}.mix.", spec.hidden, every=True) if n not in own]
    return tuple(names)


def build_weights(spec: ModelSpec, source: TensorSource) -> ModelWeights:
    """Fused and padded weights. ``wqkv`` = [q | k | v] with one bias vector (layers that share keys and values: q) or, for latent
    attention, [unrotated queries | rotated queries | latent | rotated key | gates]; heads padded to 16 elements. Norms are FP32,
    the residual factor multiplied into those behind a sub-layer and the logits' factor into the final one."""
    cfg = spec.extra["kabavik"]
    shapes = expected_tensors(spec)
    get = lambda n: source(n, shapes[n])
    h, wp, sp = spec.hidden, pad_to(spec.hidden, 8), pad_to(spec.side_dim, 8)
    mult = float(cfg["residual_mult"])
    vec = lambda n, f=1.0: (pad_cols(get(n).float(), wp) * f).contiguous()
    norm = lambda n, f=1.0: Norm("tanh", vec(n, f), vec(n + ".b", f), float(get(n + ".alpha")))
    rows_in = lambda n, *heads: pad_heads(pad_cols(get(n), wp), *heads)
    layers = []
    for i, l in enumerate(spec.layer_specs):
        p, dk, dv = f"l{i}.mix.", l.dim_pad, l.vdim_pad
        lw = LayerWeights()
        lw.extra["norms"] = {n: norm(f"l{i}.{n}", mult if n.endswith("b") else 1.0) for n in _norm_names(l)}
        lw.wo = pad_rows(pad_heads(get(p + "o").t().contiguous(), l.heads, l.vdim, dv).t(), wp).contiguous()
        if l.mixer == "latent":
            rp, tp, d = l.rank_pad, l.rot_pad, l.dim + l.rot_dim
            q = pad_cols(get(p + "q"), wp).view(l.heads, d, wp)
            down = pad_cols(get(p + "dkv"), wp)
            lw.wqkv = torch.cat([pad_heads(q[:, : l.dim].reshape(-1, wp), l.heads, l.dim, dk),
                                 pad_heads(q[:, l.dim:].reshape(-1, wp), l.heads, l.rot_dim, tp),
                                 pad_rows(down[: l.kv_rank], rp), pad_rows(down[l.kv_rank:], tp),
                                 pad_rows(pad_cols(get(p + "g"), wp), pad_to(l.heads, 8))]).contiguous()
            lw.extra["latent_norm"] = pad_cols(get(p + "dkv.norm").float(), rp).contiguous()
            # all key matrices, then all value matrices; a head's unrotated query goes into the latent space through [rank_pad, dim_pad]
            # and its result out of it through [vdim_pad, rank_pad]
            up = pad_heads(pad_cols(get(p + "uk"), rp), l.heads, l.dim, dk)
            lw.extra["w_kv"] = torch.cat([up, pad_heads(pad_cols(get(p + "uv"), rp), l.heads, l.vdim, dv)]).contiguous()
            lw.extra["w_uk"] = up.view(l.heads, dk, rp).transpose(1, 2).contiguous()
        else:
            parts = [("q", l.heads, l.dim, dk)] + ([("k", l.kv_heads, l.dim, dk), ("v", l.kv_heads, l.vdim, dv)] if l.kv_from < 0 else [])
            lw.wqkv = torch.cat([rows_in(p + n, *s) for n, *s in parts]).contiguous()
            lw.extra["bqkv"] = torch.cat([pad_heads(get(p + n + ".b"), *s) for n, *s in parts]).contiguous()
            lw.extra["bo"] = pad_cols(get(p + "o.b"), wp)
            wide = (lambda n, heads: pad_heads(get(n).float(), heads, l.dim, dk)) if l.qk_norm == "row" else (lambda n, heads: pad_cols(get(n).float(), dk))
            lw.q_norm = wide(p + "q.norm", l.heads)
            lw.k_norm = wide(p + "k.norm", l.kv_heads) if l.kv_from < 0 else None
        if l.ffn:
            p, fp = f"l{i}.mlp.", pad_to(l.ffn, 128)
            lw.wgu = ref.interleave_gate_up(*(pad_rows(pad_cols(get(p + n), wp), fp) for n in ("gate", "up")))
            lw.wdown = pad_rows(pad_cols(get(p + "down"), fp), wp).contiguous()
        if sp:
            p = f"l{i}.side."
            lw.extra["side_gate"] = pad_rows(pad_cols(get(p + "gate"), wp), sp).contiguous()
            lw.extra["side_proj"] = pad_rows(pad_cols(get(p + "proj"), sp), wp).contiguous()
            lw.extra["norms"]["side"] = Norm("rms", vec(p + "norm", mult))
        layers.append(lw)
    w = ModelWeights(spec=spec, embed=pad_cols(get("embed"), wp).contiguous(), final_norm=norm("final.norm", float(cfg["logit_scale"])),
                     lm_head=pad_rows(pad_cols(get("head"), wp), pad_to(spec.vocab, 8)).contiguous(), layers=layers, tp=TPInfo(),
                     vocab_shard=(0, spec.vocab))
    if sp:
        n = len(spec.layer_specs)
        w.extra["side_embed"] = pad_cols(get("side.embed").view(spec.vocab, n, spec.side_dim), sp).reshape(spec.vocab, n * sp).contiguous()
    return w


def random_weights(spec: ModelSpec, seed: int, device: torch.device | str) -> ModelWeights:
    """Seeded weights in which every mechanism counts."""
    device = torch.device(device)
    dtype = DTYPES[spec.dtype]

    def source(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        leaf = name.rsplit(".", 1)[-1]
        if len(shape) < 2:
            t = random_tensor(seed, name, shape, torch.float32, device, std=0.2)
            return (t if leaf == "b" else 0.7 + 0.5 * t if leaf == "alpha" else 1.0 + t).to(dtype)
        return random_tensor(seed, name, shape, dtype, device, std=1.0 if leaf == "embed" else shape[1] ** -0.5)
    return build_weights(spec, source)


# ------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------
COPY = Norm()


class KabavikModel(DecoderModel):
    mixed_batches = True               # prompt portions and single decoded tokens in one forward

    def __init__(self, weights: ModelWeights, comm=None, trace=None):
        super().__init__(weights, comm=comm, trace=trace)
        assert weights.tp.size == 1, "the Kabavik layout is served on one GPU per replica"
        spec, dev = self.spec, weights.embed.device
        self.embed_scale, self.width = float(spec.extra["kabavik"]["embed_scale"]), spec.hidden
        # rotations, one table per step for all layers that share one
        self.rotations: list[tuple[torch.Tensor, float]] = []
        self.rotation_of: list[int] = []
        known: list = []
        for l in spec.layer_specs:
            if l.rope is None:
                self.rotation_of.append(-1)
                continue
            freqs, amp = l.rope.frequencies()
            if (freqs, amp) not in known:
                known.append((freqs, amp))
                self.rotations.append((ops.rope_frequencies(freqs, dev), amp))
            self.rotation_of.append(known.index((freqs, amp)))

    # -- mixers ------------------------------------------------------------------------------
    @staticmethod
    def _split(b) -> tuple[int, int]:
        """(sequences with a portion, rows of theirs); what stands behind them takes the decode kernels."""
        if b.is_decode:
            return 0, 0
        return b.batch - b.singles, b.rows - b.singles

    def _attention_layer(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b, kv, table) -> torch.Tensor:
        dk, dv = l.dim_pad, l.vdim_pad
        src, own = (i, l.kv_heads) if l.kv_from < 0 else (l.kv_from, 0)
        k, v = kv.k[src], kv.v[src]
        qkv = ops.linear(n, lw.wqkv, bias=lw.extra["bqkv"])
        ops.head_norm_kv(qkv, b.slots, k if own else None, v if own else None, l.heads, own, l.dim, l.vdim, self.spec.rms_eps, q_weight=lw.q_norm,
                         k_weight=lw.k_norm, cos_sin=table, whole=l.qk_norm == "row", halves=table is not None and l.rope.halves,
                         temp=None if l.q_temp is None else (b.positions, *l.q_temp))
        out = torch.empty(b.rows, l.heads * dv, dtype=qkv.dtype, device=qkv.device)
        kw = dict(window=l.window, vdim=dv, keep=l.keep_first, softcap=l.softcap)
        s, rows = self._split(b)
        if s:
            ops.attn_prefill(qkv[:rows], k, v, b.block_table[:s], b.q_start[:s], b.q_lens[:s], b.ctx_lens[:s], b.max_q_len, l.heads,
                             l.kv_heads, dk, l.scale, out=out[:rows], **kw)
        if s < b.batch:
            bs = kv.block_size
            reach = min(b.max_ctx, l.window + bs + pad_to(l.keep_first, bs)) if l.window else b.max_ctx
            ops.attn_decode(qkv[rows:], k, v, b.block_table[s:], b.ctx_lens[s:], l.heads, l.kv_heads, dk, l.scale,
                            nq=b.nq if b.is_decode else 1, max_ctx=reach, out=out[rows:], **kw)
        return out

    def _latent_layer(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b, kv, table) -> torch.Tensor:
        dk, dv, rp, tp = l.dim_pad, l.vdim_pad, l.rank_pad, l.rot_pad
        p = ops.linear(n, lw.wqkv)
        rot, lat = l.heads * dk, l.heads * (dk + tp)
        q = torch.empty(b.rows, l.heads, rp + tp, dtype=p.dtype, device=p.device)
        mla_ops.latent_norm_kv(p, b.slots, kv.k[i], q, rot, lat, l.kv_rank, rp, lw.extra["latent_norm"], table, self.spec.rms_eps)
        gate = p[:, lat + rp + tp: lat + rp + tp + l.heads]
        out = torch.empty(b.rows, l.heads * dv, dtype=p.dtype, device=p.device)
        s, rows = self._split(b)
        pages = self._key_pages(b, s, l.window, kv) if s and mla_ops.expands(p, rp + tp, dk, tp, dv, b.max_q_len) else None
        first = 0                                                     # first row of the absorbed form
        if pages is not None:
            mla_ops.expanded_attention(p[:rows, :rot], q[:rows], kv.k[i], lw.extra["w_kv"], pages, b.block_table[:s], b.q_start[:s], b.q_lens[:s],
                                       b.ctx_lens[:s], b.max_q_len, dk, dv, rp, l.scale, l.window, gate[:rows], out[:rows])
            first = rows
        if first == b.rows:
            return out
        ops.head_linear(p[first:, :rot], lw.extra["w_uk"], out=q[first:].view(b.rows - first, -1), out_cols=rp + tp)
        a = torch.empty(b.rows - first, l.heads * rp, dtype=p.dtype, device=p.device)
        if s and pages is None:
            mla_ops.latent_attention(q[:rows], kv.k[i], b.block_table[:s], b.q_start[:s], b.q_lens[:s], b.ctx_lens[:s], b.max_q_len, b.max_ctx, l.scale,
                                     rp, l.window, gate[:rows], a[:rows])
        if s < b.batch:
            starts = b.q_start if b.is_decode else b.q_start[s:] - rows
            mla_ops.latent_attention(q[rows:], kv.k[i], b.block_table[s:], starts, b.q_lens[s:], b.ctx_lens[s:], b.nq if b.is_decode else 1,
                                     b.max_ctx, l.scale, rp, l.window, gate[rows:], a[rows - first:], decode=True)
        ops.head_linear(a, lw.extra["w_kv"][l.heads * dk:].view(l.heads, dv, rp), out=out[first:])
        return out

    def _key_pages(self, b, s: int, window: int, kv):
        """Pages the portions of this step see through ``window`` (one list for all layers with that window)."""
        if window not in self._pages:
            L, h = b.layout, b.host
            table = h[L.block_table: L.block_table + L.max_batch * L.max_blocks].view(L.max_batch, L.max_blocks)[:s]
            self._pages[window] = mla_ops.KeyPages.of(h[L.q_lens: L.q_lens + s].tolist(), h[L.ctx_lens: L.ctx_lens + s].tolist(), table, window,
                                                      kv.block_size, b.device)
        return self._pages[window]

    # -- forward -----------------------------------------------------------------------------
    def hidden_states(self, b, kv, inputs_embeds=None):
        assert inputs_embeds is None, "the Kabavik model takes token ids"
        assert b.tree_mask is None, "tree verification is not available with capped scores or latent attention"
        w, spec, eps = self.w, self.spec, self.spec.rms_eps
        side, sp = w.extra.get("side_embed"), pad_to(spec.side_dim, 8)
        self._pages = {}                                              # expanded pages of this step, per window
        tables = [ops.rope_angles(b.positions, f, amp) for f, amp in self.rotations]
        norms = [lw.extra["norms"] for lw in w.layers]
        add = lambda y, behind, front: residual_ops.add_normed(x, y, behind, front, eps, self.width)
        x, n = residual_ops.embed_normed(b.ids, w.embed, self.embed_scale, norms[0]["norm1"], eps, self.width)
        for i, l in enumerate(spec.layer_specs):
            lw = w.layers[i]
            mixer = self._latent_layer if l.mixer == "latent" else self._attention_layer
            a = mixer(i, l, lw, n, b, kv, tables[self.rotation_of[i]] if l.rope is not None else None)
            if self.trace is not None:
                self.trace.record(f"layer.{i}.attn", a)
            y, behind = ops.linear(a, lw.wo, bias=lw.extra.get("bo")), norms[i]["norm1b"]
            if l.ffn:
                n = add(y, behind, norms[i]["norm2"])
                y, behind = ops.linear(ops.linear_swiglu(n, lw.wgu, mode=3), lw.wdown), norms[i]["norm2b"]
            if side is not None:
                z = add(y, behind, COPY)
                g = ops.linear(z, lw.extra["side_gate"], act="gelu_tanh", mul=(side[:, i * sp: (i + 1) * sp], b.ids))
                y, behind = ops.linear(g, lw.extra["side_proj"]), norms[i]["side"]
            n = add(y, behind, norms[i + 1]["norm1"] if i + 1 < spec.layers else w.final_norm)
            if self.trace is not None:
                self.trace.record(f"layer.{i}", x[:, : self.width].clone())
        self.last_residual = None
        if self.normed_sink is not None:
            self.normed_sink.append(n)
        return n

    def logits(self, n, b):
        """FP32."""
        sel = n.index_select(0, b.logit_rows.long()) if b.n_logit_rows != n.shape[0] else n
        return ops.linear(sel.contiguous(), self.w.lm_head, out_dtype=torch.float32)[:, : self.spec.vocab]


def build_model(weights: ModelWeights, settings, comm=None) -> KabavikModel:
    return KabavikModel(weights, comm=comm)
