"""Duponex decoder: several residual streams with fixed hyper-connections, block-local attention without positions, value
mixing across layers, and a squared-ReLU feed-forward.

A token carries ``S`` FP32 residual streams X_1..X_S, all equal to the scaled embedding at first. Every sub-layer f (the
attention, then the feed-forward where the layer has one) owns a read vector a, a write vector b and an S x S matrix M:

    u   = sum_s a_s X_s                          what the sub-layer sees, through its RMSNorm
    y   = f(rmsnorm(u) * w) * c                  c: one factor per channel
    X_t = sum_s M[s, t] X_s + r b_t y            r: the model's residual factor

The write of one sub-layer, the read of the next and its norm are one kernel (``ops.stream_ops``): the streams are read and
written once per sub-layer. The model's last sub-layer reads with ones in front of the final norm, and writes nothing back.

Attention: one fused projection gives [q | k | v | gate] with the bias in the GEMM epilogue; q and k are divided by their
root mean square per head and the values of mixing layers blended with those of the first such layer
(``ops.head_norm_kv``, which also writes the cache); a query sees the keys of its own block of ``chunk`` positions that
are not after it; the heads' outputs are multiplied by sigmoid(gate) where the attention kernels store them. The
feed-forward's activation is the GEMM's epilogue.

A batch may hold portions of prompts and single decoded tokens together (``mixed_batches``): the single tokens stand behind
the portions and take the decode kernel. Sizes that are not multiples of the kernels' vectors are padded here, once, with
zeros that no product or norm sees.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import LayerSpec, ModelSpec, pad_to
from ..ops import stream_ops
from .decoder import DecoderModel
from .weights import DTYPES, LayerWeights, ModelWeights, TensorSource, TPInfo, pad_cols, pad_heads, random_tensor


# ------------------------------------------------------------------------------------------
# weights
# ------------------------------------------------------------------------------------------
def expected_tensors(spec: ModelSpec) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor names and shapes. Layer i's tensors start with ``l<i>.``."""
    h, s = spec.hidden, int(spec.extra["duponex"]["streams"])
    m: dict[str, tuple[int, ...]] = {"embed": (spec.vocab, h), "head": (spec.vocab, h), "final.norm": (h,)}
    for i, l in enumerate(spec.layer_specs):
        p = f"l{i}."
        q, k, v, o = l.heads * l.dim, l.kv_heads * l.dim, l.kv_heads * l.vdim, l.heads * l.vdim
        m.update({p + "mix.q": (q, h), p + "mix.q.b": (q,), p + "mix.k": (k, h), p + "mix.k.b": (k,), p + "mix.v": (v, h),
                  p + "mix.v.b": (v,), p + "mix.g": (o, h), p + "mix.o": (h, o), p + "mix.o.b": (h,)})
        if l.v_mix:
            m[p + "mix.vmix"] = ()
        if l.ffn:
            m.update({p + "mlp.up": (l.ffn, h), p + "mlp.down": (h, l.ffn)})
        for n in (1, 2) if l.ffn else (1,):
            m.update({p + f"norm{n}": (h,), p + f"ls{n}": (h,), p + f"hc{n}.in": (s,), p + f"hc{n}.out": (s,),
                      p + f"hc{n}.mix": (s, s)})
    return m


def unused_tensors(spec: ModelSpec) -> tuple[str, ...]:
    """Tensors of parts a layer's configuration switches off: a checkpoint may carry them, nothing reads them."""
    names = []
    for i, l in enumerate(spec.layer_specs):
        if not l.v_mix:
            names.append(f"l{i}.mix.vmix")
        if not l.ffn:
            names += [f"l{i}." + n for n in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix", "mlp.up", "mlp.down")]
    return tuple(names)


def build_weights(spec: ModelSpec, source: TensorSource) -> ModelWeights:
    """Fused and padded weights: ``wqkv`` = [q | k | v | gate] with one bias vector, heads padded to 16 elements, the
    residual width and the feed-forward width to 8."""
    shapes = expected_tensors(spec)
    get = lambda n: source(n, shapes[n])
    wp = pad_to(spec.hidden, 8)
    vec = lambda n: pad_cols(get(n), wp)
    layers = []
    for i, l in enumerate(spec.layer_specs):
        p = f"l{i}."
        dk, dv = l.dim_pad, l.vdim_pad
        lw = LayerWeights()
        lw.input_ln = vec(p + "norm1")
        parts = [("q", l.heads, l.dim, dk), ("k", l.kv_heads, l.dim, dk), ("v", l.kv_heads, l.vdim, dv), ("g", l.heads, l.vdim, dv)]
        w, b = [], []
        for name, heads, width, padded in parts:
            t = get(p + "mix." + name)
            w.append(pad_heads(pad_cols(t, wp), heads, width, padded))
            bias = get(p + f"mix.{name}.b") if name != "g" else t.new_zeros(heads * width)
            b.append(pad_heads(bias, heads, width, padded))
        lw.wqkv, lw.extra["bqkv"] = torch.cat(w).contiguous(), torch.cat(b).contiguous()
        o = pad_heads(get(p + "mix.o").t().contiguous(), l.heads, l.vdim, dv).t()
        lw.wo = pad_cols(o.t().contiguous(), wp).t().contiguous()
        lw.extra["bo"] = vec(p + "mix.o.b")
        lw.extra["vmix"] = float(get(p + "mix.vmix")) if l.v_mix else 0.0
        if l.ffn:
            lw.post_ln = vec(p + "norm2")
            fp = pad_to(l.ffn, 8)
            up, down = pad_cols(get(p + "mlp.up"), wp), pad_cols(get(p + "mlp.down"), fp)
            lw.wgu = pad_cols(up.t().contiguous(), fp).t().contiguous()
            lw.wdown = pad_cols(down.t().contiguous(), wp).t().contiguous()
            lw.wgu_interleaved = False
        for n in (1, 2) if l.ffn else (1,):
            lw.extra[f"ls{n}"] = vec(p + f"ls{n}")
            lw.extra[f"hc{n}"] = {k: get(p + f"hc{n}.{k}").float().cpu() for k in ("in", "out", "mix")}
        layers.append(lw)
    head = pad_cols(get("head"), wp)
    head = pad_cols(head.t().contiguous(), pad_to(spec.vocab, 8)).t().contiguous()
    return ModelWeights(spec=spec, embed=pad_cols(get("embed"), wp), final_norm=vec("final.norm"), lm_head=head, layers=layers,
                        tp=TPInfo(), vocab_shard=(0, spec.vocab))


def random_weights(spec: ModelSpec, seed: int, device: torch.device | str) -> ModelWeights:
    """Seeded weights in which every mechanism counts: norms, layer scales and stream matrices near one, none equal."""
    device = torch.device(device)
    dtype = DTYPES[spec.dtype]
    s = int(spec.extra["duponex"]["streams"])

    def source(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        t = random_tensor(seed, name, shape, torch.float32, device, std=1.0) if len(shape) < 2 or shape == (s, s) else \
            random_tensor(seed, name, shape, dtype, device, std=1.0 if name == "embed" else shape[1] ** -0.5)
        leaf = name.split(".", 1)[-1]
        if leaf.startswith(("norm", "ls")):
            t = 1.0 + 0.2 * t
        elif leaf == "mix.vmix":
            t = torch.sigmoid(t)
        elif leaf.endswith(".in"):
            t = (1.0 + 0.3 * t) / s
        elif leaf.endswith(".out"):
            t = 1.0 + 0.3 * t
        elif leaf.startswith("hc") and leaf.endswith(".mix"):
            t = torch.eye(s, device=device) * 0.8 + 0.1 * t
        elif leaf.endswith(".b"):
            t = 0.3 * t
        return t.to(dtype)
    return build_weights(spec, source)


# ------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------
class _Sublayer:
    """One attention or feed-forward with the tables of the stream kernel around it."""

    def __init__(self, layer: int, kind: str, norm: torch.Tensor, scale: torch.Tensor, hc: dict[str, torch.Tensor]):
        self.layer, self.kind, self.norm, self.scale, self.hc = layer, kind, norm, scale, hc
        self.coef: torch.Tensor | None = None        # [next read | residual factor * write | matrix], FP32


class DuponexModel(DecoderModel):
    mixed_batches = True               # prompt portions and single decoded tokens in one forward

    def __init__(self, weights: ModelWeights, comm=None, trace=None):
        super().__init__(weights, comm=comm, trace=trace)
        assert weights.tp.size == 1, "the Duponex layout is served on one GPU per replica"
        cfg = self.spec.extra["duponex"]
        self.streams, self.embed_scale = int(cfg["streams"]), float(cfg["embed_scale"])
        self.width = self.spec.hidden
        dev = weights.embed.device
        subs: list[_Sublayer] = []
        for i, (l, lw) in enumerate(zip(self.spec.layer_specs, weights.layers)):
            subs.append(_Sublayer(i, "mixer", lw.input_ln, lw.extra["ls1"], lw.extra["hc1"]))
            if l.ffn:
                subs.append(_Sublayer(i, "ffn", lw.post_ln, lw.extra["ls2"], lw.extra["hc2"]))
        factor = float(cfg["residual_mult"])
        for j, s in enumerate(subs):
            read = subs[j + 1].hc["in"] if j + 1 < len(subs) else torch.ones(self.streams)
            s.coef = torch.cat([read, factor * s.hc["out"], s.hc["mix"].reshape(-1)]).float().contiguous().to(dev)
        self.subs = subs
        self.first_read = subs[0].hc["in"].float().contiguous().to(dev)
        self.first_mix = next((i for i, l in enumerate(self.spec.layer_specs) if l.v_mix), -1)

    # -- attention ---------------------------------------------------------------------------
    def _attend(self, i: int, l: LayerSpec, qkvg: torch.Tensor, b, kv) -> torch.Tensor:
        rows = qkvg.shape[0]
        dk, dv = l.dim_pad, l.vdim_pad
        gate = qkvg[:, l.heads * dk + l.kv_heads * (dk + dv):]
        out = torch.empty(rows, l.heads * dv, dtype=qkvg.dtype, device=qkvg.device)
        kw = dict(chunk=l.chunk, vdim=dv)
        singles = b.batch if b.is_decode else b.singles
        n, r = b.batch - singles, rows - singles * (b.nq if b.is_decode else 1)
        if n:
            ops.attn_prefill(qkvg[:r], kv.k[i], kv.v[i], b.block_table[:n], b.q_start[:n], b.q_lens[:n], b.ctx_lens[:n], b.max_q_len,
                             l.heads, l.kv_heads, dk, l.scale, out=out[:r], gate=gate[:r], **kw)
        if singles:
            reach = min(b.max_ctx, l.chunk) if l.chunk else b.max_ctx
            ops.attn_decode(qkvg[r:], kv.k[i], kv.v[i], b.block_table[n:], b.ctx_lens[n:], l.heads, l.kv_heads, dk, l.scale,
                            nq=b.nq if b.is_decode else 1, max_ctx=reach, out=out[r:], gate=gate[r:], **kw)
        return out

    def _mixer(self, i: int, n: torch.Tensor, b, kv, first_v: torch.Tensor | None) -> tuple[torch.Tensor, torch.Tensor | None]:
        """(attention result, values of the first mixing layer)."""
        assert b.tree_mask is None, "tree verification is not available with block-local attention"
        l, lw = self.spec.layer_specs[i], self.w.layers[i]
        dk, dv = l.dim_pad, l.vdim_pad
        qkvg = ops.linear(n, lw.wqkv, bias=lw.extra["bqkv"])
        v0 = (l.heads + l.kv_heads) * dk
        own_v = qkvg[:, v0: v0 + l.kv_heads * dv]
        blend = first_v if l.v_mix and i != self.first_mix else None
        ops.head_norm_kv(qkvg, b.slots, kv.k[i], kv.v[i], l.heads, l.kv_heads, l.dim, l.vdim, self.spec.rms_eps, first_v=blend,
                         mix=lw.extra["vmix"])
        a = self._attend(i, l, qkvg, b, kv)
        if self.trace is not None:
            self.trace.record(f"layer.{i}.attn", a)
        return ops.linear(a, lw.wo, bias=lw.extra["bo"]), own_v if i == self.first_mix else first_v

    # -- forward -----------------------------------------------------------------------------
    def hidden_states(self, b, kv, inputs_embeds=None):
        assert inputs_embeds is None, "the Duponex model takes token ids"
        w, eps = self.w, self.spec.rms_eps
        x, n = stream_ops.embed(b.ids, w.embed, self.embed_scale, self.first_read, self.subs[0].norm, eps, self.width)
        first_v = None
        for j, s in enumerate(self.subs):
            last = j + 1 == len(self.subs)
            if s.kind == "mixer":
                y, first_v = self._mixer(s.layer, n, b, kv, first_v)
            else:
                lw = w.layers[s.layer]
                y = ops.linear(ops.linear(n, lw.wgu, act=self.spec.layer_specs[s.layer].ffn_act), lw.wdown)
            keep = not last or self.trace is not None
            n = stream_ops.step(x, y, s.scale, s.coef, w.final_norm if last else self.subs[j + 1].norm, eps, self.width, write=keep)
            if self.trace is not None and (last or self.subs[j + 1].kind == "mixer"):
                self.trace.record(f"layer.{s.layer}", x.sum(1)[:, : self.width])
        self.last_residual = None
        if self.normed_sink is not None:
            self.normed_sink.append(n)
        return n

    def logits(self, n, b):
        return super().logits(n, b)[:, : self.spec.vocab]


def build_model(weights: ModelWeights, settings, comm=None) -> DuponexModel:
    return DuponexModel(weights, comm=comm)
