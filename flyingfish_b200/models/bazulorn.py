"""Bazulorn decoder: parallel layers (mixer and feed-forward read one norm of an FP32 residual) whose mixer is a gated delta rule with a
decay per key channel, or windowed attention with mixed heads beside a state space; clamped experts; bigrams embedded beside tokens.

    x0 = rms(E[token] + B[bigram]) w
    x <- x + (mixer(h) + ff(h))          h = rms(x) w1

* Delta rule: one projection gives [q | k | v | inner rows of the decays and of the output gate | step sizes]; q, k and v pass a short
  convolution (``delta_ops.short_conv``, which also finds the factors that make q and k unit vectors); ``delta_ops.delta_rule`` runs the
  recurrence from the sequence's state slot; the heads are normed and gated on the way out.
* Attention beside a state space: one projection gives [q | k | v] of the one and [C | B | x | z | steps] of the other. Values are normed
  per head on their way into the cache (``ops.head_norm_kv``); the weights of all heads are mixed before they meet the values
  (``talk_ops``). The state space takes the convolution too, then ``ssd_ops.state_space`` and its gated norm. Both results are normed and
  summed in the kernel that ends the layer.
* Experts: FP32 router logits with their bias, soft-max over the chosen ones; gates clamped in the GEMM epilogues. The mixer and the
  feed-forward do not depend on each other: a decode step runs the routed experts on a second stream beside the mixer.
* The residual is FP32. Its sums, the inner norms and the next layer's norm are one kernel (``residual_ops.step``).

A sequence's state is its last token, the convolutions' last inputs and the recurrences' matrices; attention layers have the paged cache.
A batch may hold portions of prompts and single decoded tokens together (``mixed_batches``): the single tokens stand behind the portions
and take the decode kernels. Sizes that are not multiples of the kernels' vectors are padded here, once, with zeros.
"""
from __future__ import annotations

import os

import torch

from .. import ops
from ..config import LayerSpec, ModelSpec, pad_to
from ..ops import delta_ops, moe_ops, residual_ops, ssd_ops, talk_ops
from .decoder import DecoderModel
from .weights import DTYPES, LayerWeights, ModelWeights, TensorSource, TPInfo, ffn_pair, pad_cols, pad_heads, pad_rows, random_tensor


# ------------------------------------------------------------------------------------------
# weights
# ------------------------------------------------------------------------------------------
def _delta_tensors(l: LayerSpec, p: str, h: int) -> dict[str, tuple[int, ...]]:
    qk, v = l.kv_heads * l.dim, l.heads * l.vdim
    m: dict[str, tuple[int, ...]] = {}
    for n, rows in (("q", qk), ("k", qk), ("v", v)):
        m.update({p + n: (rows, h), p + n + ".conv": (rows, l.conv)})
    m.update({p + "b": (l.heads, h), p + "A_log": (l.heads,), p + "norm": (l.vdim,), p + "a1": (l.decay_rank, h),
              p + "a2": (l.heads * l.dim, l.decay_rank), p + "dt_bias": (l.heads * l.dim,), p + "g1": (l.gate_rank, h),
              p + "g2": (v, l.gate_rank), p + "o": (h, v)})
    return m


def _pair_tensors(l: LayerSpec, p: str, h: int) -> dict[str, tuple[int, ...]]:
    a, q, k, v = p + "left.", l.heads * l.dim, l.kv_heads * l.dim, l.kv_heads * l.vdim
    m: dict[str, tuple[int, ...]] = {}
    for n, rows in (("q", q), ("k", k), ("v", v)):
        m.update({a + n: (rows, h), a + n + ".b": (rows,)})
    m.update({a + "talk": (l.heads, l.heads), a + "o": (h, l.heads * l.vdim), a + "out": (h,)})
    s, b = l.beside, p + "right."
    inner = s.heads * s.vdim
    m.update({b + "in": (2 * inner + 2 * s.kv_heads * s.dim + s.heads, h), b + "conv": (s.conv_channels, s.conv), b + "conv.b": (s.conv_channels,),
              b + "dt_bias": (s.heads,), b + "A_log": (s.heads,), b + "D": (s.heads,), b + "norm": (inner,), b + "o": (h, inner), b + "out": (h,)})
    return m


def expected_tensors(spec: ModelSpec) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor names and shapes. Layer i's tensors start with ``l<i>.``."""
    h = spec.hidden
    m: dict[str, tuple[int, ...]] = {"embed": (spec.vocab, h), "bigram": (spec.extra["bazulorn"]["buckets"] + 1, h), "embed.norm": (h,), "final.norm": (h,)}
    for i, l in enumerate(spec.layer_specs):
        m[f"l{i}.norm1"] = (h,)
        m.update((_delta_tensors if l.mixer == "channel_delta" else _pair_tensors)(l, f"l{i}.mix.", h))
        p = f"l{i}.mlp."
        ffs = [("", l.ffn)] if l.ffn else []
        if l.moe is not None:
            e = l.moe
            m.update({p + "router": (e.num_experts, h), p + "router.b": (e.num_experts,)})
            ffs = [(f"e{j}.", e.expert_ffn) for j in range(e.num_experts)] + ([("shared.", e.shared_ffn)] if e.n_shared else [])
        for name, f in ffs:
            m.update({p + name + "gate": (f, h), p + name + "up": (f, h), p + name + "down": (h, f)})
    return m


def unused_tensors(spec: ModelSpec) -> tuple[str, ...]:
    return ()


def _conv_weights(parts: list[tuple[torch.Tensor, int, int, int]], bias: list[torch.Tensor] | None, nh: int, dn: int, vh: int, dv: int
                  ) -> delta_ops.ConvWeights:
    """``parts``: (weights [heads * width, taps], heads, width, padded width) in the order of the rows' channels."""
    w = torch.cat([pad_heads(t.float(), *s) for t, *s in parts]).t().contiguous()
    b = None if bias is None else torch.cat([pad_heads(t.float(), *p[1:]) for t, p in zip(bias, parts)]).contiguous()
    return delta_ops.ConvWeights(w, b, nh, dn, vh, dv)


def _delta_weights(l: LayerSpec, lw: LayerWeights, get, p: str, wp: int) -> None:
    """``wqkv`` = [q | k | v | a1 | g1 | b]; the second matrices of the pairs by themselves."""
    dk, dv, ra, rg = l.dim_pad, l.vdim_pad, pad_to(l.decay_rank, 8), pad_to(l.gate_rank, 8)
    heads = [("q", l.kv_heads, l.dim, dk), ("k", l.kv_heads, l.dim, dk), ("v", l.heads, l.vdim, dv)]
    rows = [pad_heads(pad_cols(get(p + n), wp), *s) for n, *s in heads]
    rows += [pad_rows(pad_cols(get(p + n), wp), r) for n, r in (("a1", ra), ("g1", rg), ("b", pad_to(l.heads, 8)))]
    lw.wqkv = torch.cat(rows).contiguous()
    lw.extra["conv"] = _conv_weights([(get(p + n + ".conv"), *s) for n, *s in heads], None, 2 * l.kv_heads, dk, l.heads, dv)
    lw.extra["w_decay"] = pad_heads(pad_cols(get(p + "a2"), ra), l.heads, l.dim, dk).contiguous()
    lw.extra["w_gate"] = pad_heads(pad_cols(get(p + "g2"), rg), l.heads, l.vdim, dv).contiguous()
    lw.extra["rate"] = -torch.exp(get(p + "A_log").float()).contiguous()
    lw.extra["dt_bias"] = pad_heads(get(p + "dt_bias").float(), l.heads, l.dim, dk).contiguous()
    lw.extra["norm"] = pad_cols(get(p + "norm").float(), dv).contiguous()
    lw.wo = pad_rows(pad_heads(get(p + "o").t().contiguous(), l.heads, l.vdim, dv).t(), wp).contiguous()


def _pair_weights(l: LayerSpec, lw: LayerWeights, get, p: str, wp: int, vec) -> None:
    """``wqkv`` = [q | k | v] of the attention and [C | B | x | z | steps] of the state space, with one bias vector."""
    a, b, s = p + "left.", p + "right.", l.beside
    dk, dv, N, P = l.dim_pad, l.vdim_pad, s.dim_pad, s.vdim_pad
    heads = [("q", l.heads, l.dim, dk), ("k", l.kv_heads, l.dim, dk), ("v", l.kv_heads, l.vdim, dv)]
    rows = [pad_heads(pad_cols(get(a + n), wp), *t) for n, *t in heads]
    inner, maps = s.heads * s.vdim, s.kv_heads * s.dim
    z, x, B, C, dt = torch.split(pad_cols(get(b + "in"), wp), [inner, inner, maps, maps, s.heads])
    shape = {"head": (s.heads, s.vdim, P), "map": (s.kv_heads, s.dim, N)}
    rows += [pad_heads(t, *shape[k]) for t, k in ((C, "map"), (B, "map"), (x, "head"), (z, "head"))] + [pad_rows(dt, pad_to(s.heads, 8))]
    lw.wqkv = torch.cat(rows).contiguous()
    lw.extra["bqkv"] = torch.cat([pad_heads(get(a + n + ".b"), *t) for n, *t in heads] + [dt.new_zeros(lw.wqkv.shape[0] - sum(h * w for _, h, _, w in heads))]).contiguous()
    lw.extra["talk"] = get(a + "talk").float().contiguous()
    cx, cB, cC = torch.split(get(b + "conv"), [inner, maps, maps])
    bx, bB, bC = torch.split(get(b + "conv.b"), [inner, maps, maps])
    lw.extra["conv"] = _conv_weights([(cC, *shape["map"]), (cB, *shape["map"]), (cx, *shape["head"])], [bC, bB, bx], 2 * s.kv_heads, N, s.heads, P)
    for n in ("dt_bias", "D"):
        lw.extra[n] = get(b + n).float().contiguous()
    lw.extra["rate"] = -torch.exp(get(b + "A_log").float()).contiguous()
    lw.extra["norm"] = pad_heads(get(b + "norm").float(), s.heads, s.vdim, P).contiguous()
    out = lambda n, *t: pad_rows(pad_heads(get(n).t().contiguous(), *t).t(), wp).contiguous()
    lw.wo, lw.extra["wo_right"] = out(a + "o", l.heads, l.vdim, dv), out(b + "o", s.heads, s.vdim, P)
    # the layer takes half the sum of the two
    lw.extra["out_left"], lw.extra["out_right"] = 0.5 * vec(a + "out"), 0.5 * vec(b + "out")


def build_weights(spec: ModelSpec, source: TensorSource) -> ModelWeights:
    """Fused and padded weights; heads padded to 16 elements, experts stacked. Norm weights, convolutions, decays and biases that enter
    32-bit arithmetic are FP32."""
    shapes = expected_tensors(spec)
    get = lambda n: source(n, shapes[n])
    wp = pad_to(spec.hidden, 8)
    vec = lambda n: pad_cols(get(n).float(), wp).contiguous()
    layers = []
    for i, l in enumerate(spec.layer_specs):
        lw = LayerWeights()
        lw.input_ln = vec(f"l{i}.norm1")
        if l.mixer == "channel_delta":
            _delta_weights(l, lw, get, f"l{i}.mix.", wp)
        else:
            _pair_weights(l, lw, get, f"l{i}.mix.", wp, vec)
        p = f"l{i}.mlp."
        if l.ffn:
            lw.wgu, lw.wdown = ffn_pair(get, p, wp, pad_to(l.ffn, 128))
        if l.moe is not None:
            e = l.moe
            lw.router = pad_rows(pad_cols(get(p + "router"), wp), pad_to(e.num_experts, 16)).contiguous()
            lw.router_bias = get(p + "router.b").float().contiguous()
            fp = pad_to(e.expert_ffn, 64)
            lw.experts_gu = lw.router.new_empty(e.num_experts, 2 * fp, wp)
            lw.experts_down = lw.router.new_empty(e.num_experts, wp, fp)
            for j in range(e.num_experts):
                lw.experts_gu[j], lw.experts_down[j] = ffn_pair(get, p + f"e{j}.", wp, fp)
            if e.n_shared:
                lw.shared_gu, lw.shared_down = ffn_pair(get, p + "shared.", wp, pad_to(e.shared_ffn, 128))
        layers.append(lw)
    table = pad_rows(pad_cols(get("embed"), wp), pad_to(spec.vocab, 8)).contiguous()
    w = ModelWeights(spec=spec, embed=table[: spec.vocab], final_norm=vec("final.norm"), lm_head=table, layers=layers, tp=TPInfo(),
                     vocab_shard=(0, spec.vocab))
    w.extra["bigram"], w.extra["embed_norm"] = pad_cols(get("bigram"), wp).contiguous(), vec("embed.norm")
    return w


def random_weights(spec: ModelSpec, seed: int, device: torch.device | str) -> ModelWeights:
    """Seeded weights in which every mechanism counts."""
    device = torch.device(device)
    dtype = DTYPES[spec.dtype]
    centre = {"A_log": -1.0, "dt_bias": -2.0, "b": 0.0}

    def source(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        leaf = name.rsplit(".", 1)[-1]
        if len(shape) == 1:
            t = random_tensor(seed, name, shape, torch.float32, device, std=1.0 if leaf in ("A_log", "dt_bias") else 0.2)
            return (centre.get(leaf, 1.0) + t).to(dtype)
        if leaf == "talk":
            return (torch.eye(shape[0], device=device) + random_tensor(seed, name, shape, torch.float32, device, std=0.3)).to(dtype)
        std = 1.0 if name in ("embed", "bigram") else shape[1] ** -0.5
        return random_tensor(seed, name, shape, dtype, device, std=std)
    return build_weights(spec, source)


# ------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------
# decode steps of up to this many rows run a layer's mixer and its experts side by side on two streams (0: never)
OVERLAP_ROWS = int(os.environ.get("FLYINGFISH_OVERLAP_ROWS", "64"))


class BazulornModel(DecoderModel):
    mixed_batches = True               # prompt portions and single decoded tokens in one forward
    graph_safe_state = True            # slots and row ranges come from the packed step metadata

    def __init__(self, weights: ModelWeights, comm=None, trace=None, max_sequences: int = 64):
        super().__init__(weights, comm=comm, trace=trace)
        assert weights.tp.size == 1, "the Bazulorn layout is served on one GPU per replica"
        spec, dev = self.spec, weights.embed.device
        self.width, self.bigram = spec.hidden, spec.extra["bazulorn"]
        n = self.state_slot_count = max_sequences + 1        # the last slot is scratch of padding rows
        self.last_token = torch.full((n,), -1, dtype=torch.int32, device=dev)
        self.convs = [delta_ops.ConvState(n, lw.extra["conv"], dev) for lw in weights.layers]
        self.states: list = []
        for l in spec.layer_specs:
            if l.mixer == "channel_delta":
                self.states.append(delta_ops.DeltaState(n, l.heads, l.kv_heads, l.dim_pad, l.vdim_pad, dev))
            else:
                s = l.beside
                self.states.append(ssd_ops.SsdState(n, s.heads, s.kv_heads, s.dim_pad, s.vdim_pad, dev))
        self.lane = ops.SideLane(dev) if dev.type == "cuda" else None

    def reset_state(self, slot: int) -> None:
        self.last_token[slot] = -1
        for st in self.convs + self.states:
            st.reset(slot)

    def state_bytes_per_sequence(self) -> int:
        return 4 + sum(st.bytes_per_slot() for st in self.convs + self.states)

    # -- mixers ------------------------------------------------------------------------------
    @staticmethod
    def _split(b) -> tuple[int, int]:
        """(sequences with a portion, rows of theirs); what stands behind them takes the decode kernels."""
        if b.is_decode:
            return 0, 0
        return b.batch - b.singles, b.rows - b.singles

    def _recurrence(self, b, run) -> None:
        """``run(row starts, slots, longest)`` for the portions and for the single tokens of a batch."""
        s, _ = self._split(b)
        for lo, hi, longest in ((0, s, b.max_q_len), (s, b.batch, b.nq)):
            if lo < hi:
                run(b.row_start[lo: hi + 1], b.state_slots_dev[lo:hi], longest)

    def _longest(self, b) -> int:
        return b.nq if b.is_decode else b.max_q_len

    def _delta(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b) -> torch.Tensor:
        p = ops.linear(n, lw.wqkv)
        conv, unit = delta_ops.short_conv(p, lw.extra["conv"], self.convs[i], b.row_start, b.state_slots_dev, self._longest(b), unit_scale=l.scale)
        at = l.conv_pad
        ra, rg = pad_to(l.decay_rank, 8), pad_to(l.gate_rank, 8)
        decay = ops.linear(p[:, at: at + ra], lw.extra["w_decay"], out_dtype=torch.float32)
        gate = ops.linear(p[:, at + ra: at + ra + rg], lw.extra["w_gate"])
        o = torch.empty(b.rows, l.heads, l.vdim_pad, dtype=torch.float32, device=p.device)
        self._recurrence(b, lambda rows, slots, longest: delta_ops.delta_rule(
            conv, unit, decay, p[:, at + ra + rg:], lw.extra["rate"], lw.extra["dt_bias"], self.states[i], rows, slots, o, longest))
        return delta_ops.head_out(o, gate, lw.extra["norm"], l.vdim, self.spec.rms_eps)

    def _attention_part(self, i: int, l: LayerSpec, lw: LayerWeights, p: torch.Tensor, b, kv) -> torch.Tensor:
        dv = l.vdim_pad
        ops.head_norm_kv(p, b.slots, kv.k[i], kv.v[i], l.heads, l.kv_heads, l.dim, l.vdim, self.spec.rms_eps, norm_qk=False, norm_v=l.v_norm)
        out = torch.empty(b.rows, l.heads * dv, dtype=p.dtype, device=p.device)
        s, rows = self._split(b)
        args = (l.heads, l.kv_heads, l.scale, l.window, lw.extra["talk"], l.sink_one)
        if s:
            talk_ops.talk_prefill(p[:rows], kv.k[i], kv.v[i], b.block_table[:s], b.q_start[:s], b.q_lens[:s], b.ctx_lens[:s], b.max_q_len, b.max_ctx, *args,
                                  out=out[:rows])
        if s < b.batch:
            talk_ops.talk_decode(p[rows:], kv.k[i], kv.v[i], b.block_table[s:], b.ctx_lens[s:], b.max_ctx, *args, out=out[rows:])
        return out

    def _state_space_part(self, i: int, s: LayerSpec, lw: LayerWeights, p: torch.Tensor, b) -> torch.Tensor:
        """``p``: [C | B | x | z | steps]."""
        at, inner = s.conv_pad, s.heads * s.vdim_pad
        conv, _ = delta_ops.short_conv(p, lw.extra["conv"], self.convs[i], b.row_start, b.state_slots_dev, self._longest(b))
        o = torch.empty(b.rows, s.heads, s.vdim_pad, dtype=torch.float32, device=p.device)
        self._recurrence(b, lambda rows, slots, longest: ssd_ops.state_space(
            conv, p[:, at + inner:], lw.extra["dt_bias"], lw.extra["rate"], lw.extra["D"], self.states[i], rows, slots, o, longest))
        return ssd_ops.gated_out(o, p[:, at: at + inner], lw.extra["norm"], s.vdim, s.norm_groups, self.spec.rms_eps)

    def _mixer(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b, kv) -> tuple[torch.Tensor, residual_ops.Beside | None]:
        """(the mixer's rows, or the first of two with what the second adds)."""
        if l.mixer == "channel_delta":
            a = self._delta(i, l, lw, n, b)
            if self.trace is not None:
                self.trace.record(f"layer.{i}.mixer", a)
            return ops.linear(a, lw.wo), None
        p = ops.linear(n, lw.wqkv, bias=lw.extra["bqkv"])
        a = self._attention_part(i, l, lw, p, b, kv)
        r = self._state_space_part(i, l.beside, lw, p[:, l.heads * l.dim_pad + l.kv_heads * (l.dim_pad + l.vdim_pad):], b)
        if self.trace is not None:
            self.trace.record(f"layer.{i}.left", a)
            self.trace.record(f"layer.{i}.right", r)
        return ops.linear(a, lw.wo), residual_ops.Beside(ops.linear(r, lw.extra["wo_right"]), lw.extra["out_left"], lw.extra["out_right"])

    # -- feed-forward --------------------------------------------------------------------------
    def _experts(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor) -> moe_ops.ExpertRows:
        """The routed experts' rows."""
        m = l.moe
        rows = moe_ops.routed_rows(n, lw.router, m.top_k, m.score, lw.router_bias, m.num_experts, lw.experts_gu, lw.experts_down, m.limit)
        if getattr(self, "route_hook", None) is not None:
            self.route_hook(i, rows.ids, rows.weights)
        return rows

    @staticmethod
    def _dense(l: LayerSpec, lw: LayerWeights, n: torch.Tensor) -> torch.Tensor | None:
        """The rows of the dense feed-forward or of the shared expert."""
        if l.ffn:
            return ops.linear(ops.linear_swiglu(n, lw.wgu, mode=3), lw.wdown)
        if l.moe is not None and l.moe.n_shared:
            return ops.linear(ops.linear_swiglu(n, lw.shared_gu, mode=5, limit=l.moe.shared_limit), lw.shared_down)
        return None

    # -- forward -----------------------------------------------------------------------------
    def hidden_states(self, b, kv, inputs_embeds=None):
        assert inputs_embeds is None, "the Bazulorn model takes token ids"
        assert b.tree_mask is None, "tree verification is not available with recurrent state"
        assert b.state_slots is not None and len(b.state_slots) == b.batch, "the engine must name a state slot per sequence of the batch"
        w, spec, eps = self.w, self.spec, self.spec.rms_eps
        side = self.lane is not None and b.is_decode and b.rows <= OVERLAP_ROWS
        norms = [lw.input_ln for lw in w.layers] + [w.final_norm]
        bigrams = residual_ops.bigram_rows(b.ids, self.last_token, b.row_start, b.state_slots_dev, **self.bigram)
        x, n, _ = residual_ops.embed(b.ids, w.embed, 1.0, norms[0], None, eps, self.width,
                                     second=residual_ops.Second(w.extra["bigram"], bigrams, w.extra["embed_norm"]))
        for i, l in enumerate(spec.layer_specs):
            lw, rows = w.layers[i], None
            if l.moe is not None and side:
                self.lane.fork()
                with self.lane:
                    rows = self._experts(i, l, lw, n)
            elif l.moe is not None:
                rows = self._experts(i, l, lw, n)
            y, beside = self._mixer(i, l, lw, n, b, kv)
            dense = self._dense(l, lw, n)
            if side and rows is not None:
                self.lane.join()
            n, _ = residual_ops.step(x, y, dense, rows, norms[i + 1], None, eps, self.width, beside=beside)
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


def build_model(weights: ModelWeights, settings, comm=None) -> BazulornModel:
    return BazulornModel(weights, comm=comm, max_sequences=settings.max_batch)
