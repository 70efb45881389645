"""Rudorax decoder: parallel layers (mixer and feed-forward read one residual through two norms), windowed attention with sinks
and scaled rotary positions or a matrix memory with exponential gates as the mixer, experts with identity outputs, layers that
run several times.

    x <- x + mixer(rms(x) (1 + w1)) + ff(rms(x) (1 + w2))

* Attention: one projection gives [q | k | v]; q and k are normed per head with a weight and rotated (``ops.head_norm_kv``, which
  also writes the cache); a query sees its last ``window`` positions; every head has a sink logit in the soft-max denominator.
* Matrix memory: one projection gives [q | k | v | gate], a second one, kept in FP32, the logits of the input and forget gates;
  ``ops.mlstm_ops`` runs the recurrence from the sequence's state slot; the heads are normed and gated on the way out.
* Experts: FP32 router logits, soft-max over all outputs, the choice moved by a bias the weights do not see. Outputs behind the
  experts are identities. A shared expert runs for every token.
* The mixer and the feed-forward do not depend on each other: a decode step runs the routed experts on a second stream beside the
  mixer and the shared expert.
* The residual is FP32. Its sums (mixer, shared expert, the chosen experts' rows with their weights, identity outputs) and the two
  norms of the next layer are one kernel (``ops.residual_ops``).

A layer run, not a layer, owns a cache layer or a state: the passes of a looped layer share weights and nothing else. A batch may
hold portions of prompts and single decoded tokens together (``mixed_batches``): the single tokens stand behind the portions and
take the decode kernels. Sizes that are not multiples of the kernels' vectors are padded here, once, with zeros.
"""
from __future__ import annotations

import os

import torch

from .. import ops
from ..config import LayerSpec, ModelSpec, pad_to
from ..ops import mlstm_ops, moe_ops, residual_ops
from .decoder import DecoderModel
from .weights import DTYPES, LayerWeights, ModelWeights, TensorSource, TPInfo, ffn_pair, pad_cols, pad_heads, pad_rows, random_tensor


# ------------------------------------------------------------------------------------------
# weights
# ------------------------------------------------------------------------------------------
def expected_tensors(spec: ModelSpec) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor names and shapes. Layer i's tensors start with ``l<i>.``."""
    h = spec.hidden
    m: dict[str, tuple[int, ...]] = {"embed": (spec.vocab, h), "head": (spec.vocab, h), "final.norm": (h,)}
    for i, l in enumerate(spec.layer_specs):
        p = f"l{i}.mix."
        o = l.heads * l.vdim
        m.update({f"l{i}.norm1": (h,), p + "q": (l.heads * l.dim, h), p + "k": (l.kv_heads * l.dim, h), p + "v": (l.kv_heads * l.vdim, h), p + "o": (h, o)})
        if l.mixer == "attention":
            m.update({p + "q.norm": (l.dim,), p + "k.norm": (l.dim,), p + "sink": (l.heads,)})
        else:
            m.update({p + "g": (o, h), p + "norm": (o,), p + "i": (l.heads, h), p + "i.b": (l.heads,), p + "f": (l.heads, h), p + "f.b": (l.heads,)})
        if l.moe is not None:
            e, p = l.moe, f"l{i}.mlp."
            m.update({f"l{i}.norm2": (h,), p + "router": (e.num_experts + e.identity, h), p + "correction": (e.num_experts + e.identity,)})
            for name, f in [(f"e{j}.", e.expert_ffn) for j in range(e.num_experts)] + ([("shared.", e.shared_ffn)] if e.n_shared else []):
                m.update({p + name + "gate": (f, h), p + name + "up": (f, h), p + name + "down": (h, f)})
    return m


def unused_tensors(spec: ModelSpec) -> tuple[str, ...]:
    """Tensors of parts a layer's configuration switches off: a checkpoint may carry them, nothing reads them."""
    return tuple(f"l{i}.norm2" for i, l in enumerate(spec.layer_specs) if l.moe is None)


def build_weights(spec: ModelSpec, source: TensorSource) -> ModelWeights:
    """Fused and padded weights: ``wqkv`` = [q | k | v] (matrix memory: and the output gate) with heads padded to 16 elements; the
    gate projections of a matrix memory as one matrix; experts stacked. Norm weights (with their offset), biases, sinks and
    frequencies are FP32."""
    shapes = expected_tensors(spec)
    get = lambda n: source(n, shapes[n])
    h, wp = spec.hidden, pad_to(spec.hidden, 8)
    vec = lambda n: pad_cols(1.0 + get(n).float(), wp).contiguous()
    layers = []
    for i, l in enumerate(spec.layer_specs):
        p = f"l{i}.mix."
        dk, dv = l.dim_pad, l.vdim_pad
        lw = LayerWeights()
        lw.input_ln = vec(f"l{i}.norm1")
        parts = [("q", l.heads, l.dim, dk), ("k", l.kv_heads, l.dim, dk), ("v", l.kv_heads, l.vdim, dv)]
        if l.out_gate:
            parts.append(("g", l.heads, l.vdim, dv))
        lw.wqkv = torch.cat([pad_heads(pad_cols(get(p + n), wp), *s) for n, *s in parts]).contiguous()
        lw.wo = pad_rows(pad_heads(get(p + "o").t().contiguous(), l.heads, l.vdim, dv).t(), wp).contiguous()
        if l.mixer == "attention":
            lw.q_norm, lw.k_norm = (pad_cols(get(p + n).float(), dk).contiguous() for n in ("q.norm", "k.norm"))
            lw.extra["sinks"] = get(p + "sink").float().contiguous()
        else:
            lw.extra["w_gates"] = pad_rows(torch.cat([pad_cols(get(p + n), wp) for n in ("i", "f")]), pad_to(2 * l.heads, 16)).contiguous()
            lw.extra["b_gates"] = torch.cat([get(p + n).float() for n in ("i.b", "f.b")]).contiguous()
            lw.extra["norm"] = pad_heads(get(p + "norm").float(), l.heads, l.vdim, dv).contiguous()
        if l.moe is not None:
            e, p = l.moe, f"l{i}.mlp."
            lw.post_ln = vec(f"l{i}.norm2")
            n = e.num_experts + e.identity
            lw.router = pad_rows(pad_cols(get(p + "router"), wp), pad_to(n, 16)).contiguous()
            lw.router_bias = get(p + "correction").float().contiguous()
            fp = pad_to(e.expert_ffn, 64)
            lw.experts_gu = lw.router.new_empty(e.num_experts, 2 * fp, wp)
            lw.experts_down = lw.router.new_empty(e.num_experts, wp, fp)
            for j in range(e.num_experts):
                lw.experts_gu[j], lw.experts_down[j] = ffn_pair(get, p + f"e{j}.", wp, fp)
            if e.n_shared:
                lw.shared_gu, lw.shared_down = ffn_pair(get, p + "shared.", wp, pad_to(e.shared_ffn, 128))
        layers.append(lw)
    head = pad_rows(pad_cols(get("head"), wp), pad_to(spec.vocab, 8)).contiguous()
    return ModelWeights(spec=spec, embed=pad_cols(get("embed"), wp).contiguous(), final_norm=vec("final.norm"), lm_head=head, layers=layers,
                        tp=TPInfo(), vocab_shard=(0, spec.vocab))


def random_weights(spec: ModelSpec, seed: int, device: torch.device | str) -> ModelWeights:
    """Seeded weights in which every mechanism counts."""
    device = torch.device(device)
    dtype = DTYPES[spec.dtype]
    offsets = {"q.norm": 1.0, "k.norm": 1.0, "norm": 1.0, "i.b": -1.0, "f.b": 3.0}

    def source(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        if len(shape) == 1:
            leaf = name.split(".mix.")[-1] if ".mix." in name else name.split(".")[-1]
            std = 0.02 if leaf == "correction" else 0.2
            return (offsets.get(leaf, 0.0) * (".mix." in name) + random_tensor(seed, name, shape, torch.float32, device, std=std)).to(dtype)
        return random_tensor(seed, name, shape, dtype, device, std=1.0 if name == "embed" else shape[1] ** -0.5)
    return build_weights(spec, source)


# ------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------
# decode steps of up to this many rows run a layer's mixer and its experts side by side on two streams (0: never)
OVERLAP_ROWS = int(os.environ.get("FLYINGFISH_OVERLAP_ROWS", "64"))


class RudoraxModel(DecoderModel):
    mixed_batches = True               # prompt portions and single decoded tokens in one forward
    graph_safe_state = True            # slots and row ranges come from the packed step metadata

    def __init__(self, weights: ModelWeights, comm=None, trace=None, max_sequences: int = 64):
        super().__init__(weights, comm=comm, trace=trace)
        assert weights.tp.size == 1, "the Rudorax layout is served on one GPU per replica"
        spec, dev = self.spec, weights.embed.device
        cfg = spec.extra["rudorax"]
        self.embed_scale, self.softcap = float(cfg["embed_scale"]), float(cfg["softcap"])
        self.width = spec.hidden
        self.runs = spec.runs
        memories = [(r, spec.layer_specs[i]) for r, i in enumerate(self.runs) if spec.layer_specs[i].mixer == "mlstm"]
        self.state_slot_count = max_sequences + 1 if memories else 0          # the last slot is scratch of padding rows
        self.states = {r: mlstm_ops.MemoryState(self.state_slot_count, l.heads, l.dim_pad, l.vdim_pad, dev) for r, l in memories}
        self.lane = ops.SideLane(dev) if dev.type == "cuda" else None
        # rotations, one table per step for all layers that share one
        self.rotations: list[tuple[torch.Tensor, float]] = []
        self.rotation_of: list[int] = []
        known: list = []
        for l in spec.layer_specs:
            if l.rope is None:
                self.rotation_of.append(-1)
                continue
            if l.rope not in known:
                known.append(l.rope)
                freqs, amp = l.rope.frequencies()
                self.rotations.append((ops.rope_frequencies(freqs, dev), amp))
            self.rotation_of.append(known.index(l.rope))

    def reset_state(self, slot: int) -> None:
        for st in self.states.values():
            st.reset(slot)

    def state_bytes_per_sequence(self) -> int:
        return sum(st.bytes_per_slot() for st in self.states.values())

    # -- mixers ------------------------------------------------------------------------------
    @staticmethod
    def _split(b) -> tuple[int, int]:
        """(sequences with a portion, rows of theirs); what stands behind them takes the decode kernels."""
        if b.is_decode:
            return 0, 0
        return b.batch - b.singles, b.rows - b.singles

    def _attention_run(self, r: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b, kv, table) -> torch.Tensor:
        dk, dv = l.dim_pad, l.vdim_pad
        qkv = ops.linear(n, lw.wqkv)
        ops.head_norm_kv(qkv, b.slots, kv.k[r], kv.v[r], l.heads, l.kv_heads, l.dim, l.vdim, self.spec.rms_eps, q_weight=lw.q_norm,
                         k_weight=lw.k_norm, cos_sin=table)
        out = torch.empty(b.rows, l.heads * dv, dtype=qkv.dtype, device=qkv.device)
        kw = dict(window=l.window, sinks=lw.extra["sinks"], vdim=dv)
        s, rows = self._split(b)
        if s:
            ops.attn_prefill(qkv[:rows], kv.k[r], kv.v[r], b.block_table[:s], b.q_start[:s], b.q_lens[:s], b.ctx_lens[:s], b.max_q_len,
                             l.heads, l.kv_heads, dk, l.scale, out=out[:rows], **kw)
        if s < b.batch:
            reach = min(b.max_ctx, l.window + kv.block_size) if l.window else b.max_ctx
            ops.attn_decode(qkv[rows:], kv.k[r], kv.v[r], b.block_table[s:], b.ctx_lens[s:], l.heads, l.kv_heads, dk, l.scale,
                            nq=b.nq if b.is_decode else 1, max_ctx=reach, out=out[rows:], **kw)
        return out

    def _memory_run(self, r: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor, b) -> torch.Tensor:
        assert b.state_slots is not None and len(b.state_slots) == b.batch, "the engine must name a state slot per sequence of the batch"
        dv = l.vdim_pad
        x = ops.linear(n, lw.wqkv)
        gates = ops.linear(n, lw.extra["w_gates"], out_dtype=torch.float32)
        o = torch.empty(b.rows, l.heads, dv, dtype=torch.float32, device=x.device)
        s, _ = self._split(b)
        for lo, hi, longest in ((0, s, b.max_q_len), (s, b.batch, b.nq)):
            if lo < hi:
                mlstm_ops.memory(x, gates, lw.extra["b_gates"], l.gate_cap, self.states[r], b.row_start[lo: hi + 1], b.state_slots_dev[lo:hi],
                                 l.scale, o, longest)
        return mlstm_ops.head_out(o, x[:, l.heads * (2 * l.dim_pad + dv):], lw.extra["norm"], l.vdim, self.spec.rms_eps)

    # -- feed-forward --------------------------------------------------------------------------
    def _experts(self, i: int, l: LayerSpec, lw: LayerWeights, n: torch.Tensor) -> moe_ops.ExpertRows:
        """The routed experts' rows."""
        m = l.moe
        rows = moe_ops.routed_rows(n, lw.router, m.top_k, m.score, lw.router_bias, m.num_experts + m.identity, lw.experts_gu, lw.experts_down)
        if getattr(self, "route_hook", None) is not None:
            self.route_hook(i, rows.ids, rows.weights)
        return rows

    @staticmethod
    def _shared(l: LayerSpec, lw: LayerWeights, n: torch.Tensor) -> torch.Tensor | None:
        """The shared expert's rows."""
        return ops.linear(ops.linear_swiglu(n, lw.shared_gu), lw.shared_down) if l.moe is not None and l.moe.n_shared else None

    # -- forward -----------------------------------------------------------------------------
    def hidden_states(self, b, kv, inputs_embeds=None):
        assert inputs_embeds is None, "the Rudorax model takes token ids"
        assert b.tree_mask is None, "tree verification is not available with a learnable soft-max or recurrent state"
        w, spec, eps = self.w, self.spec, self.spec.rms_eps
        side = self.lane is not None and b.is_decode and b.rows <= OVERLAP_ROWS
        tables = [ops.rope_angles(b.positions, f, amp) for f, amp in self.rotations]
        norms = [(w.layers[i].input_ln, w.layers[i].post_ln) for i in self.runs] + [(w.final_norm, None)]
        x, n1, n2 = residual_ops.embed(b.ids, w.embed, self.embed_scale, *norms[0], eps, self.width)
        for r, i in enumerate(self.runs):
            l, lw = spec.layer_specs[i], w.layers[i]
            rows = None
            if l.moe is not None and side:
                self.lane.fork()
                with self.lane:
                    rows = self._experts(i, l, lw, n2)
            elif l.moe is not None:
                rows = self._experts(i, l, lw, n2)
            if l.mixer == "attention":
                a = self._attention_run(r, l, lw, n1, b, kv, tables[self.rotation_of[i]] if l.rope is not None else None)
            else:
                a = self._memory_run(r, l, lw, n1, b)
            if self.trace is not None:
                self.trace.record(f"run.{r}.mixer", a)
            y = ops.linear(a, lw.wo)
            shared = self._shared(l, lw, n2)
            if side and rows is not None:
                self.lane.join()
            n1, n2 = residual_ops.step(x, y, shared, rows, *norms[r + 1], eps, self.width)
            if self.trace is not None:
                self.trace.record(f"run.{r}", x[:, : self.width].clone())
        self.last_residual = None
        if self.normed_sink is not None:
            self.normed_sink.append(n1)
        return n1

    def logits(self, n, b):
        """FP32, soft-capped."""
        sel = n.index_select(0, b.logit_rows.long()) if b.n_logit_rows != n.shape[0] else n
        lg = ops.linear(sel.contiguous(), self.w.lm_head, out_dtype=torch.float32)
        if self.softcap:
            lg = ops.softcap(lg, self.softcap)
        return lg[:, : self.spec.vocab]


def build_model(weights: ModelWeights, settings, comm=None) -> RudoraxModel:
    return RudoraxModel(weights, comm=comm, max_sequences=settings.max_batch)
