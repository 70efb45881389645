"""Model geometry and engine settings.

``ModelSpec`` is the normalised description of a decoder that the rest of the framework works
from (the counterpart of the reference's ``ModelSpec`` / ``Config``: src/model_spec.rs:8-104,
469-510; src/config.rs:5-104). It can be read from a Hugging Face ``config.json`` or taken from
the table of named benchmark shapes below. ``Settings`` carries the engine options of the CLI
(src/backend/mod.rs:196-224).
"""
from __future__ import annotations

import dataclasses
import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Any


@dataclass
class MoeSpec:
    num_experts: int
    top_k: int
    expert_ffn: int
    score: str = "softmax"            # softmax | biased_softmax | sigmoid | noaux | sqrt_softplus
    n_shared: int = 0                 # shared experts (each of width shared_ffn)
    shared_ffn: int = 0
    n_groups: int = 1
    topk_groups: int = 1
    routed_scaling: float = 1.0
    renormalize: bool = True
    first_dense_layers: int = 0       # leading layers with a dense FFN
    dense_ffn: int = 0
    identity: int = 0                 # router outputs behind the experts whose output is the input itself
    shared_gate: bool = False         # sigmoid gate on the shared expert (Qwen-style)
    expert_format: str = "bf16"       # bf16 | fp8_block | nvfp4
    limit: float = 0.0                # > 0: the experts' gate is clamped there (g sigmoid(1.702 g) (u + 1)) in place of SiLU
    shared_limit: float = 0.0         # the same of the shared expert


@dataclass
class MlaSpec:
    q_lora_rank: int
    kv_lora_rank: int
    qk_nope_dim: int
    qk_rope_dim: int
    v_head_dim: int


@dataclass
class RopeSpec:
    """Rotary positions on the first ``dims`` elements of a head. Pairs are neighbours (2i, 2i + 1) or, with ``halves``, elements
    (i, i + dims / 2)."""
    base: float
    dims: int
    factor: float = 1.0               # with ``original``: YaRN-scaled frequencies and amplitude; without: frequencies / factor
    original: int = 0
    fast: float = 32.0
    slow: float = 1.0
    halves: bool = False

    def frequencies(self) -> tuple[list[float], float]:
        """(angle per position of every pair, factor of cosine and sine), in double precision."""
        plain = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if not self.original:
            return [f / self.factor for f in plain], 1.0
        turn = lambda t: self.dims * math.log(self.original / (2.0 * math.pi * t)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(turn(self.fast)), 0), min(math.ceil(turn(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(self.dims // 2)]
        return [f / self.factor * r + f * (1.0 - r) for f, r in zip(plain, ramp)], 0.1 * math.log(self.factor) + 1.0


@dataclass
class LayerSpec:
    """One layer of a design whose layers need not look alike (``ModelSpec.layer_specs``)."""
    heads: int
    kv_heads: int
    dim: int                          # width of a query / key head
    vdim: int                         # width of a value head
    scale: float                      # factor of the attention scores (of the queries, for a matrix memory)
    # attention | latent (latent attention); with a per-sequence state instead of a cache: mlstm (matrix memory), channel_delta (gated
    # delta rule with a decay per key channel), ssd (state space: ``dim`` states, ``kv_heads`` groups of input and output maps)
    mixer: str = "attention"
    chunk: int = 0                    # > 0: position i sees only keys of its own block of ``chunk`` positions
    window: int = 0                   # > 0: position i sees itself and the ``window - 1`` positions before it
    keep_first: int = 0               # with a window: the sequence's first ``keep_first`` positions stay visible
    sink: bool = False                # learnable soft-max: one extra logit per head in the denominator
    sink_one: bool = False            # the denominator has one more, fixed, term: e^0
    talk: bool = False                # the heads' weights are mixed by a matrix [heads, heads] before they meet the values
    v_norm: bool = False              # values are divided by their root mean square per head (and cached so)
    rope: RopeSpec | None = None
    qk_norm: str = "head"             # RMS norm of q and k: over every head, or over the whole projection ("row")
    bias: bool = False                # the projections have biases
    softcap: float = 0.0              # > 0: scores become softcap * tanh(score / softcap)
    q_temp: tuple[float, int] | None = None       # (coef, every): the query at p is multiplied by 1 + coef ln((p + 1) // every + 1)
    kv_from: int = -1                 # >= 0: keys and values are those of that layer's cache
    kv_rank: int = 0                  # latent attention: width of the latent a token caches
    rot_dim: int = 0                  # latent attention: width of the rotated key part all heads share (and of the queries')
    gate_cap: float = 0.0             # matrix memory: soft cap of the gates' logits
    conv: int = 0                     # channel_delta, ssd: taps of the causal convolution in front of the recurrence
    decay_rank: int = 0               # channel_delta: width between the two matrices of the decays (0: the checkpoint says)
    gate_rank: int = 0                # channel_delta: the same of the output gate
    norm_groups: int = 1              # ssd: equal parts of the heads' outputs, normed each by itself
    beside: "LayerSpec | None" = None # a second mixer on the same input; the layer's result is half the sum of the two, each normed
    out_gate: bool = True             # the heads' outputs are multiplied by the sigmoid of a projection
    v_mix: bool = False               # values are mixed with those of the first layer that has the flag
    ffn: int = 0                      # width of the feed-forward (0: the layer has none, or experts)
    ffn_act: str = "relu2"            # relu2 (two matrices) | geglu (gate, up and down matrices, tanh-GELU)
    moe: MoeSpec | None = None        # experts in place of a dense feed-forward

    @property
    def dim_pad(self) -> int:
        return pad_to(self.dim, 16)

    @property
    def vdim_pad(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def rot_pad(self) -> int:
        return pad_to(self.rot_dim, 16)

    @property
    def rank_pad(self) -> int:
        return pad_to(self.kv_rank, 16)

    def keys_seen(self, ctx: int) -> int:
        """Keys the last of ``ctx`` positions sees."""
        if self.window:
            return min(ctx, self.window) + min(max(ctx - self.window, 0), self.keep_first)
        return (ctx - 1) % self.chunk + 1 if self.chunk else ctx

    def pairs_seen(self, n: int) -> int:
        """(query, key) pairs of a prompt of ``n`` positions."""
        if self.window:
            w = min(n, self.window)
            k = min(n - w, self.keep_first)        # row w + j sees j + 1 kept positions outside its window, up to keep_first
            return w * (w + 1) // 2 + (n - w) * w + k * (k + 1) // 2 + (n - w - k) * self.keep_first
        if not self.chunk:
            return n * (n + 1) // 2
        full, rest = divmod(n, self.chunk)
        return full * self.chunk * (self.chunk + 1) // 2 + rest * (rest + 1) // 2

    def cache_bytes_read(self, ctx: int, elem_bytes: int) -> int:
        """Bytes of cache or state one decoded token moves at a context of ``ctx``."""
        if self.beside is not None:
            return dataclasses.replace(self, beside=None).cache_bytes_read(ctx, elem_bytes) + self.beside.cache_bytes_read(ctx, elem_bytes)
        if self.mixer == "mlstm":
            return 2 * 4 * self.heads * self.dim * (self.vdim + 1)
        if self.mixer in ("channel_delta", "ssd"):
            return 2 * 4 * (self.heads * self.dim * self.vdim + (self.conv - 1) * self.conv_channels)
        if self.mixer == "latent":
            return elem_bytes * self.keys_seen(ctx) * (self.kv_rank + self.rot_dim)
        return elem_bytes * self.keys_seen(ctx) * self.kv_heads * (self.dim + self.vdim)

    def mixer_flops(self, n: int) -> int:
        """FLOPs of a prompt of ``n`` positions outside the projections."""
        if self.beside is not None:
            return dataclasses.replace(self, beside=None).mixer_flops(n) + self.beside.mixer_flops(n)
        if self.mixer in ("mlstm", "ssd"):    # the recurrence: state update and read of every position
            return 4 * n * self.heads * self.dim * self.vdim
        if self.mixer == "channel_delta":     # two reads and the update
            return 6 * n * self.heads * self.dim * self.vdim
        if self.mixer == "latent":        # scores and values in the latent space
            return 2 * self.heads * (2 * self.kv_rank + self.rot_dim) * self.pairs_seen(n)
        return 2 * self.heads * (self.dim + self.vdim + (self.heads if self.talk else 0)) * self.pairs_seen(n)

    @property
    def conv_channels(self) -> int:
        """Channels of the convolution: keys, queries and values, or input, input maps and output maps."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def conv_pad(self) -> int:
        return 2 * self.kv_heads * self.dim_pad + self.heads * self.vdim_pad

    @property
    def projection_cols(self) -> int:
        """Columns of the fused input projection, heads padded."""
        if self.mixer == "latent":        # [unrotated queries | rotated queries | latent | rotated key | head gates]
            return self.heads * (self.dim_pad + self.rot_pad) + self.rank_pad + self.rot_pad + pad_to(self.heads, 8)
        if self.mixer == "channel_delta":     # [q | k | v | decays' inner | gate's inner | step sizes]
            return self.conv_pad + pad_to(self.decay_rank, 8) + pad_to(self.gate_rank, 8) + pad_to(self.heads, 8)
        if self.mixer == "ssd":               # [output maps | input maps | input | gate | step sizes]
            return self.conv_pad + self.heads * self.vdim_pad + pad_to(self.heads, 8)
        if self.beside is not None:
            return dataclasses.replace(self, beside=None).projection_cols + self.beside.projection_cols
        if self.kv_from >= 0:
            return self.heads * self.dim_pad
        g = self.heads * self.vdim_pad if self.out_gate else 0
        return self.heads * self.dim_pad + self.kv_heads * (self.dim_pad + self.vdim_pad) + g

    def params(self, hidden: int, active: bool = False) -> int:
        """Matrix weights of the layer; ``active``: those one token uses."""
        if self.mixer == "latent":
            n = hidden * (self.heads * (self.dim + self.rot_dim + self.vdim + 1) + self.kv_rank + self.rot_dim) + \
                self.heads * self.kv_rank * (self.dim + self.vdim)
        elif self.mixer == "channel_delta":
            o = self.heads * self.vdim
            n = hidden * (self.conv_channels + o + self.decay_rank + self.gate_rank + self.heads) + \
                self.heads * self.dim * self.decay_rank + o * self.gate_rank + self.conv * self.conv_channels
        elif self.mixer == "ssd":
            n = hidden * (self.conv_channels + 2 * self.heads * self.vdim + self.heads) + self.conv * self.conv_channels
        else:
            own = self.kv_heads if self.kv_from < 0 else 0
            n = hidden * (self.heads * (self.dim + self.vdim * (2 if self.out_gate else 1)) + own * (self.dim + self.vdim))
        if self.beside is not None:
            n += self.beside.params(hidden) + 2 * hidden
        n += (3 if self.ffn_act == "geglu" else 2) * hidden * self.ffn + (2 * hidden * self.heads if self.mixer == "mlstm" else 0)
        if self.moe is not None:
            m = self.moe
            n += hidden * (m.num_experts + m.identity) + 3 * hidden * (m.expert_ffn * (m.top_k if active else m.num_experts) + m.shared_ffn * m.n_shared)
        return n


# architectures whose every operator has a 32-bit kernel on the GPU
GPU_FP32_ARCHS = ("duponex", "rudorax", "kabavik", "bazulorn")


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass
class ModelSpec:
    name: str
    arch: str                         # llama | qwen3 | qwen3_moe | deepseek_v3 | deepseek_v41 | glm5_next | flint | loop_vl | tiny_moe | qwen3_vl | embedding | diffusion_lm | qwen35_text | gemma | duponex | rudorax | kabavik | bazulorn
    layers: int
    hidden: int
    heads: int
    kv_heads: int
    head_dim: int
    ffn: int
    vocab: int
    rope_theta: float = 10000.0
    rms_eps: float = 1e-6
    dtype: str = "bf16"               # storage / compute dtype of dense weights
    linear_format: str = "bf16"       # bf16 | fp8_block | nvfp4
    tie_embeddings: bool = False
    qk_norm: bool = False
    swiglu_mode: int = 0
    max_position: int = 131072
    eos_token_id: int | None = None
    moe: MoeSpec | None = None
    mla: MlaSpec | None = None
    mtp_layers: int = 0               # multi-token-prediction heads shipped with the checkpoint
    layer_specs: list[LayerSpec] | None = None    # per-layer sizes, for designs whose layers differ
    loop: tuple[int, int, int] | None = None      # (start, stop, times): these layers run ``times`` times in a row; ``layers`` counts every run
    extra: dict[str, Any] = field(default_factory=dict)

    @property
    def q_dim(self) -> int:
        return self.heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.kv_heads * self.head_dim

    @property
    def qkv_dim(self) -> int:
        return self.q_dim + 2 * self.kv_dim

    @property
    def elem_bytes(self) -> int:
        return 4 if self.dtype == "fp32" else 2

    @property
    def runs(self) -> list[int]:
        """Layer (index into ``layer_specs``) of every layer run, in order. A run has a cache or state of its own."""
        n = len(self.layer_specs)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def kv_geometry(self) -> list[tuple[int, int, int]] | None:
        """(kv heads, key width, value width) of every cache layer where the layers differ, None where one size serves
        all. Widths are padded to 16 elements, the alignment of the attention kernels' tiles; a run that keeps its past in a
        per-sequence state or reads another layer's cache has none. A latent layer caches one row per token, the latent and
        the rotated key part behind it; its values are the row's first columns."""
        if self.layer_specs is None:
            return None

        def size(l: LayerSpec) -> tuple[int, int, int]:
            if l.mixer == "latent":
                return 1, l.rank_pad + l.rot_pad, 0
            return (l.kv_heads, l.dim_pad, l.vdim_pad) if l.mixer == "attention" and l.kv_from < 0 else (0, 0, 0)
        return [size(self.layer_specs[i]) for i in self.runs]

    @property
    def side_dim(self) -> int:
        """Width of a layer's part of the per-layer token embeddings (0: the design has none)."""
        return int(self.extra.get(self.arch, {}).get("side_dim", 0))

    def run_params(self) -> int:
        """Matrix weights one token passes through in all layer runs (a looped layer counts every time)."""
        return sum(self.layer_specs[i].params(self.hidden, active=True) + 2 * self.hidden * self.side_dim for i in self.runs)

    def dense_param_count(self) -> int:
        if self.layer_specs is not None:
            return sum(l.params(self.hidden) + (2 * self.hidden + self.vocab) * self.side_dim for l in self.layer_specs) + (1 if self.tie_embeddings else 2) * self.vocab * self.hidden
        per_layer = self.hidden * self.qkv_dim + self.q_dim * self.hidden + 3 * self.hidden * self.ffn + 2 * self.hidden
        return self.layers * per_layer + (1 if self.tie_embeddings else 2) * self.vocab * self.hidden + self.hidden

    def decode_weight_bytes(self) -> int:
        """Bytes of weights read by one decode step (embedding row gathers excluded, lm_head
        included) -- the numerator of the reference's decode roofline (src/bench.rs:137-160)."""
        if self.layer_specs is not None:      # experts: those one token uses
            return self.elem_bytes * (self.run_params() + self.vocab * self.hidden)
        per_layer = self.hidden * self.qkv_dim + self.q_dim * self.hidden + 3 * self.hidden * self.ffn + 2 * self.hidden
        return 2 * (self.layers * per_layer + self.vocab * self.hidden + self.hidden)

    def to_json(self) -> dict[str, Any]:
        return dataclasses.asdict(self)


# ------------------------------------------------------------------------------------------
# named shapes (the benchmark configurations; random-init, no checkpoint needed)
# ------------------------------------------------------------------------------------------
def tiny_moe() -> ModelSpec:
    return ModelSpec(
        name="tiny-moe", arch="tiny_moe", layers=2, hidden=256, heads=4, kv_heads=2, head_dim=64, ffn=512,
        vocab=1024, rope_theta=1e4, rms_eps=1e-6, dtype="fp32",
        moe=MoeSpec(num_experts=8, top_k=2, expert_ffn=512, score="softmax", n_shared=1, shared_ffn=512))


def tiny_llama() -> ModelSpec:
    """Small dense shape with the production head geometry (head_dim 128, GQA 4:1) for tests."""
    return ModelSpec(name="tiny-llama", arch="llama", layers=2, hidden=512, heads=4, kv_heads=1, head_dim=128,
                     ffn=1024, vocab=2048, rope_theta=5e5, rms_eps=1e-5)


def llama3_8b() -> ModelSpec:
    return ModelSpec(name="llama3-8b-shape", arch="llama", layers=32, hidden=4096, heads=32, kv_heads=8,
                     head_dim=128, ffn=14336, vocab=128256, rope_theta=5e5, rms_eps=1e-5)


def llama3_70b() -> ModelSpec:
    return ModelSpec(name="llama3-70b-shape", arch="llama", layers=80, hidden=8192, heads=64, kv_heads=8,
                     head_dim=128, ffn=28672, vocab=128256, rope_theta=5e5, rms_eps=1e-5)


def deepseek_v3() -> ModelSpec:
    return ModelSpec(
        name="deepseek-v3-shape", arch="deepseek_v3", layers=61, hidden=7168, heads=128, kv_heads=128, head_dim=128,
        ffn=18432, vocab=129280, rope_theta=1e4, rms_eps=1e-6, linear_format="fp8_block", mtp_layers=1,
        mla=MlaSpec(q_lora_rank=1536, kv_lora_rank=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128),
        moe=MoeSpec(num_experts=256, top_k=8, expert_ffn=2048, score="noaux", n_shared=1, shared_ffn=2048,
                    n_groups=8, topk_groups=4, routed_scaling=2.5, first_dense_layers=3, dense_ffn=18432,
                    expert_format="fp8_block"))


def deepseek_v3_tiny() -> ModelSpec:
    """Same structure as :func:`deepseek_v3` (MLA + grouped noaux routing + MTP head) at test size."""
    return ModelSpec(
        name="deepseek-v3-tiny", arch="deepseek_v3", layers=3, hidden=256, heads=4, kv_heads=4, head_dim=128,
        ffn=512, vocab=1024, rope_theta=1e4, rms_eps=1e-6, mtp_layers=1,
        mla=MlaSpec(q_lora_rank=96, kv_lora_rank=64, qk_nope_dim=32, qk_rope_dim=16, v_head_dim=32),
        moe=MoeSpec(num_experts=16, top_k=4, expert_ffn=128, score="noaux", n_shared=1, shared_ffn=128,
                    n_groups=4, topk_groups=2, routed_scaling=2.5, first_dense_layers=1, dense_ffn=512))


def deepseek_v3_mini() -> ModelSpec:
    """DeepSeek-V3 attention geometry (kv_lora 512, rope 64, nope 128, v 128) with a handful of
    heads and layers: the smallest shape the MLA CUDA kernel serves."""
    return ModelSpec(
        name="deepseek-v3-mini", arch="deepseek_v3", layers=2, hidden=512, heads=4, kv_heads=4, head_dim=128,
        ffn=1024, vocab=2048, rope_theta=1e4, rms_eps=1e-6,
        mla=MlaSpec(q_lora_rank=256, kv_lora_rank=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128),
        moe=MoeSpec(num_experts=16, top_k=4, expert_ffn=256, score="noaux", n_shared=1, shared_ffn=256,
                    n_groups=4, topk_groups=2, routed_scaling=2.5, first_dense_layers=1, dense_ffn=1024))


def deepseek_v3_fp8_mini() -> ModelSpec:
    """:func:`deepseek_v3_mini` with the published quantisation of DeepSeek-V3: every projection and expert as E4M3
    codes with 128x128 block scales (activations quantised 1x128 inside the linears), plus one MTP module."""
    s = deepseek_v3_mini()
    s.name, s.layers, s.linear_format, s.mtp_layers = "deepseek-v3-fp8-mini", 3, "fp8_block", 1
    s.moe.expert_format = "fp8_block"
    return s


def qwen3_moe_235b() -> ModelSpec:
    return ModelSpec(
        name="qwen3-moe-235b-shape", arch="qwen3_moe", layers=94, hidden=4096, heads=64, kv_heads=4, head_dim=128,
        ffn=12288, vocab=151936, rope_theta=1e6, rms_eps=1e-6, qk_norm=True,
        moe=MoeSpec(num_experts=128, top_k=8, expert_ffn=1536, score="softmax", expert_format="nvfp4"))


def qwen3_moe_tiny() -> ModelSpec:
    return ModelSpec(
        name="qwen3-moe-tiny", arch="qwen3_moe", layers=2, hidden=512, heads=4, kv_heads=1, head_dim=128, ffn=1024,
        vocab=2048, rope_theta=1e6, rms_eps=1e-6, qk_norm=True,
        moe=MoeSpec(num_experts=16, top_k=4, expert_ffn=256, score="softmax"))


def tiny_vl() -> ModelSpec:
    """Small vision-language shape: the tiny dense decoder plus a vision tower (``extra["vision"]`` holds the
    fields of ``models.vision.VisionSpec``; ``extra["image_token_id"]`` marks the rows the tower fills)."""
    spec = tiny_llama()
    spec.name, spec.arch = "tiny-vl", "qwen3_vl"
    spec.extra = {"image_token_id": 2047,
                  "vision": {"hidden": 256, "heads": 2, "depth": 2, "intermediate": 512, "patch": 16, "temporal": 2,
                             "merge": 2, "out_hidden": spec.hidden, "pos_side": 16}}
    return spec


def tiny_minicpm() -> ModelSpec:
    """Small sliced-image vision-language shape: the tiny dense decoder plus a MiniCPM-V style tower
    (``extra["vision"]``: ``kind`` "minicpm" and the fields of ``models.minicpm_vision.MiniCpmVisionSpec``); a large
    image is shown whole and as tiles, each view wrapped in marker tokens."""
    spec = tiny_llama()
    spec.name, spec.arch = "tiny-minicpm", "qwen3_vl"
    spec.extra = {"image_token_id": 2047, "image_start_id": 2040, "image_end_id": 2041, "slice_start_id": 2042, "slice_end_id": 2043,
                  "newline_id": 10, "max_slices": 4, "slice_scale": 32,
                  "vision": {"kind": "minicpm", "hidden": 64, "heads": 2, "depth": 3, "intermediate": 96, "patch": 2, "channels": 3,
                             "image_size": 32, "insert_layer": 0, "out_hidden": spec.hidden}}
    return spec


def tiny_embed() -> ModelSpec:
    """Small bidirectional text encoder (embedding model): mean pooling, optional dense head, L2 normalisation."""
    spec = tiny_llama()
    spec.name, spec.arch = "tiny-embed", "embedding"
    spec.extra = {"bidirectional": True, "embed_dense": [1024, 256]}
    return spec


def tiny_diffusion() -> ModelSpec:
    """Small masked-diffusion language model: a bidirectional decoder stack that denoises a canvas of mask tokens."""
    spec = tiny_llama()
    spec.name, spec.arch = "tiny-diffusion", "diffusion_lm"
    spec.extra = {"bidirectional": True, "mask_token_id": 2046}
    return spec


def tiny_hybrid() -> ModelSpec:
    """Small hybrid shape: gated-delta-net mixers with full attention in every fourth layer."""
    spec = tiny_llama()
    spec.name, spec.arch, spec.layers = "tiny-hybrid", "qwen35_text", 4
    spec.extra = {"gdn": {"v_heads": 4, "k_heads": 2, "full_attention_interval": 4}}
    return spec


def qwen3_moe_fp4_tiny() -> ModelSpec:
    """The tiny MoE shape with NVFP4 experts (decode reads the packed experts, prefill their BF16 expansion)."""
    spec = qwen3_moe_tiny()
    spec.name = "qwen3-moe-fp4-tiny"
    spec.moe.expert_format = "nvfp4"
    return spec


def tiny_gemma() -> ModelSpec:
    """Small Gemma-layout shape: five local layers (window 48) per global layer, tanh-GELU gate, soft-capped logits."""
    spec = tiny_llama()
    spec.name, spec.arch, spec.layers = "tiny-gemma", "gemma", 6
    spec.qk_norm, spec.swiglu_mode, spec.tie_embeddings, spec.rope_theta = True, 2, True, 1e6
    spec.extra = {"gemma": {"window": 48, "global_every": 6, "local_rope_theta": 1e4, "final_softcap": 30.0}}
    return spec


def deepseek_v41_tiny() -> ModelSpec:
    """Small DeepSeek-V4.1-style shape: four hyper-connection streams, a latent mixer with an FP8 window ring (window 32),
    one top-k sparse layer with a pooled indexer, n-gram memory rows in the first layer, shared + routed experts with
    square-root-soft-plus routing after a dense first layer."""
    return ModelSpec(
        name="deepseek-v41-tiny", arch="deepseek_v41", layers=3, hidden=256, heads=4, kv_heads=1, head_dim=128, ffn=512,
        vocab=2048, rope_theta=1e4, rms_eps=1e-6,
        moe=MoeSpec(num_experts=8, top_k=2, expert_ffn=128, score="sqrt_softplus", n_shared=1, shared_ffn=128,
                    routed_scaling=1.5, first_dense_layers=1, dense_ffn=512),
        extra={"v41": {"hc_mult": 4, "hc_iters": 3, "hc_eps": 1e-6, "q_lora": 128, "rope_tail": 32, "window": 32,
                       "o_groups": 2, "o_rank": 128, "sparse_layers": [1], "index_topk": 4,
                       "engram": {"layers": [0], "ngram": 3, "heads": 2, "compressed_vocab": 512, "table_rows": 509,
                                  "cache_rows": 256}}})


def flint_tiny() -> ModelSpec:
    """Small Flint-style shape: local layers (window 33, rotary) and global layers without positions, QK-norm, a
    learnable soft-max sink per head, two dense layers then sigmoid-routed experts with a shared expert."""
    return ModelSpec(
        name="flint-tiny", arch="flint", layers=5, hidden=512, heads=4, kv_heads=1, head_dim=128, ffn=1024, vocab=2048,
        rope_theta=1e4, rms_eps=1e-6, qk_norm=True,
        moe=MoeSpec(num_experts=8, top_k=2, expert_ffn=128, score="sigmoid", n_shared=1, shared_ffn=256,
                    first_dense_layers=2, dense_ffn=1024),
        extra={"flint": {"window": 33, "no_rope_layers": [0, 1, 4]}})


def _loop_spec(name: str, hidden: int, heads: int, ffn: int, vocab: int, per_stack: int, h_cycles: int, l_cycles: int,
               original_max: int) -> ModelSpec:
    return ModelSpec(
        name=name, arch="loop_vl", layers=h_cycles * (l_cycles + 1) * per_stack, hidden=hidden, heads=heads, kv_heads=heads,
        head_dim=128, ffn=ffn, vocab=vocab, rope_theta=1e4, rms_eps=1e-6,
        extra={"hrm": {"layers_per_stack": per_stack, "h_cycles": h_cycles, "l_cycles": l_cycles,
                       "embedding_scale": float(hidden) ** 0.5,
                       "yarn": {"factor": 2.0, "original_max": original_max, "beta_fast": 32.0, "beta_slow": 1.0}}})


def loop_tiny() -> ModelSpec:
    """Small looped two-stack decoder: two weight stacks of 2 layers, 2 H cycles of 3 L calls + 1 H call = 16 cache
    layers, gated full attention, YaRN positions."""
    return _loop_spec("loop-tiny", 256, 2, 512, 2048, per_stack=2, h_cycles=2, l_cycles=3, original_max=64)


def loopvl_text() -> ModelSpec:
    """The published LoopVL text geometry: 1536 hidden, 12 heads, two stacks of 16 layers applied 2 x (3 + 1) times
    (128 cache layers), vocabulary 65536."""
    return _loop_spec("loopvl-text-shape", 1536, 12, 4096, 65536, per_stack=16, h_cycles=2, l_cycles=3, original_max=4096)


def _duponex_spec_of(name: str, hidden: int, vocab: int, layers: list[LayerSpec], streams: int, residual_mult: float,
                     embed_scale: float, eps: float) -> ModelSpec:
    if not layers:
        raise ConfigError("a Duponex model needs at least one layer")
    mixing = [l for l in layers if l.v_mix]
    if any((l.kv_heads, l.vdim) != (mixing[0].kv_heads, mixing[0].vdim) for l in mixing):
        raise ConfigError("layers that mix values need the same number and width of value heads")
    for l in layers:
        if l.heads % l.kv_heads:
            raise ConfigError("heads must be a multiple of kv_heads")
        if min(l.heads, l.kv_heads, l.dim, l.vdim) < 1 or l.chunk < 0 or not l.scale > 0:
            raise ConfigError(f"unusable mixer sizes {l}")
    if not 1 <= streams <= 16:
        raise ConfigError(f"{streams} residual streams (1 to 16 are supported)")
    wide = max(layers, key=lambda l: l.heads * l.dim)
    return ModelSpec(
        name=name, arch="duponex", layers=len(layers), hidden=hidden, heads=wide.heads, kv_heads=wide.kv_heads, head_dim=wide.dim,
        ffn=max(l.ffn for l in layers), vocab=vocab, rms_eps=eps, layer_specs=layers,
        extra={"duponex": {"streams": streams, "residual_mult": residual_mult, "embed_scale": embed_scale}})


def duponex_tiny() -> ModelSpec:
    """Small Duponex shape whose layers differ: three residual streams, attention inside blocks of 72 or 40 positions,
    unequal key and value widths, one layer without value mixing and one without a feed-forward."""
    layer = dict(heads=4, kv_heads=2, dim=32, vdim=40, scale=0.2, v_mix=True, chunk=72, ffn=192)
    return _duponex_spec_of("duponex-tiny", 160, 512, [LayerSpec(**layer), LayerSpec(**dict(layer, heads=6, dim=48, chunk=40)),
                                                       LayerSpec(**dict(layer, v_mix=False, vdim=16, kv_heads=1)),
                                                       LayerSpec(**dict(layer, ffn=0))],
                            streams=3, residual_mult=0.5, embed_scale=4.0, eps=1e-5)


def duponex_8b() -> ModelSpec:
    """Duponex layers at the size of an 8-billion-parameter decoder (random weights, for measurements): 4096 wide, 32 / 8
    heads of 128, blocks of 2048 positions, four residual streams."""
    layers = [LayerSpec(heads=32, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, v_mix=True, chunk=2048, ffn=14336) for _ in range(8)]
    return _duponex_spec_of("duponex-8b-shape", 4096, 128256, layers, streams=4, residual_mult=0.5, embed_scale=8.0, eps=1e-5)


def duponex_2b() -> ModelSpec:
    """As :func:`duponex_8b` at 2048 wide: 16 / 4 heads of 128, 16 layers."""
    layers = [LayerSpec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, v_mix=True, chunk=2048, ffn=8192) for _ in range(16)]
    return _duponex_spec_of("duponex-2b-shape", 2048, 65536, layers, streams=4, residual_mult=0.5, embed_scale=8.0, eps=1e-5)


def _rudorax_spec_of(name: str, hidden: int, vocab: int, layers: list[LayerSpec], embed_scale: float, eps: float,
                     loop: tuple[int, int, int] | None = None, softcap: float = 0.0) -> ModelSpec:
    if not layers:
        raise ConfigError("a Rudorax model needs at least one layer")
    for l in layers:
        if min(l.heads, l.kv_heads, l.dim, l.vdim) < 1 or l.heads % l.kv_heads or l.window < 0 or not l.scale > 0:
            raise ConfigError(f"unusable mixer sizes {l}")
        if l.rope is not None and (l.rope.dims % 2 or not 0 < l.rope.dims <= l.dim or not l.rope.base > 1):
            raise ConfigError(f"unusable rotation {l.rope} of heads of {l.dim}")
        if l.mixer == "mlstm" and (not l.gate_cap > 0 or l.kv_heads != l.heads):
            raise ConfigError("a matrix memory needs a positive gate cap and one key head per query head")
        m = l.moe
        if m is not None and (m.num_experts < 1 or m.identity < 0 or not 1 <= m.top_k <= min(m.num_experts + m.identity, 32) or m.expert_ffn < 1):
            raise ConfigError(f"unusable experts {m}")
    if loop is not None and not (0 <= loop[0] <= loop[1] <= len(layers) and loop[2] >= 1):
        raise ConfigError(f"loop {loop} outside the layers")
    wide = max(layers, key=lambda l: l.heads * l.dim)
    spec = ModelSpec(
        name=name, arch="rudorax", layers=len(layers), hidden=hidden, heads=wide.heads, kv_heads=wide.kv_heads, head_dim=wide.dim,
        ffn=0, vocab=vocab, rms_eps=eps, qk_norm=True, layer_specs=layers, loop=loop,
        extra={"rudorax": {"embed_scale": embed_scale, "softcap": softcap}})
    spec.layers = len(spec.runs)
    return spec


def rudorax_tiny() -> ModelSpec:
    """Small Rudorax shape: windowed attention with sinks and scaled rotary positions, a matrix-memory layer, layers run
    twice, experts with identity outputs and a shared expert."""
    moe = MoeSpec(num_experts=6, top_k=3, expert_ffn=72, identity=2, n_shared=1, shared_ffn=104)
    attn = dict(heads=4, kv_heads=2, dim=32, vdim=40, scale=0.2, window=72, sink=True, out_gate=False, moe=moe,
                rope=RopeSpec(base=1e4, dims=24, factor=2.0, original=256))
    mem = dict(heads=3, kv_heads=3, dim=24, vdim=48, scale=24 ** -0.5, mixer="mlstm", gate_cap=10.0, moe=moe)
    return _rudorax_spec_of("rudorax-tiny", 160, 512, [LayerSpec(**attn), LayerSpec(**mem), LayerSpec(**dict(attn, kv_heads=1, window=40)),
                                                       LayerSpec(**dict(attn, moe=None))],
                            embed_scale=4.0, eps=1e-5, loop=(1, 3, 2), softcap=20.0)


def _rudorax_bench(name: str, hidden: int, heads: int, kv_heads: int, experts: int, ff: int, vocab: int) -> ModelSpec:
    moe = MoeSpec(num_experts=experts, top_k=8, expert_ffn=ff, identity=experts // 8, n_shared=1, shared_ffn=ff)
    attn = LayerSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, window=2048, sink=True, out_gate=False, moe=moe,
                     rope=RopeSpec(base=1e6, dims=128, factor=4.0, original=8192))
    mem = LayerSpec(heads=hidden // 256, kv_heads=hidden // 256, dim=128, vdim=256, scale=128 ** -0.5, mixer="mlstm", gate_cap=15.0, moe=moe)
    return _rudorax_spec_of(name, hidden, vocab, [attn, mem, attn, mem], embed_scale=8.0, eps=1e-5, loop=(1, 3, 2), softcap=30.0)


def rudorax_2k() -> ModelSpec:
    """Rudorax layers 2048 wide (random weights, for measurements): 16 / 4 attention heads of 128, 8 memories of 128 x 256,
    64 experts of 768 and 8 identity outputs, top 8, six layer runs."""
    return _rudorax_bench("rudorax-2k-shape", 2048, 16, 4, 64, 768, 65536)


def rudorax_4k() -> ModelSpec:
    """As :func:`rudorax_2k` at 4096: 32 / 8 heads, 16 memories, 64 experts of 1536."""
    return _rudorax_bench("rudorax-4k-shape", 4096, 32, 8, 64, 1536, 128256)


def _kabavik_spec_of(name: str, hidden: int, vocab: int, layers: list[LayerSpec], embed_scale: float, residual_mult: float,
                     logit_scale: float, side_dim: int, eps: float) -> ModelSpec:
    if not layers:
        raise ConfigError("a Kabavik model needs at least one layer")
    for i, l in enumerate(layers):
        if min(l.heads, l.kv_heads, l.dim, l.vdim) < 1 or l.heads % l.kv_heads or min(l.window, l.keep_first, l.ffn) < 0 or not l.scale > 0:
            raise ConfigError(f"layer {i}: unusable mixer sizes {l}")
        turned = l.rot_dim if l.mixer == "latent" else l.dim
        if l.rope is not None and (l.rope.dims % 2 or not 0 < l.rope.dims <= turned or not l.rope.base > 1 or not l.rope.factor > 0):
            raise ConfigError(f"layer {i}: unusable rotation {l.rope} of {turned} elements")
        if l.mixer == "latent" and (min(l.kv_rank, l.rot_dim) < 1 or l.rope is None or l.rope.halves):
            raise ConfigError(f"layer {i}: latent attention needs a latent and a part whose neighbours rotate")
        if l.q_temp is not None and l.q_temp[1] < 1:
            raise ConfigError(f"layer {i}: unusable query temperature {l.q_temp}")
        if l.kv_from >= 0:
            src = layers[l.kv_from] if l.kv_from < i else None
            if src is None or src.kv_from >= 0 or (src.mixer, src.kv_heads, src.dim, src.vdim) != (l.mixer, l.kv_heads, l.dim, l.vdim):
                raise ConfigError(f"layer {i}: cannot take keys and values from layer {l.kv_from}")
    wide = max(layers, key=lambda l: l.heads * l.dim)
    return ModelSpec(
        name=name, arch="kabavik", layers=len(layers), hidden=hidden, heads=wide.heads, kv_heads=wide.kv_heads, head_dim=wide.dim,
        ffn=max(l.ffn for l in layers), vocab=vocab, rms_eps=eps, qk_norm=True, layer_specs=layers,
        extra={"kabavik": {"embed_scale": embed_scale, "residual_mult": residual_mult, "logit_scale": logit_scale, "side_dim": side_dim}})


def kabavik_tiny() -> ModelSpec:
    """Small Kabavik shape: windowed attention that keeps the first positions, a layer that shares its keys and values,
    latent attention, and full attention with capped scores and a query temperature."""
    win = dict(heads=4, kv_heads=2, dim=32, vdim=40, scale=0.2, window=72, keep_first=5, qk_norm="row", bias=True, out_gate=False, ffn=192,
               ffn_act="geglu", rope=RopeSpec(base=1e4, dims=24, factor=2.0, halves=True))
    lat = dict(heads=3, kv_heads=1, dim=24, vdim=40, scale=0.2, mixer="latent", window=56, kv_rank=40, rot_dim=16, out_gate=False, ffn=192,
               ffn_act="geglu", rope=RopeSpec(base=1e4, dims=16, factor=4.0, original=128))
    cap = dict(heads=4, kv_heads=1, dim=48, vdim=16, scale=0.2, softcap=20.0, q_temp=(0.2, 64), bias=True, out_gate=False, ffn=192, ffn_act="geglu")
    return _kabavik_spec_of("kabavik-tiny", 160, 512, [LayerSpec(**win), LayerSpec(**lat), LayerSpec(**cap), LayerSpec(**dict(win, kv_from=0)),
                                                       LayerSpec(**dict(cap, ffn=0))],
                            embed_scale=1.0, residual_mult=0.8, logit_scale=0.5, side_dim=24, eps=1e-5)


def _bazulorn_spec_of(name: str, hidden: int, vocab: int, layers: list[LayerSpec], buckets: int, mul_prev: int, mul_cur: int,
                      eps: float) -> ModelSpec:
    if not layers:
        raise ConfigError("a Bazulorn model needs at least one layer")
    if buckets < 1 or min(mul_prev, mul_cur) < 0 or max(mul_prev, mul_cur) * vocab >= 1 << 62:
        raise ConfigError("unusable bigram table")
    for i, l in enumerate(layers):
        for m in [l] + ([l.beside] if l.beside is not None else []):
            if min(m.heads, m.kv_heads, m.dim, m.vdim) < 1 or m.heads % m.kv_heads or m.ffn < 0 or not m.scale > 0:
                raise ConfigError(f"layer {i}: unusable mixer sizes {m}")
            if m.mixer in ("channel_delta", "ssd") and not 1 <= m.conv <= 8:
                raise ConfigError(f"layer {i}: convolutions have 1 to 8 taps, not {m.conv}")
            if m.mixer == "ssd" and (m.norm_groups < 1 or m.heads * m.vdim % m.norm_groups):
                raise ConfigError(f"layer {i}: {m.heads * m.vdim} outputs in {m.norm_groups} equal parts")
        if l.beside is not None and l.window < 1:
            raise ConfigError(f"layer {i}: unusable window {l.window}")
        if l.mixer == "channel_delta":        # until a checkpoint says otherwise
            l.decay_rank, l.gate_rank = l.decay_rank or l.dim, l.gate_rank or l.vdim
    wide = max(layers, key=lambda l: l.heads * l.dim)
    return ModelSpec(
        name=name, arch="bazulorn", layers=len(layers), hidden=hidden, heads=wide.heads, kv_heads=wide.kv_heads, head_dim=wide.dim,
        ffn=max(l.ffn for l in layers), vocab=vocab, rms_eps=eps, tie_embeddings=True, layer_specs=layers,
        extra={"bazulorn": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}})


def bazulorn_tiny() -> ModelSpec:
    """Small Bazulorn shape: delta-rule layers with a dense and an expert feed-forward, attention with mixed heads beside a state space,
    a layer without a feed-forward."""
    moe = MoeSpec(num_experts=6, top_k=3, expert_ffn=72, score="biased_softmax", limit=1.5, n_shared=1, shared_ffn=104, shared_limit=2.5)
    delta = dict(mixer="channel_delta", heads=4, kv_heads=2, dim=24, vdim=40, scale=24 ** -0.5, conv=4, decay_rank=20, gate_rank=12, out_gate=False)
    ssd = LayerSpec(mixer="ssd", heads=6, kv_heads=3, dim=32, vdim=24, scale=1.0, conv=3, norm_groups=4, out_gate=False)
    both = dict(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.2, window=72, bias=True, sink_one=True, talk=True, v_norm=True, out_gate=False, beside=ssd)
    return _bazulorn_spec_of("bazulorn-tiny", 160, 512, [LayerSpec(**delta, ffn=200, ffn_act="geglu"), LayerSpec(**both, moe=moe),
                                                         LayerSpec(**delta, moe=moe), LayerSpec(**both)],
                             buckets=211, mul_prev=13, mul_cur=5, eps=1e-5)


def _bazulorn_bench(name: str, hidden: int, heads: int, kv_heads: int, experts: int, ff: int, vocab: int) -> ModelSpec:
    moe = MoeSpec(num_experts=experts, top_k=8, expert_ffn=ff, score="biased_softmax", limit=7.0, n_shared=1, shared_ffn=ff, shared_limit=7.0)
    delta = LayerSpec(mixer="channel_delta", heads=heads, kv_heads=heads, dim=128, vdim=128, scale=128 ** -0.5, conv=4, decay_rank=128, gate_rank=128,
                      out_gate=False, moe=moe)
    ssd = LayerSpec(mixer="ssd", heads=hidden // 64, kv_heads=8, dim=128, vdim=64, scale=1.0, conv=4, norm_groups=8, out_gate=False)
    both = LayerSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, window=1024, bias=True, sink_one=True, talk=True,
                     v_norm=True, out_gate=False, moe=moe, beside=ssd)
    return _bazulorn_spec_of(name, hidden, vocab, [delta, delta, both] * 2, buckets=65537, mul_prev=131, mul_cur=3, eps=1e-5)


def bazulorn_2k() -> ModelSpec:
    """Bazulorn layers 2048 wide (random weights, for measurements): 16 delta heads of 128, 16 / 4 attention heads of 128 beside 32
    state-space heads of 128 x 64, 64 experts of 768, top 8."""
    return _bazulorn_bench("bazulorn-2k-shape", 2048, 16, 4, 64, 768, 65536)


def bazulorn_4k() -> ModelSpec:
    """As :func:`bazulorn_2k` at 4096: 32 delta heads, 32 / 8 attention heads, 64 state-space heads, experts of 1536."""
    return _bazulorn_bench("bazulorn-4k-shape", 4096, 32, 8, 64, 1536, 128256)


def _kabavik_bench(name: str, hidden: int, heads: int, kv_heads: int, ff: int, vocab: int) -> ModelSpec:
    own = dict(out_gate=False, ffn=ff, ffn_act="geglu", scale=128 ** -0.5)
    win = LayerSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, window=2048, keep_first=64, qk_norm="row", bias=True,
                    rope=RopeSpec(base=1e6, dims=128, factor=2.0, halves=True), **own)
    lat = LayerSpec(heads=heads, kv_heads=1, dim=128, vdim=128, mixer="latent", window=2048, kv_rank=512, rot_dim=64,
                    rope=RopeSpec(base=1e6, dims=64, factor=4.0, original=8192), **own)
    cap = LayerSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, softcap=30.0, q_temp=(0.1, 4096), bias=True, **own)
    return _kabavik_spec_of(name, hidden, vocab, [win, lat, cap, dataclasses.replace(win, kv_from=0)] * 2, embed_scale=1.0, residual_mult=0.7,
                            logit_scale=0.5, side_dim=256, eps=1e-5)


def kabavik_2k() -> ModelSpec:
    """Kabavik layers 2048 wide (random weights, for measurements): 16 / 4 heads of 128, latents of 512 + 64, feed-forward 8192."""
    return _kabavik_bench("kabavik-2k-shape", 2048, 16, 4, 8192, 65536)


def kabavik_4k() -> ModelSpec:
    """As :func:`kabavik_2k` at 4096: 32 / 8 heads, feed-forward 14336."""
    return _kabavik_bench("kabavik-4k-shape", 4096, 32, 8, 14336, 128256)


def glm5_next_tiny() -> ModelSpec:
    """Small GLM-5-style shape: the hyper-connection program with every stage collapsing on its own pre-mix, top-k sparse
    attention with the pooled indexer in every layer, sigmoid routing with selection bias."""
    s = deepseek_v41_tiny()
    s.name, s.arch = "glm5-next-tiny", "glm5_next"
    s.moe.score, s.moe.routed_scaling = "noaux", 1.0
    s.extra = {"v41": dict(s.extra["v41"], hc_policy="own", sparse_layers=[0, 1, 2], engram=None)}
    return s


NAMED_SHAPES = {
    "tiny-gemma": tiny_gemma, "qwen3-moe-fp4-tiny": qwen3_moe_fp4_tiny, "tiny-hybrid": tiny_hybrid, "tiny-embed": tiny_embed, "tiny-diffusion": tiny_diffusion, "tiny-vl": tiny_vl, "tiny-minicpm": tiny_minicpm, "tiny-moe": tiny_moe, "tiny-llama": tiny_llama, "llama3-8b-shape": llama3_8b, "llama3-70b-shape": llama3_70b,
    "deepseek-v3-shape": deepseek_v3, "deepseek-v3-tiny": deepseek_v3_tiny, "deepseek-v3-mini": deepseek_v3_mini,
    "deepseek-v3-fp8-mini": deepseek_v3_fp8_mini, "deepseek-v41-tiny": deepseek_v41_tiny, "glm5-next-tiny": glm5_next_tiny, "flint-tiny": flint_tiny,
    "duponex-tiny": duponex_tiny, "duponex-8b-shape": duponex_8b, "duponex-2b-shape": duponex_2b,
    "rudorax-tiny": rudorax_tiny, "rudorax-2k-shape": rudorax_2k, "rudorax-4k-shape": rudorax_4k,
    "kabavik-tiny": kabavik_tiny, "kabavik-2k-shape": kabavik_2k, "kabavik-4k-shape": kabavik_4k,
    "bazulorn-tiny": bazulorn_tiny, "bazulorn-2k-shape": bazulorn_2k, "bazulorn-4k-shape": bazulorn_4k,
    "loop-tiny": loop_tiny, "loopvl-text-shape": loopvl_text,
    "qwen3-moe-235b-shape": qwen3_moe_235b, "qwen3-moe-tiny": qwen3_moe_tiny,
}


def named_shape(name: str) -> ModelSpec:
    if name not in NAMED_SHAPES:
        raise KeyError(f"unknown shape {name!r}; known: {sorted(NAMED_SHAPES)}")
    return NAMED_SHAPES[name]()


# ------------------------------------------------------------------------------------------
# config.json normalisation
# ------------------------------------------------------------------------------------------
class ConfigError(ValueError):
    pass


_ARCH_MAP = {
    "LlamaForCausalLM": "llama", "MistralForCausalLM": "llama", "Qwen2ForCausalLM": "qwen3",
    "Qwen3ForCausalLM": "qwen3", "Qwen3MoeForCausalLM": "qwen3_moe", "DeepseekV3ForCausalLM": "deepseek_v3",
    "DeepseekV2ForCausalLM": "deepseek_v3", "FlintForCausalLM": "flint", "LoopVLForConditionalGeneration": "loop_vl",
}


def _loopvl_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``LoopVLForConditionalGeneration`` (src/model_spec.rs:2273-2400 of the reference), text side: the looped two-stack
    decoder described by ``text_config`` (``hrm_text``); the vision encoder and projector of the checkpoint are not
    loaded."""
    t = cfg.get("text_config")
    if not isinstance(t, dict) or t.get("model_type") != "hrm_text":
        raise ConfigError("LoopVL text_config (hrm_text) missing")
    if cfg.get("quantization_config") is not None:
        raise ConfigError("LoopVL checkpoints are BF16 / F32")
    for key, want in (("hidden_act", "silu"), ("prefix_lm", True), ("tie_word_embeddings", False), ("attention_bias", False),
                      ("mlp_bias", False)):
        if t.get(key, want) != want:
            raise ConfigError(f"unsupported LoopVL setting {key}={t.get(key)!r}")
    rope = t.get("rope_parameters") or {}
    if rope.get("rope_type") != "yarn":
        raise ConfigError("LoopVL positions are YaRN-scaled")
    language = (cfg.get("loopvl_config") or {}).get("language") or {}
    for key in ("hidden_size", "num_attention_heads", "head_dim", "H_cycles", "L_cycles", "max_position_embeddings"):
        if key in language and language[key] != t.get(key):
            raise ConfigError(f"LoopVL language / text_config mismatch: {key}")
    if int(t["head_dim"]) != 128 or int(t["num_key_value_heads"]) != int(t["num_attention_heads"]):
        raise ConfigError("LoopVL heads are 128 wide without grouping")
    per, hc, lc = int(t["num_layers_per_stack"]), int(t["H_cycles"]), int(t["L_cycles"])
    if int(t.get("num_hidden_layers", hc * (lc + 1) * per)) != hc * (lc + 1) * per:
        raise ConfigError("num_hidden_layers differs from H_cycles * (L_cycles + 1) * num_layers_per_stack")
    spec = _loop_spec(name, int(t["hidden_size"]), int(t["num_attention_heads"]), int(t["intermediate_size"]), int(t["vocab_size"]),
                      per_stack=per, h_cycles=hc, l_cycles=lc, original_max=int(rope["original_max_position_embeddings"]))
    spec.rope_theta, spec.rms_eps = float(t.get("rope_theta", 10000.0)), float(t.get("rms_norm_eps", 1e-6))
    spec.max_position = int(t["max_position_embeddings"])
    spec.eos_token_id = t.get("eos_token_id")
    hrm = spec.extra["hrm"]
    hrm["embedding_scale"] = float(t.get("embedding_scale", hrm["embedding_scale"]))
    hrm["yarn"] = {"factor": float(rope["factor"]), "original_max": int(rope["original_max_position_embeddings"]),
                   "beta_fast": float(rope.get("beta_fast", 32.0)), "beta_slow": float(rope.get("beta_slow", 1.0))}
    return spec


def _flint_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``FlintForCausalLM`` (src/model_spec.rs:2723-2905 of the reference): sliding-window layers with rotary positions,
    the listed layers global and without positions, QK-norm, a learnable soft-max offset per head, dense FFNs in the
    ``mlp_only_layers`` prefix and sigmoid-routed experts with one shared expert after it."""
    for key, want in (("hidden_act", "silu"), ("attention_bias", False), ("router_score_function", "sigmoid"),
                      ("softmax_type", "learnable"), ("norm_topk_prob", True), ("use_sliding_window", True), ("decoder_sparse_step", 1)):
        if cfg.get(key, want) != want:
            raise ConfigError(f"unsupported Flint setting {key}={cfg.get(key)!r}")
    layers = int(cfg["num_hidden_layers"])
    no_rope = sorted(int(i) for i in cfg["no_rope_layer_indices"])
    if any(not (0 <= i < layers) for i in no_rope) or len(set(no_rope)) != len(no_rope):
        raise ConfigError("no_rope_layer_indices outside the layer range")
    types = cfg.get("layer_types")
    if types is not None:
        want = ["full_attention" if i in set(no_rope) else "sliding_attention" for i in range(layers)]
        if list(types) != want:
            raise ConfigError("layer_types disagree with no_rope_layer_indices (global layers carry no positions)")
    dense = sorted(int(i) for i in cfg.get("mlp_only_layers", []))
    if dense != list(range(len(dense))):
        raise ConfigError("mlp_only_layers must be a prefix of the layers")
    if int(cfg["head_dim"]) != 128:
        raise ConfigError("Flint heads are 128 wide")
    td = cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))
    dtype = {"bfloat16": "bf16", "float16": "f16", "float32": "fp32"}.get(td)
    if dtype is None:
        raise ConfigError(f"unsupported torch_dtype {td!r}")
    eos = cfg.get("eos_token_id")
    extra: dict[str, Any] = {"flint": {"window": int(cfg["sliding_window"]), "no_rope_layers": no_rope}}
    if isinstance(eos, list):
        extra["eos_token_ids"] = eos
        eos = eos[0] if eos else None
    heads, kv_heads = int(cfg["num_attention_heads"]), int(cfg["num_key_value_heads"])
    if heads % kv_heads:
        raise ConfigError("num_attention_heads must be a multiple of num_key_value_heads")
    return ModelSpec(
        name=name, arch="flint", layers=layers, hidden=int(cfg["hidden_size"]), heads=heads, kv_heads=kv_heads, head_dim=128,
        ffn=int(cfg["intermediate_size"]), vocab=int(cfg["vocab_size"]), rope_theta=float(cfg.get("rope_theta", 10000.0)),
        rms_eps=float(cfg.get("rms_norm_eps", 1e-6)), dtype=dtype, tie_embeddings=bool(cfg.get("tie_word_embeddings", False)),
        qk_norm=True, max_position=int(cfg.get("max_position_embeddings", 262144)), eos_token_id=eos,
        moe=MoeSpec(num_experts=int(cfg["num_experts"]), top_k=int(cfg["num_experts_per_tok"]),
                    expert_ffn=int(cfg["moe_intermediate_size"]), score="sigmoid", n_shared=1,
                    shared_ffn=int(cfg["shared_expert_intermediate_size"]), first_dense_layers=len(dense),
                    dense_ffn=int(cfg["intermediate_size"])),
        extra=extra)


def _duponex_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``"architecture": "Duponex"``: a list of layers, each with its own mixer sizes and feed-forward."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        if entry.get("type") != "attention":
            raise ConfigError(f"layer {i}: unsupported mixer {entry.get('type')!r}")
        m, mlp = entry["mixer"], entry.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ConfigError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
        layers.append(LayerSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                scale=float(m["scale"]), chunk=int((m.get("mask") or {}).get("size", 0)),
                                v_mix=bool(m.get("v_mix", False)), ffn=int(mlp["ff"]) if mlp is not None else 0))
    return _duponex_spec_of(name, int(cfg["width"]), int(cfg["vocab"]), layers, streams=int(cfg["streams"]),
                            residual_mult=float(cfg["residual_mult"]), embed_scale=float(cfg["embedding"]["scale"]),
                            eps=float(cfg["norm"]["eps"]))


def _rudorax_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``"architecture": "Rudorax"``: a list of layers with attention or matrix-memory mixers and expert feed-forwards, a range of
    which may run several times."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, moe = entry["mixer"], entry.get("mlp"), None
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise ConfigError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
            r, sh = mlp["router"], mlp.get("shared")
            moe = MoeSpec(num_experts=int(r["experts"]), top_k=int(r["top"]), expert_ffn=int(mlp["expert"]["ff"]), score="softmax",
                          identity=int(r.get("identity") or 0), n_shared=1 if sh else 0, shared_ffn=int(sh["ff"]) if sh else 0)
        sizes = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), moe=moe)
        if entry.get("type") == "attention":
            rot = m.get("rot")
            rope = None
            if rot is not None:
                sc = rot.get("scaling")
                rope = RopeSpec(base=float(rot["base"]), dims=int(rot["dims"]))
                if sc is not None:
                    rope = dataclasses.replace(rope, factor=float(sc["factor"]), original=int(sc["original"]), fast=float(sc["fast"]),
                                               slow=float(sc["slow"]))
            layers.append(LayerSpec(kv_heads=int(m["kv_heads"]), scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size", 0)),
                                    sink=True, rope=rope, out_gate=False, **sizes))
        elif entry.get("type") == "mlstm":
            layers.append(LayerSpec(kv_heads=sizes["heads"], scale=sizes["dim"] ** -0.5, mixer="mlstm", gate_cap=float(m["gate_cap"]), **sizes))
        else:
            raise ConfigError(f"layer {i}: unsupported mixer {entry.get('type')!r}")
    loop = cfg.get("loop")
    return _rudorax_spec_of(name, int(cfg["width"]), int(cfg["vocab"]), layers, embed_scale=float(cfg["embedding"]["scale"]),
                            eps=float(cfg["norm"]["eps"]), softcap=float(cfg.get("logit_softcap") or 0.0),
                            loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)


def _kabavik_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``"architecture": "Kabavik"``: a list of layers with windowed, latent or capped full attention, gated feed-forwards and a
    per-layer token input."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, kind = entry["mixer"], entry.get("mlp"), entry.get("type")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ConfigError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
        mask, rot = m.get("mask") or {}, m.get("rot")
        sizes = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), window=int(mask.get("size", 0)),
                     keep_first=int(mask.get("keep_first", 0)), kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else -1,
                     out_gate=False, ffn=int(mlp["ff"]) if mlp is not None else 0, ffn_act="geglu")
        rope = None
        if rot is not None:
            sc = rot.get("scaling") or {}
            rope = RopeSpec(base=float(rot["base"]), dims=int(rot["dims"]), factor=float(sc.get("factor", 1.0)), halves=kind == "attention")
            if kind == "latent_attention" and sc:
                rope = dataclasses.replace(rope, original=int(sc["original"]), fast=float(sc["fast"]), slow=float(sc["slow"]))
        if kind == "attention":
            layers.append(LayerSpec(kv_heads=int(m["kv_heads"]), qk_norm="row", bias=True, rope=rope, **sizes))
        elif kind == "attention_2":
            temp = m.get("q_temp")
            layers.append(LayerSpec(kv_heads=int(m["kv_heads"]), bias=True, softcap=float(m.get("softcap") or 0.0),
                                    q_temp=(float(temp["coef"]), int(temp["every"])) if temp else None, **sizes))
        elif kind == "latent_attention":
            layers.append(LayerSpec(kv_heads=1, mixer="latent", kv_rank=int(m["kv_rank"]), rot_dim=int(m["rot_dim"]), rope=rope, **sizes))
        else:
            raise ConfigError(f"layer {i}: unsupported mixer {kind!r}")
    side = cfg.get("token_side")
    return _kabavik_spec_of(name, int(cfg["width"]), int(cfg["vocab"]), layers, embed_scale=float(cfg["embedding"]["scale"]),
                            residual_mult=float(cfg["residual_mult"]), logit_scale=float(cfg["logit_scale"]),
                            side_dim=int(side["dim"]) if side else 0, eps=float(cfg["norm"]["eps"]))


def _bazulorn_moe(mlp: dict[str, Any], where: str) -> MoeSpec:
    r, sh = mlp["router"], mlp.get("shared")
    moe = MoeSpec(num_experts=int(r["experts"]), top_k=int(r["top"]), expert_ffn=int(mlp["expert"]["ff"]), score="biased_softmax",
                  limit=float(mlp["expert"]["limit"]), n_shared=1 if sh else 0, shared_ffn=int(sh["ff"]) if sh else 0,
                  shared_limit=float(sh["limit"]) if sh else 0.0)
    if moe.num_experts < 1 or not 1 <= moe.top_k <= min(moe.num_experts, 32) or moe.expert_ffn < 1 or not moe.limit > 0 or \
            (sh and (moe.shared_ffn < 1 or not moe.shared_limit > 0)):
        raise ConfigError(f"{where}: unusable experts {moe}")
    return moe


def _bazulorn_spec(cfg: dict[str, Any], name: str) -> ModelSpec:
    """``"architecture": "Bazulorn"``: a list of layers whose mixer is a channel-wise gated delta rule or windowed attention with
    mixed heads beside a state space, with dense or expert feed-forwards; bigrams are embedded beside tokens. The widths inside the
    decays' and the gate's matrix pairs are those of the checkpoint's tensors (:func:`read_model_spec`)."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, kind = entry["mixer"], entry.get("mlp"), entry.get("type")
        ff: dict[str, Any] = {}
        if mlp is not None:
            if mlp.get("kind") == "dense":
                ff = dict(ffn=int(mlp["ff"]), ffn_act="geglu")
            elif mlp.get("kind") == "moe":
                ff = dict(moe=_bazulorn_moe(mlp, f"layer {i}"))
            else:
                raise ConfigError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
        if kind == "channel_delta":
            layers.append(LayerSpec(mixer="channel_delta", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                                    vdim=int(m["vdim"]), scale=int(m["dim"]) ** -0.5, conv=int(m["conv"]), out_gate=False, **ff))
        elif kind == "parallel":
            a, s = m["left"], m["right"]
            right = LayerSpec(mixer="ssd", heads=int(s["heads"]), kv_heads=int(s["groups"]), dim=int(s["state"]), vdim=int(s["vdim"]), scale=1.0,
                              conv=int(s["conv"]), norm_groups=int(s["norm_groups"]), out_gate=False)
            layers.append(LayerSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                    scale=float(a["scale"]), window=int(a["mask"]["size"]), bias=True, sink_one=True, talk=True, v_norm=True,
                                    out_gate=False, beside=right, **ff))
        else:
            raise ConfigError(f"layer {i}: unsupported mixer {kind!r}")
    b = cfg["embedding"]["bigram"]
    return _bazulorn_spec_of(name, int(cfg["width"]), int(cfg["vocab"]), layers, buckets=int(b["buckets"]), mul_prev=int(b["mul_prev"]),
                             mul_cur=int(b["mul_cur"]), eps=float(cfg["norm"]["eps"]))


def _ranks_from_tensors(spec: ModelSpec, shape) -> None:
    """Widths inside the matrix pairs of channel_delta layers from the shapes of a checkpoint's tensors."""
    for i, l in enumerate(spec.layer_specs):
        if l.mixer == "channel_delta":
            try:
                l.decay_rank, l.gate_rank = int(shape(f"l{i}.mix.a1")[0]), int(shape(f"l{i}.mix.g1")[0])
            except KeyError as e:
                raise ConfigError(f"layer {i}: the checkpoint lacks {e}") from None


def spec_from_hf_config(cfg: dict[str, Any], name: str = "model") -> ModelSpec:
    """Normalise a Hugging Face ``config.json``. Hard checks mirror the reference's: SiLU
    activation only, 16-bit or 32-bit floats, no unsupported rope scaling for plain Llama."""
    if cfg.get("architecture") == "Duponex":
        return _duponex_spec(cfg, name)
    if cfg.get("architecture") == "Rudorax":
        return _rudorax_spec(cfg, name)
    if cfg.get("architecture") == "Kabavik":
        return _kabavik_spec(cfg, name)
    if cfg.get("architecture") == "Bazulorn":
        return _bazulorn_spec(cfg, name)
    archs = cfg.get("architectures") or []
    arch = next((_ARCH_MAP[a] for a in archs if a in _ARCH_MAP), None)
    if arch is None:
        raise ConfigError(f"unsupported architectures {archs}")
    if arch == "flint":
        return _flint_spec(cfg, name)
    if arch == "loop_vl":
        return _loopvl_spec(cfg, name)
    act = cfg.get("hidden_act", "silu")
    if act not in ("silu", "swish"):
        raise ConfigError(f"unsupported activation {act!r}")
    td = cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))
    dtype = {"bfloat16": "bf16", "float16": "f16", "float32": "fp32"}.get(td)
    if dtype is None:
        raise ConfigError(f"unsupported torch_dtype {td!r}")
    hidden = int(cfg["hidden_size"])
    heads = int(cfg["num_attention_heads"])
    kv_heads = int(cfg.get("num_key_value_heads", heads))
    head_dim = int(cfg.get("head_dim") or hidden // heads)
    if heads % kv_heads:
        raise ConfigError("num_attention_heads must be a multiple of num_key_value_heads")
    scaling = cfg.get("rope_scaling")
    extra: dict[str, Any] = {}
    if scaling:
        kind = scaling.get("rope_type", scaling.get("type"))
        if kind not in ("llama3", "yarn", "default", None):
            raise ConfigError(f"unsupported rope scaling {kind!r}")
        extra["rope_scaling"] = scaling
    quant = cfg.get("quantization_config") or {}
    linear_format = "bf16"
    if quant.get("quant_method") == "fp8" and quant.get("weight_block_size") == [128, 128]:
        linear_format = "fp8_block"
    elif quant.get("quant_algo") == "NVFP4" or quant.get("quant_method") == "modelopt":
        linear_format = "nvfp4"
    moe = None
    if arch == "qwen3_moe":
        moe = MoeSpec(num_experts=int(cfg["num_experts"]), top_k=int(cfg["num_experts_per_tok"]),
                      expert_ffn=int(cfg["moe_intermediate_size"]), score="softmax",
                      renormalize=bool(cfg.get("norm_topk_prob", True)),
                      expert_format=linear_format if linear_format != "bf16" else "bf16")
    mla = None
    if arch == "deepseek_v3":
        moe = MoeSpec(num_experts=int(cfg["n_routed_experts"]), top_k=int(cfg["num_experts_per_tok"]),
                      expert_ffn=int(cfg["moe_intermediate_size"]),
                      score="noaux" if cfg.get("topk_method", "noaux_tc") == "noaux_tc" else "softmax",
                      n_shared=int(cfg.get("n_shared_experts", 0)),
                      shared_ffn=int(cfg["moe_intermediate_size"]) * int(cfg.get("n_shared_experts", 0) or 0),
                      n_groups=int(cfg.get("n_group", 1)), topk_groups=int(cfg.get("topk_group", 1)),
                      routed_scaling=float(cfg.get("routed_scaling_factor", 1.0)),
                      renormalize=bool(cfg.get("norm_topk_prob", True)),
                      first_dense_layers=int(cfg.get("first_k_dense_replace", 0)),
                      dense_ffn=int(cfg["intermediate_size"]),
                      expert_format=linear_format)
        mla = MlaSpec(q_lora_rank=int(cfg.get("q_lora_rank") or 0), kv_lora_rank=int(cfg["kv_lora_rank"]),
                      qk_nope_dim=int(cfg["qk_nope_head_dim"]), qk_rope_dim=int(cfg["qk_rope_head_dim"]),
                      v_head_dim=int(cfg["v_head_dim"]))
    eos = cfg.get("eos_token_id")
    if isinstance(eos, list):
        extra["eos_token_ids"] = eos
        eos = eos[0] if eos else None
    return ModelSpec(
        name=name, arch=arch, layers=int(cfg["num_hidden_layers"]), hidden=hidden, heads=heads, kv_heads=kv_heads,
        head_dim=head_dim, ffn=int(cfg.get("intermediate_size", 0)), vocab=int(cfg["vocab_size"]),
        rope_theta=float(cfg.get("rope_theta", 10000.0)), rms_eps=float(cfg.get("rms_norm_eps", 1e-6)), dtype=dtype,
        linear_format=linear_format, tie_embeddings=bool(cfg.get("tie_word_embeddings", False)),
        qk_norm=arch in ("qwen3", "qwen3_moe"), max_position=int(cfg.get("max_position_embeddings", 131072)),
        eos_token_id=eos, moe=moe, mla=mla, mtp_layers=int(cfg.get("num_nextn_predict_layers", 0)), extra=extra)


def read_model_spec(model_dir: str | Path) -> ModelSpec:
    p = Path(model_dir)
    cfg = json.loads((p / "config.json").read_text())
    spec = spec_from_hf_config(cfg, name=p.name)
    if spec.layer_specs is not None and any(l.mixer == "channel_delta" for l in spec.layer_specs):
        from .loaders.safetensors_io import MappedCheckpoint
        if any(p.glob("*.safetensors")):
            ck = MappedCheckpoint(p)
            try:
                _ranks_from_tensors(spec, lambda n: ck.shape(n))
            finally:
                ck.close()
    return spec


# ------------------------------------------------------------------------------------------
# engine settings
# ------------------------------------------------------------------------------------------
@dataclass
class Settings:
    """Engine options shared by every entry point (CLI flags of the same names)."""
    device: int = 0
    capacity: int = 4096                  # tokens of KV per sequence the engine plans for
    chunk: int | None = None              # prefill chunk rows (planner-derived when None)
    device_budget_gib: float | None = None
    draft_model: str | None = None
    tree_builder: str = "waves"           # waves | serial | markov
    spec_budget: str = "chain"            # chain | tree16 | tree32 | tree64
    spec_graph: bool = True
    prefix_cache: bool = False
    kv_format: str = "bf16"               # bf16 | affine8
    kv_recent: int = 2048                 # affine8: tokens behind the newest that stay BF16 (groups older than that are sealed)
    runtime_dir: str | None = None
    dram_gb_s: float = 6550.0             # roofline denominators (measured on the target box)
    gemm_tflops: float = 1385.0
    verbose: bool = False
    tp: int = 1
    ep: int = 1
    max_batch: int = 64
    kv_block: int = 64
    kv_tokens: int | None = None          # tokens the whole KV pool holds (planner-derived when None)
    dtype: str | None = None              # compute dtype override: bf16 | fp32 (the checkpoint's when None)
    graph: bool = True

    def resolved_runtime_dir(self) -> Path:
        import os
        d = self.runtime_dir or os.environ.get("FLYINGFISH_RUNTIME_DIR") or str(Path.home() / ".flyingfish")
        return Path(d)
