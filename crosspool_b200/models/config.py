"""Decoder model shapes: typed view of a Hugging Face ``config.json`` plus named presets.

The attention side needs heads / KV heads / head_dim / RoPE / norms; the FFN side needs the MLP or
MoE description (that part is compiled into an :class:`crosspool_b200.ffn.FfnModelSpec` by the
architecture adapters). The reference reads the same fields through ``FfnSourceConfig``
(src/xpool/runtime/ffnagent/architecture.py:133-215) and ``SglangModelShape.load``
(src/xpool/integrations/sglang/topology.py).
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, replace
from pathlib import Path
from typing import Any


@dataclass(frozen=True)
class MlaShape:
    """Multi-head latent attention (DeepSeek-V2, GLM-4-MoE-Lite): queries optionally through a rank-``q_lora_rank``
    bottleneck; keys and values expanded per head from one ``kv_lora_rank`` latent plus a ``qk_rope_head_dim`` rotary
    key shared by all heads."""

    q_lora_rank: int            # 0: a plain query projection
    kv_lora_rank: int
    qk_nope_head_dim: int
    qk_rope_head_dim: int
    v_head_dim: int

    @property
    def qk_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim


@dataclass(frozen=True)
class RotaryScaling:
    """Rotary frequencies for contexts beyond ``original`` tokens: wavelengths above ``original / low`` are stretched by
    ``factor``, those below ``original / high`` are kept, the ones between blend linearly in ``original / wavelength``.
    ``original`` = 0: all of them are stretched by ``factor``."""

    factor: float
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of a vector, paired (i, i + dims / 2), or (2 i, 2 i + 1) with
    ``interleaved``: the pair at position p turns by ``p * f_i``, ``f_i = base ** (-2 i / dims)``, scaled where there is a
    ``scaling``."""

    dims: int
    base: float
    scaling: RotaryScaling | None = None
    interleaved: bool = False


def ceil8(n: int) -> int:
    return (n + 7) // 8 * 8


# (query/key width, value width) of the tensor-core attention kernels, narrowest first
ATTENTION_SHAPES = ((64, 64), (128, 64), (128, 128), (192, 128))


def attention_shape(dim: int, vdim: int) -> tuple[int, int] | None:
    """Padded head widths of the tensor-core attention kernels, None when no kernel covers the sizes."""
    if vdim % 8:
        return None
    for dq, dv in ATTENTION_SHAPES:
        if dim <= dq and vdim <= dv:
            return dq, dv
    return None


@dataclass(frozen=True)
class LatentMixer:
    """Latent attention as a layer's mixer: per-head keys and values are linear maps of one cached ``kv_rank`` latent,
    plus one rotary key part of ``rot_dim`` shared by the heads. The output is gated by a sigmoid, one number per head or, with
    ``gate_elems``, per element. ``q_rank`` > 0: queries come from a normed latent of their own of that size. ``window`` > 0: a
    token sees itself and the ``window - 1`` tokens before it."""

    heads: int
    dim: int                    # unrotated query/key dimensions per head
    rot_dim: int                # rotated query/key dimensions per head
    vdim: int
    kv_rank: int
    rot: RotarySpec
    scale: float
    q_rank: int = 0
    window: int = 0
    gate_elems: bool = False
    kind: str = "latent_attention"

    @property
    def cache_width(self) -> int:
        """Elements of one token's cache row: latent and rotated key, padded to whole 16-element tensor-core steps."""
        return (self.kv_rank + self.rot_dim + 15) // 16 * 16

    @property
    def cache_rows(self) -> tuple[tuple[int, int], ...]:
        return ((1, self.cache_width),)

    @property
    def state_elems(self) -> int:
        return 0

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def gate_features(self) -> int:
        return self.out_features if self.gate_elems else self.heads

    def visible(self, length: int) -> int:
        """Bound on the tokens a query at the end of ``length`` tokens sees."""
        return min(length, self.window) if self.window else length

    def param_count(self, hidden: int) -> int:
        q = self.heads * (self.dim + self.rot_dim)
        q = self.q_rank * (hidden + 1 + q) if self.q_rank else hidden * q
        return (q + hidden * (self.kv_rank + self.rot_dim + self.gate_features + self.out_features) + self.kv_rank
                + self.kv_rank * self.heads * (self.dim + self.vdim))


class _RecurrentMixer:
    """Common part of mixers that keep one fp32 ``dim x vdim`` state per head and sequence instead of cached tokens."""

    cache_rows: tuple[tuple[int, int], ...] = ()

    @property
    def cache_width(self) -> int:
        return 0

    @property
    def state_shape(self) -> tuple[int, ...]:
        return (self.heads, self.dim, self.vdim)

    @property
    def state_elems(self) -> int:
        return math.prod(self.state_shape)

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class LinearMixer(_RecurrentMixer):
    """Decayed linear attention (one fp32 ``dim x vdim`` state per head and sequence, a fixed decay per head), its heads
    normalised together and gated."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    kind: str = "lightning"

    def param_count(self, hidden: int) -> int:
        return hidden * self.heads * (2 * self.dim + 3 * self.vdim) + self.out_features


@dataclass(frozen=True)
class GroupedMixer:
    """Grouped-query attention: ``heads`` query heads share ``kv_heads`` cached keys and values, scores saturate at +-``softcap``
    (0: they do not).

    ``norm``: queries and keys are RMS-normed per head, with a ``"weight"`` or as ``"unit"`` vectors of root mean square one
    (``""``: not at all). ``biases``: of the projections. ``gate``: a sigmoid gates the output, one number per ``"head"`` or
    ``"element"`` (``""``: none). ``conv``: queries, keys and values pass a causal convolution of that many taps before anything
    else (0: none). ``window``: a token sees itself and the ``window - 1`` tokens before it, and the first ``keep_first`` tokens
    of the sequence (0: all before it). ``kv_from``: the layer has no keys and values of its own and reads those that layer
    caches. ``sink``: a number per head joins the softmax's sum and has no value. ``sigmoid``: no softmax, a token's weight is
    the sigmoid of its score plus a number per head. ``pool`` > 0: beside its window a token sees the mean key and value of
    every block of that many tokens that lies wholly behind the window. ``tied``: values are the projected keys."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0
    norm: str = "weight"
    biases: bool = True
    gate: str = "head"
    conv: int = 0
    rot: RotarySpec | None = None
    window: int = 0
    keep_first: int = 0
    kv_from: int | None = None
    sink: bool = False
    sigmoid: bool = False
    pool: int = 0
    tied: bool = False
    kind: str = "grouped_attention"

    @property
    def head_norms(self) -> bool:
        return bool(self.norm)

    @property
    def gate_features(self) -> int:
        return {"head": self.heads, "element": self.out_features, "": 0}[self.gate]

    def pool_page(self, page_size: int) -> int:
        """Rows for block means beside every page of ``page_size`` tokens: at least as many as blocks end in it, so that block b
        lies beside page ``b // pool_page`` of its sequence; a power of two of at least eight (the copies of the tensor-core
        kernels bring eight rows)."""
        n = 8
        while n * self.pool < page_size:
            n *= 2
        return n

    def pool_shapes(self, page_size: int) -> tuple[tuple[int, int, int], ...]:
        """Block means beside one page, keys and values: (rows, heads, elements per head)."""
        return tuple((self.pool_page(page_size), *r) for r in self.row_shapes) if self.pool else ()

    @property
    def row_shapes(self) -> tuple[tuple[int, int], ...]:
        """(heads, elements per head) of a token's key and value rows, padded to the widths of the tensor-core kernels
        where one covers the sizes."""
        return tuple((self.kv_heads, n) for n in attention_shape(self.dim, self.vdim) or (ceil8(self.dim), ceil8(self.vdim)))

    @property
    def cache_rows(self) -> tuple[tuple[int, int], ...]:
        return () if self.kv_from is not None else self.row_shapes

    @property
    def cache_width(self) -> int:
        return sum(h * n for h, n in self.cache_rows)

    @property
    def state_elems(self) -> int:
        return 0

    @property
    def conv_channels(self) -> int:
        """Channels that pass the convolution: queries, and the layer's own keys and values."""
        return self.heads * self.dim + (0 if self.kv_from is not None else self.kv_heads * (self.dim + self.vdim))

    @property
    def conv_state_elems(self) -> int:
        return self.conv * self.conv_channels

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    def visible(self, length: int) -> int:
        """Bound on the tokens a query at the end of ``length`` tokens sees."""
        blocks = max(0, length - self.window) // self.pool if self.pool else 0
        return min(length, self.window + self.keep_first) + blocks if self.window else length

    def param_count(self, hidden: int) -> int:
        rows = self.heads * self.dim
        if self.kv_from is None:
            rows += self.kv_heads * (self.dim + (0 if self.tied else self.vdim))
        n = rows * (hidden + int(self.biases)) + hidden * (self.gate_features + self.out_features) + self.conv_state_elems
        n += self.heads * (int(self.sink) + int(self.sigmoid)) + (2 * self.dim if self.norm == "weight" else 0)
        return n + (hidden if self.biases and self.gate == "head" else 0)        # (with a bias behind the output map as well)


@dataclass(frozen=True)
class GatedLinearMixer(_RecurrentMixer):
    """Linear attention whose state decays per key channel, ``sigmoid(z) ** (1 / tau)`` with ``z`` a low-rank map of the
    input; every head's output is RMS-normed and gated. ``rank`` of the map belongs to the checkpoint (0: unknown)."""

    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 0
    kind: str = "gated_linear"

    def param_count(self, hidden: int) -> int:
        return (hidden * self.heads * (2 * self.dim + 3 * self.vdim) + self.vdim + self.rank * (hidden + self.heads * self.dim)
                + self.heads * self.dim)


@dataclass(frozen=True)
class DeltaMixer(_RecurrentMixer):
    """Gated delta rule: the state decays by one factor per head and token, and a write replaces the share ``beta`` of what
    it holds under the key. Queries, keys and values pass a causal convolution of ``conv`` taps; ``kv_heads`` queries and
    keys (unit vectors) are shared by the ``heads`` values."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    kind: str = "delta"

    @property
    def conv_channels(self) -> int:
        """Channels that pass the convolution: queries, keys, values."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def conv_state_elems(self) -> int:
        """Convolution inputs a sequence carries (a ring of ``conv`` tokens: the ones behind, and the token at hand)."""
        return self.conv * self.conv_channels

    def param_count(self, hidden: int) -> int:
        return (hidden * (self.conv_channels + 2 * self.heads + 2 * self.out_features) + self.conv * self.conv_channels
                + 2 * self.heads + self.vdim)


@dataclass(frozen=True)
class MemoryMixer(_RecurrentMixer):
    """Matrix memory with exponential gates: the state decays by a forget gate and takes a key's value in by an input gate,
    both as logarithms that saturate at +-``gate_cap`` before the forget gate's sigmoid; a vector of decayed keys normalises
    what is read, and a running maximum of the logarithms scales all three."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float
    kind: str = "mlstm"

    @property
    def head_state(self) -> int:
        """fp32 elements of a head: the matrix, the key sum and the maximum, rounded up to whole 16 bytes."""
        return (self.dim * self.vdim + self.dim + 1 + 3) // 4 * 4

    @property
    def state_shape(self) -> tuple[int, ...]:
        return (self.heads, self.head_state)

    def param_count(self, hidden: int) -> int:
        return hidden * self.heads * (2 * self.dim + 3 * self.vdim + 2) + self.out_features + 2 * self.heads


@dataclass(frozen=True)
class ParallelMixer:
    """Two mixers that read the same input; half the sum of their outputs, each RMS-normed over the model width first."""

    left: GroupedMixer
    right: GatedLinearMixer
    kind: str = "parallel"

    @property
    def cache_rows(self) -> tuple[tuple[int, int], ...]:
        return self.left.cache_rows

    @property
    def cache_width(self) -> int:
        return self.left.cache_width

    @property
    def state_elems(self) -> int:
        return self.right.state_elems

    @property
    def out_features(self) -> int:
        return self.left.out_features + self.right.out_features

    def param_count(self, hidden: int) -> int:
        return self.left.param_count(hidden) + self.right.param_count(hidden) + 2 * hidden


def sub_mixers(m) -> tuple:
    """The mixers that do the work: both sides of a parallel pair, else the mixer itself."""
    return (m.left, m.right) if isinstance(m, ParallelMixer) else (m,)


Mixer = LatentMixer | LinearMixer | GroupedMixer | GatedLinearMixer | DeltaMixer | MemoryMixer | ParallelMixer


GLU_ALPHA = 1.702    # slope of the sigmoid in the clamped gated activation


# g sigmoid(alpha g (1 + cubic g^2)): the tanh form of gelu as a gated activation
GELU_ALPHA = 2.0 * math.sqrt(2.0 / math.pi)
GELU_CUBIC = 0.044715


@dataclass(frozen=True)
class MoeSpec:
    """Routed FFN of a layered decoder: ``experts`` gated (silu) FFNs of ``ff`` features and ``identity`` experts that return
    their input; a token takes ``top`` of them by softmax score plus a correction, weighted by their scores normalised to
    ``scale``. ``shared_ff`` > 0: one more expert for every token, its output times a sigmoid per token with ``shared_gate``.
    ``relu2``: experts are ungated, ``down(max(up x, 0)^2)``. ``logit_choice``: the router has biases, its largest logits are
    chosen and their softmax weighs them (no correction)."""

    experts: int
    top: int
    ff: int
    identity: int = 0
    scale: float = 1.0
    shared_ff: int = 0
    shared_gate: bool = True
    relu2: bool = False
    logit_choice: bool = False

    @property
    def maps(self) -> int:
        """Matrices of an expert."""
        return 2 if self.relu2 else 3

    @property
    def folds_shared(self) -> bool:
        """The shared expert runs as one more routed expert that every token takes: it has the experts' form and about their
        width, and no gate."""
        return (self.relu2 and not self.shared_gate and self.ff <= 2 * self.shared_ff <= 2 * self.ff and self.identity == 0 and self.top < 32
                and self.experts < 256)

    @property
    def in_features(self) -> int:
        """Rows of an expert's input map."""
        return self.ff * (self.maps - 1)

    @property
    def routed(self) -> int:
        """Outputs of the router."""
        return self.experts + self.identity


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a layered (hybrid) decoder: its mixer and the width of its FFN (0: no FFN, or a routed one, ``moe``).
    ``gate_limit`` > 0: the FFN is gated and clamped, ``min(g, limit) sigmoid(1.702 g) (clamp(u, +-limit) + 1)``; ``gelu``: it
    is gated, ``gelu_tanh(g) u``; otherwise it is ungated."""

    mixer: Mixer
    ff: int = 0
    gate_limit: float = 0.0
    gelu: bool = False
    moe: MoeSpec | None = None

    @property
    def has_ffn(self) -> bool:
        return self.ff > 0 or self.moe is not None

    @property
    def ffn_maps(self) -> int:
        """Matrices of ``hidden x ff`` elements."""
        return 3 if self.gate_limit > 0 or self.gelu else 2

    def ffn_params(self, hidden: int) -> int:
        m = self.moe
        if m is None:
            return self.ffn_maps * hidden * self.ff
        shared = hidden * (m.maps * m.shared_ff + int(m.shared_gate)) if m.shared_ff else 0
        return m.maps * m.experts * hidden * m.ff + m.routed * (hidden + 1) + shared


@dataclass(frozen=True)
class ModelConfig:
    name: str
    architecture: str  # HF ``architectures[0]``
    hidden_size: int
    num_layers: int
    num_q_heads: int
    num_kv_heads: int
    head_dim: int
    intermediate_size: int
    vocab_size: int
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    qk_norm: bool = True
    tie_word_embeddings: bool = False
    attention_bias: bool = False
    mlp_bias: bool = False
    hidden_act: str = "silu"
    max_position_embeddings: int = 40960
    # MoE (0 experts = dense)
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    num_shared_experts: int = 0
    first_k_dense: int = 0
    routed_scaling_factor: float = 1.0
    router_scoring: str = "softmax"  # or "sigmoid"
    router_precision: str = "payload"  # "fp32_logits" (payload weights, fp32 logits) or "fp32" (fp32 weights too)
    dtype: str = "bfloat16"
    # attention forms beyond rotary GQA with RMSNorm (the only one the GPU attention engine runs; the PyTorch oracle and the
    # CPU deployment run all of them)
    norm: str = "rmsnorm"            # or "layernorm" (weights and biases, mean-centred): OPT
    positions: str = "rope"          # or "learned" (a position table added to the embeddings): OPT
    sliding_window: int = 0          # > 0: layers named "sliding_attention" in extra["layer_types"] see this many keys
    attention_sinks: bool = False    # one learned logit per head joins every softmax and takes no value: GPT-OSS
    o_bias: bool = False
    mla: MlaShape | None = None
    # Layered decoders: every layer names its own mixer and FFN. norm "dyt" is dynamic tanh (elementwise, no statistics), "scalar"
    # an RMS norm with one weight for all coordinates; ``residual_gate``: each sublayer's result is multiplied by sigmoid(W h + b) of its input and summed in fp32.
    # ``output_norm``: sublayers' results are normed before they are added to the residual, which the sublayers read as it
    # is, or with ``input_norm`` through a norm of their own.
    # ``token_side`` > 0: behind the FFN every layer adds a small gated map of the residual and of a second embedding of its
    # token (that many dimensions per layer).
    layer_specs: tuple[LayerSpec, ...] = ()
    residual_gate: bool = False
    output_norm: bool = False
    input_norm: bool = False
    token_side: int = 0
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    extra: dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    @property
    def layered(self) -> bool:
        return bool(self.layer_specs)

    @property
    def recurrent(self) -> bool:
        """Some layer carries a per-sequence state (or a convolution's inputs), which cannot be shared between sequences like
        a cache page."""
        return any(s.mixer.state_elems or getattr(s.mixer, "conv_state_elems", 0) for s in self.layer_specs)

    def pages_shareable(self, page_size: int) -> bool:
        """Whether a page holds nothing but what its own tokens say: no state beside the pages, and no mean of a block that ends
        behind its page."""
        pools = [s.mixer for s in self.layer_specs if getattr(s.mixer, "pool", 0)]
        return not self.recurrent and all(m.pool_page(page_size) * m.pool == page_size for m in pools)

    @property
    def gpu_attention_supported(self) -> bool:
        if self.layered:
            return True
        return (self.norm == "rmsnorm" and self.positions == "rope" and self.mla is None and not self.attention_sinks
                and not self.sliding_window and not self.o_bias and not self.extra.get("rope_scaling"))

    def layer_window(self, layer: int) -> int:
        """Keys a query of ``layer`` may look back over (itself included); 0 = all of them."""
        kinds = self.extra.get("layer_types")
        if not self.sliding_window or (kinds and kinds[layer] != "sliding_attention"):
            return 0
        return self.sliding_window

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def q_size(self) -> int:
        return self.num_q_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def layer_is_moe(self, layer: int) -> bool:
        return self.is_moe and layer >= self.first_k_dense

    def attention_param_bytes(self) -> int:
        if self.layered:
            norm = {"dyt": 2 * self.hidden_size + 1, "scalar": 1}.get(self.norm, self.hidden_size)
            n = self.hidden_size * self.vocab_size * (1 if self.tie_word_embeddings else 2) + norm
            if self.token_side:
                n += self.num_layers * (self.token_side * (self.vocab_size + 2 * self.hidden_size) + norm)
            for s in self.layer_specs:
                subs = 1 + s.has_ffn
                n += s.mixer.param_count(self.hidden_size) + subs * norm * (2 if self.input_norm else 1)
                if self.residual_gate:
                    n += subs * self.hidden_size * (self.hidden_size + 1)
            return 2 * n
        per_layer = (self.q_size + 2 * self.kv_size) * self.hidden_size + self.hidden_size * self.q_size
        per_layer += 2 * self.hidden_size + 2 * self.head_dim
        emb = self.vocab_size * self.hidden_size * (1 if self.tie_word_embeddings else 2)
        return 2 * (per_layer * self.num_layers + emb + self.hidden_size)

    def ffn_param_bytes_per_layer(self, layer: int = 0) -> int:
        if self.layered:
            return 2 * self.layer_specs[layer].ffn_params(self.hidden_size)
        if self.layer_is_moe(layer):
            e = self.num_experts * 3 * self.hidden_size * self.moe_intermediate_size
            e += self.num_experts * self.hidden_size
            e += self.num_shared_experts * 3 * self.hidden_size * self.moe_intermediate_size
            return 2 * e
        return 2 * 3 * self.hidden_size * self.intermediate_size

    def kv_bytes_per_token(self) -> int:
        if self.layered:
            return 2 * sum(s.mixer.cache_width for s in self.layer_specs)        # (without the block means of pooling layers)
        return 2 * self.num_layers * self.kv_size * 2

    def state_bytes_per_sequence(self) -> int:
        """State of one running sequence over all layers: fp32 recurrences, convolution inputs in the activation type."""
        return sum(4 * s.mixer.state_elems + 2 * getattr(s.mixer, "conv_state_elems", 0) for s in self.layer_specs)

    def with_layers(self, n: int) -> "ModelConfig":
        if self.layered:
            return replace(self, num_layers=n, layer_specs=tuple(self.layer_specs[i % len(self.layer_specs)] for i in range(n)))
        return replace(self, num_layers=n)


def _qwen3(name, layers, hidden, q, kv, inter, **kw) -> ModelConfig:
    return ModelConfig(name=name, architecture="Qwen3ForCausalLM", hidden_size=hidden, num_layers=layers,
                       num_q_heads=q, num_kv_heads=kv, head_dim=128, intermediate_size=inter, vocab_size=151936,
                       **kw)


PRESETS: dict[str, ModelConfig] = {
    # CPU plumbing shape of the acceptance configuration
    "tiny-qwen3": ModelConfig(name="tiny-qwen3", architecture="Qwen3ForCausalLM", hidden_size=256, num_layers=2,
                              num_q_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=768, vocab_size=4096,
                              dtype="float32"),
    # the partner of Qwen3-0.6B in the reference's small benchmark pair (benches/benches.toml): 14 query / 2 KV heads
    # of 64, q/k/v biases, no q/k norm, rope theta 1e6
    "Qwen/Qwen2.5-0.5B": ModelConfig(name="Qwen/Qwen2.5-0.5B", architecture="Qwen2ForCausalLM", hidden_size=896, num_layers=24,
                                     num_q_heads=14, num_kv_heads=2, head_dim=64, intermediate_size=4864, vocab_size=151936,
                                     rope_theta=1e6, qk_norm=False, attention_bias=True, tie_word_embeddings=True),
    "Qwen/Qwen3-0.6B": _qwen3("Qwen/Qwen3-0.6B", 28, 1024, 16, 8, 3072, tie_word_embeddings=True),
    "Qwen/Qwen3-1.7B": _qwen3("Qwen/Qwen3-1.7B", 28, 2048, 16, 8, 6144, tie_word_embeddings=True),
    "Qwen/Qwen3-8B": _qwen3("Qwen/Qwen3-8B", 36, 4096, 32, 8, 12288),
    "Qwen/Qwen3-14B": _qwen3("Qwen/Qwen3-14B", 40, 5120, 40, 8, 17408),
    "Qwen/Qwen3-32B": _qwen3("Qwen/Qwen3-32B", 64, 5120, 64, 8, 25600),
    "Qwen/Qwen3-30B-A3B": ModelConfig(name="Qwen/Qwen3-30B-A3B", architecture="Qwen3MoeForCausalLM", hidden_size=2048,
                                      num_layers=48, num_q_heads=32, num_kv_heads=4, head_dim=128,
                                      intermediate_size=6144, vocab_size=151936, num_experts=128,
                                      num_experts_per_tok=8, moe_intermediate_size=768, norm_topk_prob=True),
    "tiny-qwen3-moe": ModelConfig(name="tiny-qwen3-moe", architecture="Qwen3MoeForCausalLM", hidden_size=256,
                                  num_layers=2, num_q_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=768,
                                  vocab_size=4096, num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128),
}


def preset(name: str) -> ModelConfig:
    try:
        return PRESETS[name]
    except KeyError:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(PRESETS)}") from None


def _ints(m: dict[str, Any], *names: str) -> dict[str, int]:
    return {n: int(m[n]) for n in names}


def _grouped_heads(m: dict[str, Any]) -> None:
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ValueError(f"{m['heads']} heads do not share {m['kv_heads']} key heads evenly")


def _mixer_from_config(kind: str, m: dict[str, Any]) -> Mixer:
    if kind == "delta":
        _grouped_heads(m)
        return DeltaMixer(**_ints(m, "heads", "kv_heads", "dim", "vdim", "conv"))
    if kind == "parallel":
        left, right = m["left"], m["right"]
        _grouped_heads(left)
        return ParallelMixer(
            GroupedMixer(**_ints(left, "heads", "kv_heads", "dim", "vdim"), scale=float(left["scale"]), softcap=float(left["softcap"])),
            GatedLinearMixer(**_ints(right, "heads", "dim", "vdim"), tau=float(right["tau"])))
    if kind == "latent_attention":
        rot = RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"]))
        mixer = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), rot, float(m["scale"]))
        if rot.dims % 2 or rot.dims > mixer.rot_dim:
            raise ValueError(f"rotary dims {rot.dims} do not fit the {mixer.rot_dim}-wide rotary part")
        return mixer
    if kind == "lightning":
        decay = tuple(float(d) for d in m["decay"])
        if len(decay) != int(m["heads"]):
            raise ValueError(f"{len(decay)} decays for {m['heads']} heads")
        return LinearMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), decay)
    raise ValueError(f"unsupported mixer {kind!r}")


def _dense_mlp(layer: dict[str, Any]) -> dict[str, Any]:
    mlp = layer.get("mlp")
    if mlp is not None and mlp.get("kind", "dense") != "dense":
        raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
    return mlp or {"ff": 0}


def segirax_config(cfg: dict[str, Any], name: str = "") -> ModelConfig:
    """Segirax: dynamic-tanh norms, gated fp32 residual stream, latent-attention and lightning mixers in any order, and
    ungated PolyNorm FFNs; its ``config.json`` lists every layer."""
    specs = []
    for l in cfg["layers"]:
        if l["type"] not in ("latent_attention", "lightning"):
            raise ValueError(f"unsupported mixer {l['type']!r}")
        specs.append(LayerSpec(_mixer_from_config(l["type"], l["mixer"]), int(_dense_mlp(l)["ff"])))
    first = specs[0].mixer
    return ModelConfig(
        name=name or cfg["architecture"], architecture=cfg["architecture"], hidden_size=int(cfg["width"]), num_layers=len(specs),
        num_q_heads=first.heads, num_kv_heads=1, head_dim=first.dim, intermediate_size=max(s.ff for s in specs),
        vocab_size=int(cfg["vocab"]), rms_norm_eps=float(cfg["norm"]["eps"]), qk_norm=False, tie_word_embeddings=True,
        hidden_act="polynorm", max_position_embeddings=1 << 30, norm="dyt", layer_specs=tuple(specs), residual_gate=True,
        logit_scale=float(cfg["logit_scale"]))


def saninex_config(cfg: dict[str, Any], name: str = "") -> ModelConfig:
    """Saninex: no norm before a sublayer and an RMS norm (weight stored as its distance from one) behind it, gated delta
    rule mixers and parallel pairs of capped softmax attention and gated linear attention in any order, clamped gated FFNs;
    its ``config.json`` lists every layer."""
    specs = []
    for l in cfg["layers"]:
        if l["type"] not in ("delta", "parallel"):
            raise ValueError(f"unsupported mixer {l['type']!r}")
        mlp = _dense_mlp(l)
        if mlp["ff"] and not float(mlp["limit"]) > 0:
            raise ValueError(f"feed-forward limit {mlp['limit']!r} is not positive")
        specs.append(LayerSpec(_mixer_from_config(l["type"], l["mixer"]), int(mlp["ff"]), float(mlp.get("limit", 0.0))))
    first = sub_mixers(specs[0].mixer)[0]
    return ModelConfig(
        name=name or cfg["architecture"], architecture=cfg["architecture"], hidden_size=int(cfg["width"]), num_layers=len(specs),
        num_q_heads=first.heads, num_kv_heads=first.kv_heads, head_dim=first.dim, intermediate_size=max(s.ff for s in specs),
        vocab_size=int(cfg["vocab"]), rms_norm_eps=float(cfg["norm"]["eps"]), qk_norm=True, tie_word_embeddings=True,
        hidden_act="clamped_glu", max_position_embeddings=1 << 30, norm="rmsnorm", layer_specs=tuple(specs), output_norm=True)


def _rotary(r: dict[str, Any] | None, dim: int, interleaved: bool = False) -> RotarySpec | None:
    if not r or not int(r["dims"]):
        return None
    sc = r.get("scaling")
    rot = RotarySpec(int(r["dims"]), float(r["base"]),
                     RotaryScaling(*(float(sc[n]) for n in ("factor", "low", "high", "original") if n in sc)) if sc else None, interleaved)
    if rot.dims % 2 or not 0 < rot.dims <= dim:
        raise ValueError(f"rotary dims {rot.dims} do not fit a head of {dim}")
    return rot


def _kadavik_attention(m: dict[str, Any]) -> GroupedMixer:
    _grouped_heads(m)
    mask = m.get("mask") or {}
    window, keep = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
    if window < 0 or keep < 0 or (mask and not window):
        raise ValueError(f"attention mask {mask!r} is not a window")
    kv_from = m.get("kv_from")
    return GroupedMixer(**_ints(m, "heads", "kv_heads", "dim", "vdim"), scale=float(m["scale"]), norm="", biases=False, gate="element",
                        conv=int(m.get("conv") or 0), rot=_rotary(m.get("rot"), int(m["dim"])), window=window,
                        keep_first=keep, kv_from=None if kv_from is None else int(kv_from))


def _kadavik_mlp(mixer: Mixer, mlp: dict[str, Any] | None) -> LayerSpec:
    if mlp is None:
        return LayerSpec(mixer)
    if mlp["kind"] == "dense":
        return LayerSpec(mixer, int(mlp["ff"]), gelu=True)
    if mlp["kind"] != "moe":
        raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
    r, shared = mlp["router"], mlp.get("shared")
    moe = MoeSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(r.get("identity") or 0), float(r.get("scale", 1.0)),
                  int(shared["ff"]) if shared else 0)
    if not 0 < moe.top <= min(moe.routed, 32) or moe.routed > 256 or moe.experts < 1:
        raise ValueError(f"a router of {moe.routed} outputs that takes {moe.top} is not supported (at most 32 of 256)")
    return LayerSpec(mixer, moe=moe)


def kadavik_config(cfg: dict[str, Any], name: str = "") -> ModelConfig:
    """Kadavik: norms before and behind every sublayer, matrix memories (mlstm) and windowed grouped-query attention with short
    convolutions in any order, attention layers that read another layer's keys and values, gelu or routed FFNs, and a second
    token embedding that every layer adds through a gate; its ``config.json`` lists every layer."""
    specs: list[LayerSpec] = []
    for i, l in enumerate(cfg["layers"]):
        m = l["mixer"]
        if l["type"] == "mlstm":
            mixer: Mixer = MemoryMixer(**_ints(m, "heads", "dim", "vdim"), gate_cap=float(m["gate_cap"]))
            if not mixer.gate_cap > 0:
                raise ValueError(f"gate cap {mixer.gate_cap} is not positive")
        elif l["type"] == "attention":
            mixer = _kadavik_attention(m)
            if mixer.kv_from is not None:
                src = specs[mixer.kv_from].mixer if 0 <= mixer.kv_from < i else None
                if not isinstance(src, GroupedMixer) or src.kv_from is not None or \
                        (src.kv_heads, src.dim, src.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ValueError(f"layer {i} cannot read the keys and values of layer {mixer.kv_from}")
        else:
            raise ValueError(f"unsupported mixer {l['type']!r}")
        specs.append(_kadavik_mlp(mixer, l.get("mlp")))
    first = specs[0].mixer
    side = cfg.get("token_side")
    return ModelConfig(
        name=name or cfg["architecture"], architecture=cfg["architecture"], hidden_size=int(cfg["width"]), num_layers=len(specs),
        num_q_heads=first.heads, num_kv_heads=getattr(first, "kv_heads", first.heads), head_dim=first.dim,
        intermediate_size=max(s.moe.ff if s.moe else s.ff for s in specs), vocab_size=int(cfg["vocab"]),
        rms_norm_eps=float(cfg["norm"]["eps"]), qk_norm=False, tie_word_embeddings=True, hidden_act="gelu_pytorch_tanh",
        max_position_embeddings=1 << 30, layer_specs=tuple(specs), output_norm=True, input_norm=True,
        token_side=int(side["dim"]) if side else 0, embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)),
        logit_scale=float(cfg.get("logit_scale", 1.0)))


def _window(m: dict[str, Any]) -> int:
    """Tokens a layer sees, itself included (0: all of them)."""
    mask = m.get("mask") or {}
    window = int(mask.get("size") or 0)
    if window < 0 or (mask and not window):
        raise ValueError(f"attention mask {mask!r} is not a window")
    return window


def _dofevik_mixer(kind: str, m: dict[str, Any]) -> Mixer:
    if kind == "attention":
        _grouped_heads(m)
        return GroupedMixer(**_ints(m, "heads", "kv_heads", "dim", "vdim"), scale=float(m["scale"]), norm="unit", gate="", window=_window(m),
                            rot=_rotary(m.get("rot"), int(m["dim"]), interleaved=True), sink=True)
    if kind == "attention_2":
        _grouped_heads(m)
        if int(m.get("vdim", m["dim"])) != int(m["dim"]):
            raise ValueError(f"values of {m['vdim']} dimensions cannot be keys of {m['dim']}")
        window, pool = _window(m), int((m.get("mask") or {}).get("pool") or 0)
        if pool < 0:
            raise ValueError(f"blocks of {pool} tokens")
        return GroupedMixer(**_ints(m, "heads", "kv_heads", "dim"), vdim=int(m["dim"]), scale=float(m["scale"]), biases=False, gate="",
                            window=window, sigmoid=True, pool=pool, tied=True)
    if kind == "latent_attention":
        mixer = LatentMixer(**_ints(m, "heads", "dim", "rot_dim", "vdim", "kv_rank"), rot=_rotary(m["rot"], int(m["rot_dim"])),
                            scale=float(m["scale"]), q_rank=int(m["q_rank"]), window=_window(m), gate_elems=True)
        if mixer.q_rank < 1:
            raise ValueError(f"a query latent of {mixer.q_rank} dimensions")
        return mixer
    raise ValueError(f"unsupported mixer {kind!r}")


def _dofevik_mlp(mixer: Mixer, mlp: dict[str, Any] | None) -> LayerSpec:
    if mlp is None:
        return LayerSpec(mixer)
    if mlp.get("kind", "moe") != "moe":
        raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
    r, shared = mlp["router"], mlp.get("shared")
    moe = MoeSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), shared_ff=int(shared["ff"]) if shared else 0, shared_gate=False,
                  relu2=True, logit_choice=True)
    if not 0 < moe.top <= min(moe.experts, 32) or moe.experts > 256:
        raise ValueError(f"a router of {moe.experts} outputs that takes {moe.top} is not supported (at most 32 of 256)")
    return LayerSpec(mixer, moe=moe)


def dofevik_config(cfg: dict[str, Any], name: str = "") -> ModelConfig:
    """Dofevik: RMS norms with one weight in front of every sublayer; windowed attention with unit queries and keys and a sink,
    attention with sigmoid weights over a window and the means of the blocks behind it, and windowed latent attention whose queries
    come from a latent, in any order; routed FFNs of squared-relu experts; its ``config.json`` lists every layer."""
    specs = tuple(_dofevik_mlp(_dofevik_mixer(l["type"], l["mixer"]), l.get("mlp")) for l in cfg["layers"])
    first = specs[0].mixer
    return ModelConfig(
        name=name or cfg["architecture"], architecture=cfg["architecture"], hidden_size=int(cfg["width"]), num_layers=len(specs),
        num_q_heads=first.heads, num_kv_heads=getattr(first, "kv_heads", first.heads), head_dim=first.dim,
        intermediate_size=max(s.moe.ff if s.moe else 0 for s in specs), vocab_size=int(cfg["vocab"]), rms_norm_eps=float(cfg["norm"]["eps"]),
        qk_norm=False, hidden_act="relu2", max_position_embeddings=1 << 30, norm="scalar", layer_specs=specs)


LAYERED_CONFIGS = {"Segirax": segirax_config, "Saninex": saninex_config, "Kadavik": kadavik_config, "Dofevik": dofevik_config}


def from_hf_config(cfg: dict[str, Any], name: str = "") -> ModelConfig:
    """Builds a :class:`ModelConfig` from a parsed ``config.json``."""
    if cfg.get("architecture") in LAYERED_CONFIGS:
        return LAYERED_CONFIGS[cfg["architecture"]](cfg, name)
    arch = (cfg.get("architectures") or ["Qwen3ForCausalLM"])[0]
    hidden = int(cfg["hidden_size"])
    heads = int(cfg["num_attention_heads"])
    kv = heads if arch.startswith("OPT") else int(cfg.get("num_key_value_heads") or heads)   # OPT has no grouped KV heads
    head_dim = int(cfg.get("head_dim") or hidden // heads)
    n_exp = int(cfg.get("num_experts") or cfg.get("n_routed_experts") or cfg.get("num_local_experts") or 0)
    rope = dict(cfg.get("rope_parameters") or cfg.get("rope_scaling") or {})
    rope_type = rope.get("rope_type", rope.get("type", "default"))
    mla = None
    if cfg.get("kv_lora_rank"):
        mla = MlaShape(int(cfg.get("q_lora_rank") or 0), int(cfg["kv_lora_rank"]), int(cfg["qk_nope_head_dim"]),
                       int(cfg["qk_rope_head_dim"]), int(cfg["v_head_dim"]))
    opt = arch.startswith("OPT")
    if opt and (not cfg.get("do_layer_norm_before", True) or int(cfg.get("word_embed_proj_dim", hidden)) != hidden):
        raise ValueError("OPT variants with post-layer norms or a projected embedding width are not supported")
    gpt_oss = arch.startswith("GptOss")
    extra = {k: v for k, v in cfg.items() if k in ("swiglu_limit", "sliding_window", "quantization_config", "layer_types",
                                                   "rope_interleave")}
    if rope_type not in ("default", None):
        extra["rope_scaling"] = {**rope, "rope_type": rope_type}
    if gpt_oss and not extra.get("layer_types"):     # the family alternates, starting with a windowed layer
        extra["layer_types"] = ["sliding_attention" if i % 2 == 0 else "full_attention" for i in range(int(cfg["num_hidden_layers"]))]
    window = int(cfg.get("sliding_window") or 0) if "sliding_attention" in (extra.get("layer_types") or ()) else 0
    return ModelConfig(
        name=name or cfg.get("_name_or_path", arch),
        architecture=arch,
        hidden_size=hidden,
        num_layers=int(cfg["num_hidden_layers"]),
        num_q_heads=heads,
        num_kv_heads=kv,
        head_dim=head_dim,
        intermediate_size=int(cfg.get("intermediate_size") or cfg.get("ffn_dim") or 0),
        vocab_size=int(cfg["vocab_size"]),
        rms_norm_eps=float(cfg.get("rms_norm_eps", cfg.get("layer_norm_eps", 1e-5 if opt else 1e-6))),
        rope_theta=float(cfg.get("rope_theta") or (cfg.get("rope_parameters") or {}).get("rope_theta") or 10000.0),
        qk_norm=arch.startswith("Qwen3"),
        tie_word_embeddings=bool(cfg.get("tie_word_embeddings", False)),
        attention_bias=bool(cfg.get("attention_bias", cfg.get("enable_bias", True) if opt else arch.startswith("Qwen2"))),
        mlp_bias=bool(cfg.get("mlp_bias", False)),
        hidden_act=str(cfg.get("hidden_act", cfg.get("activation_function", "silu"))),
        max_position_embeddings=int(cfg.get("max_position_embeddings", 32768)),
        num_experts=n_exp,
        num_experts_per_tok=int(cfg.get("num_experts_per_tok", 0) or 0),
        moe_intermediate_size=int(cfg.get("moe_intermediate_size", 0) or 0),
        norm_topk_prob=bool(cfg.get("norm_topk_prob", True)),
        num_shared_experts=int(cfg.get("n_shared_experts", 0) or 0),
        first_k_dense=int(cfg.get("first_k_dense_replace", 0) or 0),
        routed_scaling_factor=float(cfg.get("routed_scaling_factor", 1.0) or 1.0),
        router_scoring=str(cfg.get("scoring_func", "softmax")),
        router_precision={"DeepseekV2ForCausalLM": "fp32_logits", "Glm4MoeLiteForCausalLM": "fp32"}.get(arch, "payload"),
        dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
        norm="layernorm" if opt else "rmsnorm",
        positions="learned" if opt else "rope",
        sliding_window=window,
        attention_sinks=gpt_oss,
        o_bias=bool(cfg.get("attention_bias", False)) and (gpt_oss or mla is not None) or opt and bool(cfg.get("enable_bias", True)),
        mla=mla,
        extra=extra,
    )


def load(path_or_preset: str) -> ModelConfig:
    """A preset name, a directory holding ``config.json``, or a path to one."""
    if path_or_preset in PRESETS:
        return PRESETS[path_or_preset]
    p = Path(path_or_preset)
    if p.is_dir():
        p = p / "config.json"
    if not p.exists():
        raise FileNotFoundError(f"{path_or_preset!r} is neither a preset nor a config.json")
    return from_hf_config(json.loads(p.read_text()), name=str(p.parent.name))
