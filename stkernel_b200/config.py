"""Typed, frozen configuration for the whole engine.

One ``EngineConfig`` (model / parallel / cache / scheduler / speculative / kernel
sections) is built once from CLI + JSON, validated, printed resolved and never
re-read on a hot path.  This replaces the reference's three tiers of shell knobs,
``VLLM_*`` environment switches and ``vllm serve`` flags
(launchers/start-hy4-tp4.sh:16-155,370-391; overlay/attention.py:98-117).

Validation is fail-closed: an invalid knob raises ``ConfigError`` (the launcher
maps it to exit status 2, as launchers/start-hy4-tp4.sh:59-118 does).
"""
from __future__ import annotations

import dataclasses
import json
import math
from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Sequence, Tuple, Union


class ConfigError(ValueError):
    """Raised for any knob that fails validation (fail-closed)."""


KV_QUANT_BLOCK = 64          # elements per UE8M0 scale in an fp8_ds_mla row
KV_SCALE_BYTES = 8           # scale bytes per row (nope/64 used, rest padding)
FP8_BLOCK = 128              # block edge of dense FP8 weight scales / act groups
NVFP4_GROUP = 16             # elements per e4m3 scale (NVFP4)
MXFP4_GROUP = 32             # elements per ue8m0 scale (MXFP4 checkpoint layout)
FP8_MAX = 448.0


def _check_field_types(cfg) -> None:
    """Every field holds a value of its declared kind (a `config.json` with a string where a number belongs must fail as
    a configuration error that names the field, not as a TypeError somewhere in the arithmetic)."""
    for f in dataclasses.fields(cfg):
        v, d = getattr(cfg, f.name), f.default
        if isinstance(d, bool):
            ok = isinstance(v, bool)
        elif isinstance(d, int):
            ok = isinstance(v, int) and not isinstance(v, bool)
        elif isinstance(d, float):
            ok = isinstance(v, (int, float)) and not isinstance(v, bool) and v == v and abs(v) != float("inf")
        elif isinstance(d, str):
            ok = isinstance(v, str)
        elif isinstance(d, tuple):
            ok = isinstance(v, tuple) and all(isinstance(x, int) and not isinstance(x, bool) for x in v)
        else:
            ok = True
        if not ok:
            raise ConfigError(f"{f.name}: {v!r} is not a valid {type(d).__name__}")


@dataclass(frozen=True)
class ModelConfig:
    """Architecture of a DeepSeek-V4-style decoder.

    Field names follow the HF config consumed by the reference
    (overlay/attention.py:276-298, overlay/nvidia_model.py:775-808,1076-1078).
    """

    vocab_size: int = 129280
    hidden_size: int = 4096
    num_hidden_layers: int = 48
    num_attention_heads: int = 64
    head_dim: int = 512                     # latent KV width = nope + rope
    qk_rope_head_dim: int = 64
    q_lora_rank: int = 1536
    o_lora_rank: int = 1024
    o_groups: int = 8
    sliding_window: int = 128
    compress_ratios: Tuple[int, ...] = ()   # per layer: <=1 SWA-only, 4 C4A, 128 C128A
    index_n_heads: int = 64
    index_head_dim: int = 128
    index_topk: int = 2048
    index_topk_freq: int = 4
    use_index_cache: bool = True
    # Indexer operand format: "fp8" = e4m3 q with the scale folded into the head weights and e4m3 keys with one scale
    # per row (when the KV cache is fp8_ds_mla, else bf16); "mxfp4" = e2m1 q and keys with one ue8m0 scale per 32
    # values (overlay/ops_fused_indexer_q.py:175-282): half the indexer-K bytes.  Reference (CPU) path only.
    indexer_dtype: str = "fp8"
    hc_mult: int = 4
    hc_sinkhorn_iters: int = 20
    hc_eps: float = 1e-6
    n_routed_experts: int = 256
    num_experts_per_tok: int = 6
    moe_intermediate_size: int = 2048
    n_shared_experts: int = 1
    swiglu_limit: float = 10.0
    norm_topk_prob: bool = True
    scoring_func: str = "sigmoid"           # "sigmoid" | "sqrtsoftplus"
    topk_method: str = "noaux_tc"           # bias-corrected selection
    routed_scaling_factor: float = 1.0
    num_hash_layers: int = 0
    expert_dtype: str = "nvfp4"             # "nvfp4" | "mxfp4" | "bf16"
    dense_dtype: str = "fp8"                # "fp8" (128x128 block) | "bf16"
    kv_cache_dtype: str = "fp8_ds_mla"      # "fp8_ds_mla" | "bf16"
    n_mtp_layers: int = 0
    dspark_target_layer_ids: Tuple[int, ...] = ()
    dspark_markov_rank: int = 256
    dspark_block_size: int = 8
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    max_position_embeddings: int = 430000

    # ---- model-family interface (shared with HybridConfig) ------------
    family = "dsv4"                         # key of models/registry.py (a class attribute, not a field)

    def check_engine(self, e: "EngineConfig") -> None:
        """Engine settings this architecture cannot run with."""
        if self.num_attention_heads % e.parallel.tp_size:
            raise ConfigError("tp_size must divide num_attention_heads")
        if self.o_groups % e.parallel.tp_size and e.parallel.tp_size % self.o_groups:
            raise ConfigError("tp_size and o_groups must divide one another")

    # ---- derived -----------------------------------------------------
    @property
    def nope_dim(self) -> int:
        return self.head_dim - self.qk_rope_head_dim

    @property
    def kv_row_data_bytes(self) -> int:
        """fp8 nope bytes + bf16 rope bytes (576 for the production shape)."""
        return self.nope_dim + 2 * self.qk_rope_head_dim

    @property
    def kv_row_bytes(self) -> int:
        """Bytes per cached token row incl. scales (584 for the production shape)."""
        return self.kv_row_data_bytes + KV_SCALE_BYTES

    @property
    def mix_hc(self) -> int:
        return (2 + self.hc_mult) * self.hc_mult

    def layer_kind(self, layer: int) -> str:
        r = self.compress_ratios[layer] if layer < len(self.compress_ratios) else 0
        if r <= 1:
            return "swa"
        if r == 4:
            return "c4a"
        if r == 128:
            return "c128a"
        raise ConfigError(f"unsupported compress ratio {r} at layer {layer}")

    def compress_ratio(self, layer: int) -> int:
        r = self.compress_ratios[layer] if layer < len(self.compress_ratios) else 0
        return r if r > 1 else 0

    def validate(self) -> None:
        _check_field_types(self)
        for name in ("vocab_size", "hidden_size", "num_hidden_layers", "num_attention_heads", "head_dim", "q_lora_rank",
                     "o_lora_rank", "o_groups", "index_n_heads", "index_head_dim", "index_topk", "hc_mult",
                     "n_routed_experts", "num_experts_per_tok", "moe_intermediate_size", "sliding_window"):
            if getattr(self, name) < 1:
                raise ConfigError(f"{name} must be positive")
        if self.qk_rope_head_dim < 0 or self.n_mtp_layers < 0 or self.n_shared_experts < 0 or self.num_hash_layers < 0:
            raise ConfigError("qk_rope_head_dim, n_mtp_layers, n_shared_experts and num_hash_layers must not be negative")
        if self.head_dim <= self.qk_rope_head_dim:
            raise ConfigError("head_dim must exceed qk_rope_head_dim")
        if self.nope_dim % KV_QUANT_BLOCK:
            raise ConfigError(f"nope dim {self.nope_dim} must be a multiple of {KV_QUANT_BLOCK}")
        if self.nope_dim // KV_QUANT_BLOCK > KV_SCALE_BYTES:
            raise ConfigError("nope dim too large for 8 scale bytes per row")
        if self.qk_rope_head_dim % 2:
            raise ConfigError("rope dim must be even")
        if self.num_attention_heads % self.o_groups:
            raise ConfigError("o_groups must divide num_attention_heads")
        if len(self.compress_ratios) not in (0, self.num_hidden_layers,
                                             self.num_hidden_layers + self.n_mtp_layers):
            raise ConfigError("compress_ratios must have one entry per layer")
        for i in range(self.num_hidden_layers):
            self.layer_kind(i)
        if self.scoring_func not in ("sigmoid", "sqrtsoftplus"):
            raise ConfigError(f"unknown scoring_func {self.scoring_func!r}")
        if self.expert_dtype not in ("nvfp4", "mxfp4", "bf16"):
            raise ConfigError(f"unknown expert_dtype {self.expert_dtype!r}")
        if self.dense_dtype not in ("fp8", "bf16"):
            raise ConfigError(f"unknown dense_dtype {self.dense_dtype!r}")
        if self.kv_cache_dtype not in ("fp8_ds_mla", "bf16"):
            raise ConfigError(f"unknown kv_cache_dtype {self.kv_cache_dtype!r}")
        if self.num_experts_per_tok > self.n_routed_experts:
            raise ConfigError("top-k exceeds expert count")
        if self.index_topk_freq < 1:
            raise ConfigError("index_topk_freq must be >= 1")
        if self.index_head_dim < self.qk_rope_head_dim:
            raise ConfigError("index_head_dim must be >= rope dim")
        if self.indexer_dtype not in ("fp8", "mxfp4"):
            raise ConfigError(f"unknown indexer_dtype {self.indexer_dtype!r}")
        if self.indexer_dtype == "mxfp4" and (self.qk_rope_head_dim % 32 or (self.index_head_dim - self.qk_rope_head_dim) % 32):
            raise ConfigError("mxfp4 indexer operands need the rope and non-rope parts of index_head_dim in blocks of 32")


def alternating_ratios(n_layers: int, first: int = 4, second: int = 0) -> Tuple[int, ...]:
    """Layers alternate compressed-sparse attention with sliding-window-only."""
    return tuple(first if i % 2 == 0 else second for i in range(n_layers))


def flash_config(num_layers: int = 48, **over: Any) -> ModelConfig:
    """The DeepSeek-V4-Flash-shaped architecture used by the headline benchmark."""
    kw: Dict[str, Any] = dict(num_hidden_layers=num_layers,
                              compress_ratios=alternating_ratios(num_layers))
    kw.update(over)
    cfg = ModelConfig(**kw)
    cfg.validate()
    return cfg


def tiny_config(**over: Any) -> ModelConfig:
    """2-layer CPU-sized decoder: one C4A layer + one SWA layer, 8 experts top-2."""
    kw: Dict[str, Any] = dict(
        vocab_size=1024, hidden_size=256, num_hidden_layers=2, num_attention_heads=4,
        head_dim=80, qk_rope_head_dim=16, q_lora_rank=96, o_lora_rank=64, o_groups=2,
        sliding_window=32, compress_ratios=(4, 0), index_n_heads=2, index_head_dim=32,
        index_topk=16, index_topk_freq=4, hc_mult=4, hc_sinkhorn_iters=20,
        n_routed_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
        n_shared_experts=1, scoring_func="sigmoid", expert_dtype="bf16", dense_dtype="bf16",
        kv_cache_dtype="bf16", max_position_embeddings=4096,
    )
    kw.update(over)
    cfg = ModelConfig(**kw)
    cfg.validate()
    return cfg


# ----------------------------------------------------------------------------
# decoders described layer by layer
# ----------------------------------------------------------------------------
FULL_CONTEXT = 1 << 40       # window of an attention layer that sees every earlier position


@dataclass(frozen=True)
class YarnScaling:
    """YaRN context extension of a rotary embedding: frequencies below the `slow` bound are divided by `factor`, those
    above the `fast` bound stay, with a linear ramp between them; cos and sin are scaled by 1 + 0.1 ln(factor)."""
    factor: float
    original: float              # context length the unscaled frequencies were made for
    fast: float                  # full turns over `original` above which a frequency is kept
    slow: float                  # full turns over `original` below which a frequency is divided by `factor`


@dataclass(frozen=True)
class LinearScaling:
    """Linear context extension of a rotary embedding: every frequency is divided by `factor`."""
    factor: float


@dataclass(frozen=True)
class RotaryConfig:
    """Rotation of the first `dims` dimensions of a head: dimension i paired with i + dims/2, or with its neighbour
    (2i with 2i + 1) when `interleaved`."""
    base: float
    dims: int
    scaling: Optional[Union[YarnScaling, LinearScaling]] = None
    interleaved: bool = False

    def frequencies(self) -> Tuple[List[float], float]:
        """-> (radians per position of every pair, factor on cos and sin)."""
        d = self.dims
        f = [self.base ** (-2.0 * i / d) for i in range(d // 2)]
        s = self.scaling
        if s is None:
            return f, 1.0
        if isinstance(s, LinearScaling):
            return [x / s.factor for x in f], 1.0
        at = lambda turns: d * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo = max(math.floor(at(s.fast)), 0)
        hi = min(math.ceil(at(s.slow)), d - 1)
        span = max(hi - lo, 0.001)
        out = []
        for i, x in enumerate(f):
            r = min(max((i - lo) / span, 0.0), 1.0)
            out.append(x / s.factor * r + x * (1.0 - r))
        return out, 0.1 * math.log(s.factor) + 1.0


@dataclass(frozen=True)
class AttentionMixer:
    """Grouped-query sliding-window attention whose values are the unrotated keys (no value projection), with a tanh cap
    on the scaled scores and one learned sink per head in the softmax denominator."""
    heads: int
    kv_heads: int
    dim: int
    window: int                  # keys a position sees, itself included
    scale: float
    rotary: Optional[RotaryConfig] = None
    softcap: float = 0.0         # 0: scores are not capped
    sink: bool = True
    kind = "attention"

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def rot_dims(self) -> int:
        return self.rotary.dims if self.rotary is not None else 0

    @property
    def out_dim(self) -> int:
        return self.heads * self.dim


@dataclass(frozen=True)
class LatentAttentionMixer:
    """Causal attention over low-rank latents: queries come out of a normed latent of size q_rank, keys and values are read out
    of a normed latent of size kv_rank per token (per head `dim` unrotated key dimensions and `vdim` value dimensions) plus one
    rotated key part of rot_dim dimensions that all heads share.  A head's output is multiplied by the sigmoid of a gate."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rotary: Optional[RotaryConfig] = None
    kv_from: Optional[int] = None         # layer whose cached latents and rotated key parts this one attends over
    kind = "latent_attention"
    window = FULL_CONTEXT

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class MlstmMixer:
    """Matrix-memory recurrence with exponential input gate and running-maximum stabiliser (mLSTM)."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float              # tanh cap of both gate pre-activations
    kind = "mlstm"

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class QueryTemperature:
    """Queries at position p are multiplied by 1 + coef * ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: float


@dataclass(frozen=True)
class GroupedAttentionMixer:
    """Grouped-query causal attention over the full context with key and value projections of their own sizes and no rotation.

    qk_norm: queries and keys are divided by their root mean square per head; null_sink: the softmax has one more key of score 0
    and no value; gate: the heads' outputs are multiplied element by element with the sigmoid of a projection of the same input."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature] = None
    bias: bool = True                     # q, k and v projections have biases
    qk_norm: bool = True
    null_sink: bool = True
    gate: bool = True
    kind = "grouped_attention"
    window = FULL_CONTEXT

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class TalkingAttentionMixer:
    """Grouped-query attention whose heads' scaled scores are mixed by a matrix [heads, heads] before the softmax.

    chunk: a position sees the earlier positions of its own chunk only (chunks of that many positions, counted from position 0; None:
    the full context); bias: q, k and v projections have biases; qk_norm: queries and keys are RMS-normed per head, with a weight that
    the heads share, before their rotation; sink: one score without key and value per head, learned; gate: every head's output is
    multiplied with the sigmoid of one number that is projected from the same input."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int] = None
    rotary: Optional[RotaryConfig] = None
    bias: bool = True
    qk_norm: bool = True
    sink: bool = True
    gate: bool = True
    kind = "talking_attention"

    @property
    def window(self) -> int:
        return FULL_CONTEXT if self.chunk is None else self.chunk

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class TimeMixMixer:
    """Linear attention with a decay per head and key channel that the token chooses, S <- diag(w) S + k v^T, read out before the update
    with a bonus u for the current token, o = (S + diag(u) k v^T)^T r.  Every projection reads a blend of its own between the token's
    input and the previous token's; log w = -exp(W2 tanh(W1 x) + w0), W1 with `rank` rows (None: as many as the checkpoint has).  A
    head's read-out is divided by its root mean square, weighted, and multiplied with silu of a gate."""
    heads: int
    dim: int
    rank: Optional[int] = None
    kind = "time_mix"

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def out_dim(self) -> int:
        return self.heads * self.dim


@dataclass(frozen=True)
class RetentionMixer:
    """Linear attention with a fixed decay per head: S <- decay S + k v^T, read with the query; queries and keys are rotated,
    every head's read-out is divided by its root mean square and multiplied with silu of a gate."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rotary: Optional[RotaryConfig] = None
    kind = "retention"

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class Mamba2Mixer:
    """Mamba-2: a short causal convolution over (x, B, C), then S <- exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x per head; the
    gated output is RMS-normed in norm_groups equal parts.  Heads share B and C within each of `groups` groups."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                             # taps, the current token's included
    norm_groups: int
    kind = "mamba2"

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_dim(self) -> int:
        return self.out_dim + 2 * self.groups * self.state


@dataclass(frozen=True)
class ParallelMixer:
    """Two mixers over the same input: left_scale * left + right_scale * right.  At most one of them keeps a cache and at most
    one a recurrent state.  out_norm: each side's output is RMS-normed over the model width first, with a weight of its own."""
    left: Union[GroupedAttentionMixer, TalkingAttentionMixer]
    right: Union[RetentionMixer, TimeMixMixer]
    left_scale: float = 1.0
    right_scale: float = 1.0
    out_norm: bool = False
    kind = "parallel"

    @property
    def out_dim(self) -> int:
        return self.left.out_dim + self.right.out_dim


@dataclass(frozen=True)
class DenseMlp:
    """W_down(act(W_gate h) * W_up h), or W_down act(W_up h) for an activation without a gate.  "xielu" has two learned numbers (a, b):
    softplus(a) z^2 + z / 2 for z > 0, (softplus(b) + 1/2) (exp(z) - 1 - z) + z / 2 otherwise."""
    ff: int
    act: str = "silu"                     # "silu" | "relu" (gated), "xielu" (no gate)
    kind = "dense"

    @property
    def gated(self) -> bool:
        return self.act != "xielu"


@dataclass(frozen=True)
class MoeMlp:
    """`top` of `experts` feed-forward layers W_down act(W_up h) per token, chosen by the largest router logits (bias included)
    and weighted by the softmax over the chosen logits (which is the softmax over all of them, renormalised); a shared expert of
    the same form, if there is one, is added for every token.

    act "silu" has a gate: W_down (silu(W_gate h) * W_up h).  scoring "sigmoid": experts are chosen by the sigmoid of their logit plus a
    correction (with groups > 1 only experts of the `keep` best of that many equal groups of neighbours, a group's score being the
    sum of its two largest), and weighted by the sigmoid alone, renormalised over the chosen, times `scale`."""
    experts: int
    top: int
    ff: int
    act: str = "relu2"                    # "relu2" (relu squared) | "gelu" (exact) | "silu" (gated)
    router_bias: bool = True
    shared_ff: int = 0                    # 0: no shared expert
    scoring: str = "softmax_topk"         # "softmax_topk" | "sigmoid"
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    kind = "moe"

    @property
    def gated(self) -> bool:
        return self.act == "silu"

    @property
    def shared_parts(self) -> int:
        """The shared expert runs as this many always-chosen experts (W_down act(W_up h) is a sum over slices of its columns)."""
        return 0 if not self.shared_ff else min(-(-self.shared_ff // self.ff), 8, 32 - self.top)

    @property
    def expert_width(self) -> int:
        """Hidden columns of a stored expert: those of an expert, or of a part of the shared one if that is wider."""
        return self.ff if not self.shared_ff else max(self.ff, -(-self.shared_ff // self.shared_parts))


Mixer = Union[AttentionMixer, MlstmMixer, LatentAttentionMixer, GroupedAttentionMixer, TalkingAttentionMixer, RetentionMixer,
              TimeMixMixer, Mamba2Mixer, ParallelMixer]
Mlp = Union[DenseMlp, MoeMlp]

ATTENTION_KINDS = ("attention", "latent_attention", "grouped_attention", "talking_attention")
RECURRENT_KINDS = ("mlstm", "retention", "mamba2", "time_mix")


def mixer_parts(m: Mixer) -> Tuple[Mixer, ...]:
    """The mixers a layer runs (a parallel mixer's two sides, otherwise itself)."""
    return (m.left, m.right) if m.kind == "parallel" else (m,)


def attention_part(m: Mixer) -> Optional[Mixer]:
    """The part of a mixer that keeps a paged cache."""
    return next((p for p in mixer_parts(m) if p.kind in ATTENTION_KINDS), None)


def recurrent_part(m: Mixer) -> Optional[Mixer]:
    """The part of a mixer that keeps a recurrent state."""
    return next((p for p in mixer_parts(m) if p.kind in RECURRENT_KINDS), None)


@dataclass(frozen=True)
class HybridLayer:
    mixer: Mixer
    mlp: Optional[Mlp] = None
    weights_of: Optional[int] = None      # layer whose tensors this one runs with (cache and state are its own)


@dataclass(frozen=True)
class BigramTable:
    """A second embedding, of the token and the one before it: row (previous * mul_prev + token * mul_cur) mod buckets; a sequence's
    first token takes row `buckets`, the table's last."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class HybridConfig:
    """A decoder given as a list of layers, each with its own mixer (attention or recurrence) and optional feed-forward.

    block "parallel":  both sublayers read one layer norm's output and are added to the fp32 residual together;
    block "post_norm": the sublayers follow one another, read the residual itself, and their outputs are RMS-normed before
                       they are added to it;
    block "streams":   several residual streams; a sublayer reads the layer norm (with bias) of a weighted sum of them, and every
                       stream becomes a weighted sum of all of them plus a multiple of the sublayer's output.  The model's
                       output is the sum of the streams;
    block "shifted":   both sublayers read one RMS norm's output and are added to the fp32 residual together; what the mixer reads
                       is blended, element by element, with the previous token's norm output (token shift)."""
    vocab_size: int
    hidden_size: int
    layers: Tuple[HybridLayer, ...]
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    dtype: str = "bfloat16"               # "bfloat16": projections and activations; "float32": everything
    max_position_embeddings: int = 1 << 30
    architecture: str = "Timalorn"
    block: str = "parallel"               # "parallel" | "post_norm" | "streams" | "shifted"
    streams: int = 1                      # residual streams ("streams" blocks)
    tied_head: bool = False               # logits are read with the embedding table
    logit_scale: float = 1.0
    bigram: Optional[BigramTable] = None  # added to the embedding ("shifted" blocks)
    family = "hybrid"
    # fields of the other family that family-neutral code asks for
    n_mtp_layers = 0
    n_routed_experts = 0

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def weight_layer(self, i: int) -> int:
        """The layer whose tensors layer i uses (itself unless `weights_of` says otherwise)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ConfigError(f"layers[{i}].weights_of refers to itself")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def windows(self) -> List[int]:
        """Distinct attention windows, one page group each (FULL_CONTEXT: pages stay until the request ends)."""
        parts = [attention_part(l.mixer) for l in self.layers]
        return sorted({p.window for p in parts if p is not None})

    def cache_layer(self, i: int) -> int:
        """The layer whose cache layer i reads (itself unless `kv_from` says otherwise)."""
        j = getattr(self.layers[i].mixer, "kv_from", None)
        return i if j is None else j

    def mechanisms(self) -> Tuple[str, ...]:
        """Kinds of mixers and feed-forwards in this model, which decide what kernels it needs."""
        return tuple(sorted({p.kind for l in self.layers for p in mixer_parts(l.mixer)}
                            | {l.mlp.kind for l in self.layers if l.mlp is not None}
                            | ({"token_shift"} if self.block == "shifted" else set())))

    def validate(self) -> None:
        def positive(name: str, v: Any, integer: bool = True) -> None:
            ok = (isinstance(v, int) if integer else isinstance(v, (int, float))) and not isinstance(v, bool)
            if not ok or not math.isfinite(v) or v <= 0:
                raise ConfigError(f"{name}: {v!r} must be a positive {'integer' if integer else 'number'}")

        positive("vocab_size", self.vocab_size)
        positive("hidden_size", self.hidden_size)
        positive("norm_eps", self.norm_eps, False)
        def number(name: str, v: Any) -> None:
            if not isinstance(v, (int, float)) or isinstance(v, bool) or not math.isfinite(v):
                raise ConfigError(f"{name} must be a finite number")

        number("embedding_scale", self.embedding_scale)
        number("logit_scale", self.logit_scale)
        positive("streams", self.streams)
        if self.streams > 8 or (self.streams != 1 and self.block != "streams"):
            raise ConfigError("streams: at most 8, and 1 unless the block is \"streams\"")
        if self.dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"unknown dtype {self.dtype!r}")
        if not self.layers:
            raise ConfigError("layers must not be empty")
        if self.block not in ("parallel", "post_norm", "streams", "shifted"):
            raise ConfigError(f"unknown block {self.block!r}")
        if self.bigram is not None:
            if self.block != "shifted":
                raise ConfigError("a bigram embedding is available in shifted blocks")
            positive("embedding.bigram.buckets", self.bigram.buckets)
            for f in ("mul_prev", "mul_cur"):
                v = getattr(self.bigram, f)
                if not isinstance(v, int) or isinstance(v, bool) or not 0 <= v < 1 << 31:
                    raise ConfigError(f"embedding.bigram.{f}: {v!r} must be an integer from 0 to 2^31 - 1")

        def rotary(at: str, r: RotaryConfig, dim: int, of: str) -> None:
            positive(f"{at}.rot.base", r.base, False)
            positive(f"{at}.rot.dims", r.dims)
            if r.dims % 2 or r.dims > dim:
                raise ConfigError(f"{at}.rot.dims must be even and at most {of}")
            if r.scaling is not None:
                for f in dataclasses.fields(r.scaling):
                    positive(f"{at}.rot.scaling.{f.name}", getattr(r.scaling, f.name), False)

        def mixer(at: str, i: int, m: Mixer) -> None:
            """at: name of the mixer's section."""
            positive(f"{at}.heads", m.heads)
            if m.kind != "mamba2":
                positive(f"{at}.dim", m.dim)
                if m.dim > 1024:
                    raise ConfigError(f"{at}.dim: at most 1024")
            if m.kind in ATTENTION_KINDS:
                number(f"{at}.scale", m.scale)
            if m.kind == "attention":
                positive(f"{at}.kv_heads", m.kv_heads)
                positive(f"{at}.mask.size", m.window)
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: kv_heads must divide heads")
                if m.softcap < 0 or not math.isfinite(m.softcap):
                    raise ConfigError(f"{at}.softcap must not be negative")
                if m.rotary is not None:
                    rotary(at, m.rotary, m.dim, "dim")
            elif m.kind == "latent_attention":
                for f in ("vdim", "q_rank", "kv_rank"):
                    positive(f"{at}.{f}", getattr(m, f))
                if m.rot_dim != 0:
                    positive(f"{at}.rot_dim", m.rot_dim)
                if m.kv_rank + m.rot_dim > 2048 or m.vdim > 1024:
                    raise ConfigError(f"{at}: kv_rank + rot_dim must be at most 2048, vdim at most 1024")
                if m.rotary is not None:
                    rotary(at, m.rotary, m.rot_dim, "rot_dim")
                if (m.rotary.dims if m.rotary is not None else 0) != m.rot_dim:
                    raise ConfigError(f"{at}.rot.dims must equal rot_dim")
                j = m.kv_from
                if j is not None:
                    if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < i:
                        raise ConfigError(f"{at}.kv_from: {j!r} is not an earlier layer")
                    src = self.layers[j].mixer
                    if (src.kind != "latent_attention" or src.kv_from is not None
                            or (src.kv_rank, src.rot_dim, src.rotary) != (m.kv_rank, m.rot_dim, m.rotary)):
                        raise ConfigError(f"{at}.kv_from: layer {j} must cache latents of its own of the same kv_rank, "
                                          "rot_dim and rotation")
            elif m.kind == "grouped_attention":
                positive(f"{at}.kv_heads", m.kv_heads)
                positive(f"{at}.vdim", m.vdim)
                if m.vdim > 1024:
                    raise ConfigError(f"{at}.vdim: at most 1024")
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: kv_heads must divide heads")
                if m.q_temp is not None:
                    number(f"{at}.q_temp.coef", m.q_temp.coef)
                    positive(f"{at}.q_temp.every", m.q_temp.every, False)
            elif m.kind == "talking_attention":
                positive(f"{at}.kv_heads", m.kv_heads)
                positive(f"{at}.vdim", m.vdim)
                if m.chunk is not None:
                    positive(f"{at}.mask.size", m.chunk)
                if m.vdim > 1024:
                    raise ConfigError(f"{at}.vdim: at most 1024")
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: kv_heads must divide heads")
                if m.rotary is not None:
                    rotary(at, m.rotary, m.dim, "dim")
            elif m.kind == "time_mix":
                if m.rank is not None:
                    positive(f"{at}.rank", m.rank)
            elif m.kind == "retention":
                positive(f"{at}.vdim", m.vdim)
                if not isinstance(m.decay, tuple) or len(m.decay) != m.heads:
                    raise ConfigError(f"{at}.decay: one number per head")
                for d in m.decay:
                    positive(f"{at}.decay", d, False)
                if m.rotary is not None:
                    rotary(at, m.rotary, m.dim, "dim")
            elif m.kind == "mamba2":
                for f in ("vdim", "state", "groups", "conv", "norm_groups"):
                    positive(f"{at}.{f}", getattr(m, f))
                if m.state > 1024 or m.conv > 64:
                    raise ConfigError(f"{at}: state must be at most 1024, conv at most 64")
                if m.heads % m.groups:
                    raise ConfigError(f"{at}: groups must divide heads")
                if m.out_dim % m.norm_groups:
                    raise ConfigError(f"{at}: norm_groups must divide heads * vdim")
            else:
                positive(f"{at}.vdim", m.vdim)
                positive(f"{at}.gate_cap", m.gate_cap, False)

        for i, l in enumerate(self.layers):
            at, m = f"layers[{i}]", l.mixer
            if self.block == "parallel" and (m.kind not in ("attention", "mlstm") or (l.mlp is not None and l.mlp.kind != "dense")):
                raise ConfigError(f"{at}: {m.kind} with this feed-forward is not available in parallel blocks")
            if m.kind == "parallel":
                number(f"{at}.mixer.left_scale", m.left_scale)
                number(f"{at}.mixer.right_scale", m.right_scale)
                sides = (m.left.kind, m.right.kind)
                if sides == ("talking_attention", "time_mix"):
                    if self.block != "shifted" or not m.out_norm:
                        raise ConfigError(f"{at}.mixer: talking attention beside time mixing needs shifted blocks and norms on the outputs")
                elif sides != ("grouped_attention", "retention"):
                    raise ConfigError(f"{at}.mixer: this build combines grouped attention with retention, and talking attention with "
                                      "time mixing")
                elif m.out_norm or self.block == "shifted":
                    raise ConfigError(f"{at}.mixer: grouped attention beside retention has no norms on its outputs and no token shift")
                mixer(f"{at}.mixer.left", i, m.left)
                mixer(f"{at}.mixer.right", i, m.right)
            else:
                if m.kind in ("grouped_attention", "retention", "talking_attention", "time_mix"):
                    raise ConfigError(f"{at}.type: {m.kind} is one side of a parallel mixer")
                mixer(f"{at}.mixer", i, m)
            if l.mlp is not None:
                positive(f"{at}.mlp.ff", l.mlp.ff)
                if l.mlp.kind == "dense":
                    if l.mlp.act not in ("silu", "relu", "xielu") or (l.mlp.act == "xielu" and self.block == "parallel"):
                        raise ConfigError(f"{at}.mlp.act: unknown activation {l.mlp.act!r}")
                else:
                    p = l.mlp
                    positive(f"{at}.mlp.router.experts", p.experts)
                    positive(f"{at}.mlp.router.top", p.top)
                    if p.act not in ("relu2", "gelu", "silu"):
                        raise ConfigError(f"{at}.mlp.act: unknown activation {p.act!r}")
                    if p.scoring not in ("softmax_topk", "sigmoid"):
                        raise ConfigError(f"{at}.mlp.router: unknown scoring {p.scoring!r}")
                    number(f"{at}.mlp.router.scale", p.scale)
                    positive(f"{at}.mlp.router.groups.count", p.groups)
                    positive(f"{at}.mlp.router.groups.keep", p.keep)
                    if p.groups > 1 and (p.scoring != "sigmoid" or p.groups > 32 or p.experts % p.groups
                                         or p.experts // p.groups < 2):
                        raise ConfigError(f"{at}.mlp.router.groups: at most 32 equal groups of two experts or more, with sigmoid scores")
                    if p.keep > p.groups or p.experts // p.groups * p.keep < p.top:
                        raise ConfigError(f"{at}.mlp.router.groups.keep: at most count, and enough for `top` experts")
                    if p.shared_ff and (p.gated or p.scoring != "softmax_topk"):
                        raise ConfigError(f"{at}.mlp.shared: not available with gated experts or sigmoid scores")
                    if p.shared_ff != 0:
                        positive(f"{at}.mlp.shared.ff", p.shared_ff)
                    most = 31 if p.shared_ff else 32
                    if p.top > p.experts or p.top > most or p.experts + p.shared_parts > 512:
                        raise ConfigError(f"{at}.mlp.router: top must be at most experts and {most}, experts (and the parts of the "
                                          "shared one) at most 512")
            if l.weights_of is not None:
                j = l.weights_of
                if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < len(self.layers):
                    raise ConfigError(f"{at}.weights_of: no layer {j!r}")
                src = self.layers[self.weight_layer(i)]
                if src.mixer != m or src.mlp != l.mlp:
                    raise ConfigError(f"{at} must equal layer {j}, whose weights it uses")

    def check_engine(self, e: "EngineConfig") -> None:
        p = e.parallel
        if p.tp_size != 1 or p.pp_size != 1 or p.dcp_size != 1:
            raise ConfigError(f"{self.architecture} runs on one GPU (no tensor, pipeline or context parallelism)")
        if e.spec.method != "none":
            raise ConfigError(f"{self.architecture} has no draft layers for speculative decoding")
        if p.eplb_record or p.eplb_redundant:
            raise ConfigError(f"{self.architecture} has no expert placement to balance")


def _take(d: Any, at: str, required: Sequence[str], optional: Sequence[str] = ()) -> Dict[str, Any]:
    """The keys of a JSON object, none missing and none unknown (an unknown key that is null or false asks for nothing)."""
    if not isinstance(d, Mapping):
        raise ConfigError(f"{at}: {d!r} is not an object")
    for k in required:
        if k not in d:
            raise ConfigError(f"{at}: {k} is missing")
    unknown = {k for k in unknown_keys(d, required, optional) if d[k] is not None and d[k] is not False}
    if unknown:
        raise ConfigError(f"{at}: unknown keys {sorted(unknown)}")
    return {k: v for k, v in d.items() if k not in unknown_keys(d, required, optional)}


def unknown_keys(d: Mapping[str, Any], required: Sequence[str], optional: Sequence[str]) -> set:
    return set(d) - set(required) - set(optional)


def _check_model_keys(d: Mapping[str, Any], more: Sequence[str] = ("embedding",)) -> None:
    for k in ("vocab", "width", "layers", "norm") + tuple(more):
        if k not in d:
            raise ConfigError(f"config.json: {k} is missing")
    if not isinstance(d["layers"], Sequence) or isinstance(d["layers"], str):
        raise ConfigError("config.json: layers is not a list")


def timalorn_config_from_json(d: Mapping[str, Any], dtype: str = "bfloat16") -> HybridConfig:
    """The `config.json` of a Timalorn model: parallel blocks of windowed attention and mLSTM layers."""
    _check_model_keys(d)
    layers: List[HybridLayer] = []
    for i, l in enumerate(d["layers"]):
        at = f"layers[{i}]"
        l = _take(l, at, ("type", "mixer"), ("mlp", "weights_of"))
        if l["type"] == "attention":
            m = _take(l["mixer"], f"{at}.mixer", ("heads", "kv_heads", "dim", "mask", "scale"),
                      ("vdim", "rot", "softcap"))
            if m.get("vdim", m["dim"]) != m["dim"]:
                raise ConfigError(f"{at}.mixer.vdim: the values are the keys, so it must equal dim")
            rot = None
            if m.get("rot") is not None:
                r = _take(m["rot"], f"{at}.mixer.rot", ("base", "dims"), ("scaling",))
                sc = r.get("scaling")
                if sc is not None:
                    sc = YarnScaling(**_take(sc, f"{at}.mixer.rot.scaling", ("factor", "original", "fast", "slow")))
                rot = RotaryConfig(r["base"], r["dims"], sc)
            mixer: Mixer = AttentionMixer(
                m["heads"], m["kv_heads"], m["dim"], _take(m["mask"], f"{at}.mixer.mask", ("size",))["size"], m["scale"], rot,
                m.get("softcap") or 0.0)
        elif l["type"] == "mlstm":
            mixer = MlstmMixer(**_take(l["mixer"], f"{at}.mixer", ("heads", "dim", "vdim", "gate_cap")))
        else:
            raise ConfigError(f"{at}.type: unknown mixer {l['type']!r}")
        mlp = None
        if l.get("mlp") is not None:
            p = _take(l["mlp"], f"{at}.mlp", ("kind", "ff"))
            if p["kind"] != "dense":
                raise ConfigError(f"{at}.mlp.kind: unknown feed-forward {p['kind']!r}")
            mlp = DenseMlp(p["ff"])
        layers.append(HybridLayer(mixer, mlp, l.get("weights_of")))
    cfg = HybridConfig(d["vocab"], d["width"], tuple(layers), _take(d["norm"], "norm", ("eps",))["eps"],
                       _take(d["embedding"], "embedding", ("scale",))["scale"], dtype)
    cfg.validate()
    return cfg


def timalorn_config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    """The inverse of `timalorn_config_from_json`."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        if m.kind == "attention":
            mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim,
                                     "mask": {"size": m.window}, "scale": m.scale, "softcap": m.softcap}
            if m.rotary is not None:
                mixer["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
                if m.rotary.scaling is not None:
                    mixer["rot"]["scaling"] = dataclasses.asdict(m.rotary.scaling)
        else:
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
        d: Dict[str, Any] = {"type": m.kind, "mixer": mixer,
                             "mlp": {"kind": "dense", "ff": l.mlp.ff} if l.mlp is not None else None}
        if l.weights_of is not None:
            d["weights_of"] = l.weights_of
        layers.append(d)
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "layers": layers,
            "norm": {"eps": cfg.norm_eps}, "embedding": {"scale": cfg.embedding_scale}}


def domilix_config_from_json(d: Mapping[str, Any], dtype: str = "bfloat16") -> HybridConfig:
    """The `config.json` of a Domilix model: latent attention (cached latents may be shared between layers), dense or
    mixture-of-experts feed-forwards, RMS norms on the sublayers' outputs."""
    _check_model_keys(d)
    layers: List[HybridLayer] = []
    for i, l in enumerate(d["layers"]):
        at = f"layers[{i}]"
        l = _take(l, at, ("type", "mixer"), ("mlp",))
        if l["type"] != "latent_attention":
            raise ConfigError(f"{at}.type: unknown mixer {l['type']!r}")
        m = _take(l["mixer"], f"{at}.mixer", ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale"), ("rot", "kv_from"))
        rot = m.pop("rot", None)
        if rot is not None:
            rot = RotaryConfig(**_take(rot, f"{at}.mixer.rot", ("base", "dims")), interleaved=True)
        mlp: Optional[Mlp] = None
        if l.get("mlp") is not None:
            p = l["mlp"]
            kind = p.get("kind") if isinstance(p, Mapping) else None
            if kind == "dense":
                mlp = DenseMlp(_take(p, f"{at}.mlp", ("kind", "ff"))["ff"], "relu")
            elif kind == "moe":
                p = _take(p, f"{at}.mlp", ("kind", "expert", "router"))
                r = _take(p["router"], f"{at}.mlp.router", ("experts", "top"))
                mlp = MoeMlp(r["experts"], r["top"], _take(p["expert"], f"{at}.mlp.expert", ("ff",))["ff"])
            else:
                raise ConfigError(f"{at}.mlp.kind: unknown feed-forward {kind!r}")
        layers.append(HybridLayer(LatentAttentionMixer(**m, rotary=rot), mlp))
    cfg = HybridConfig(d["vocab"], d["width"], tuple(layers), _take(d["norm"], "norm", ("eps",))["eps"],
                       _take(d["embedding"], "embedding", ("scale",))["scale"], dtype, architecture="Domilix", block="post_norm")
    cfg.validate()
    return cfg


def domilix_config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    """The inverse of `domilix_config_from_json`."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        mixer: Dict[str, Any] = {k: getattr(m, k) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale")}
        if m.rotary is not None:
            mixer["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
        if m.kv_from is not None:
            mixer["kv_from"] = m.kv_from
        p = l.mlp
        mlp = None if p is None else {"kind": "dense", "ff": p.ff} if p.kind == "dense" else \
            {"kind": "moe", "expert": {"ff": p.ff}, "router": {"experts": p.experts, "top": p.top}}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "layers": layers,
            "norm": {"eps": cfg.norm_eps}, "embedding": {"scale": cfg.embedding_scale}}


def fanulix_config_from_json(d: Mapping[str, Any], dtype: str = "bfloat16") -> HybridConfig:
    """The `config.json` of a Fanulix model: residual streams over layers of Mamba-2, or of softmax attention beside retention, each
    with an optional mixture of experts."""
    _check_model_keys(d, ("streams", "logit_scale"))
    layers: List[HybridLayer] = []
    for i, l in enumerate(d["layers"]):
        at = f"layers[{i}]"
        l = _take(l, at, ("type", "mixer"), ("mlp",))
        if l["type"] == "mamba2":
            mixer: Mixer = Mamba2Mixer(**_take(l["mixer"], f"{at}.mixer", ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        elif l["type"] == "parallel":
            m = _take(l["mixer"], f"{at}.mixer", ("left", "right", "left_scale", "right_scale"))
            a = _take(m["left"], f"{at}.mixer.left", ("heads", "kv_heads", "dim", "vdim", "scale", "q_temp"))
            a["q_temp"] = QueryTemperature(**_take(a["q_temp"], f"{at}.mixer.left.q_temp", ("coef", "every")))
            r = _take(m["right"], f"{at}.mixer.right", ("heads", "dim", "vdim", "decay", "rot"))
            rot = RotaryConfig(**_take(r.pop("rot"), f"{at}.mixer.right.rot", ("base", "dims")))
            if not isinstance(r["decay"], Sequence) or isinstance(r["decay"], str):
                raise ConfigError(f"{at}.mixer.right.decay is not a list")
            r["decay"] = tuple(r["decay"])
            mixer = ParallelMixer(GroupedAttentionMixer(**a), RetentionMixer(**r, rotary=rot), m["left_scale"], m["right_scale"])
        else:
            raise ConfigError(f"{at}.type: unknown mixer {l['type']!r}")
        mlp: Optional[Mlp] = None
        if l.get("mlp") is not None:
            p = _take(l["mlp"], f"{at}.mlp", ("kind", "expert", "router", "shared"))
            if p["kind"] != "moe":
                raise ConfigError(f"{at}.mlp.kind: unknown feed-forward {p['kind']!r}")
            r = _take(p["router"], f"{at}.mlp.router", ("experts", "top"))
            ff = [_take(p[k], f"{at}.mlp.{k}", ("ff",))["ff"] for k in ("expert", "shared")]
            for k, v in (("expert", ff[0]), ("shared", ff[1]), ("router", r["top"])):
                if not isinstance(v, int) or isinstance(v, bool) or v < 1:
                    raise ConfigError(f"{at}.mlp.{k}: {v!r} must be a positive integer")
            mlp = MoeMlp(r["experts"], r["top"], ff[0], "gelu", False, ff[1])
        layers.append(HybridLayer(mixer, mlp))
    cfg = HybridConfig(d["vocab"], d["width"], tuple(layers), _take(d["norm"], "norm", ("eps",))["eps"], 1.0, dtype,
                       architecture="Fanulix", block="streams", streams=d["streams"], tied_head=True, logit_scale=d["logit_scale"])
    cfg.validate()
    return cfg


def fanulix_config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    """The inverse of `fanulix_config_from_json`."""
    layers = []
    for l in cfg.layers:
        m, p = l.mixer, l.mlp
        if m.kind == "mamba2":
            mixer: Dict[str, Any] = dataclasses.asdict(m)
        else:
            a, r = m.left, m.right
            left = {k: getattr(a, k) for k in ("heads", "kv_heads", "dim", "vdim", "scale")}
            left["q_temp"] = dataclasses.asdict(a.q_temp)
            right = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay),
                     "rot": {"base": r.rotary.base, "dims": r.rotary.dims}}
            mixer = {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}
        mlp = None if p is None else {"kind": "moe", "expert": {"ff": p.ff}, "router": {"experts": p.experts, "top": p.top},
                                      "shared": {"ff": p.shared_ff}}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "streams": cfg.streams,
            "layers": layers, "norm": {"eps": cfg.norm_eps}, "logit_scale": cfg.logit_scale}


def fogizen_config_from_json(d: Mapping[str, Any], dtype: str = "bfloat16") -> HybridConfig:
    """The `config.json` of a Fogizen model: shifted blocks of talking-heads attention beside time mixing, with a dense feed-forward, a
    mixture of experts or none, over token and bigram embeddings."""
    _check_model_keys(d)
    layers: List[HybridLayer] = []
    for i, l in enumerate(d["layers"]):
        at = f"layers[{i}]"
        l = _take(l, at, ("type", "mixer"), ("mlp",))
        if l["type"] != "parallel":
            raise ConfigError(f"{at}.type: unknown mixer {l['type']!r}")
        m = _take(l["mixer"], f"{at}.mixer", ("left", "right"))
        a = _take(m["left"], f"{at}.mixer.left", ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"))
        chunk = _take(a.pop("mask"), f"{at}.mixer.left.mask", ("size",))["size"]
        if chunk is None:
            raise ConfigError(f"{at}.mixer.left.mask.size: None must be a positive integer")
        r = _take(a.pop("rot"), f"{at}.mixer.left.rot", ("base", "dims"), ("scaling",))
        sc = r.get("scaling")
        if sc is not None:
            sc = LinearScaling(**_take(sc, f"{at}.mixer.left.rot.scaling", ("factor",)))
        left = TalkingAttentionMixer(**a, chunk=chunk, rotary=RotaryConfig(r["base"], r["dims"], sc, interleaved=True))
        right = TimeMixMixer(**_take(m["right"], f"{at}.mixer.right", ("heads", "dim")))
        mlp: Optional[Mlp] = None
        if l.get("mlp") is not None:
            p = l["mlp"]
            kind = p.get("kind") if isinstance(p, Mapping) else None
            if kind == "dense":
                mlp = DenseMlp(_take(p, f"{at}.mlp", ("kind", "ff"))["ff"], "xielu")
            elif kind == "moe":
                p = _take(p, f"{at}.mlp", ("kind", "expert", "router"))
                r = _take(p["router"], f"{at}.mlp.router", ("experts", "top", "scale"), ("groups",))
                g = _take(r["groups"], f"{at}.mlp.router.groups", ("count", "keep")) if r.get("groups") is not None else {"count": 1, "keep": 1}
                mlp = MoeMlp(r["experts"], r["top"], _take(p["expert"], f"{at}.mlp.expert", ("ff",))["ff"], "silu", False,
                             scoring="sigmoid", groups=g["count"], keep=g["keep"], scale=r["scale"])
            else:
                raise ConfigError(f"{at}.mlp.kind: unknown feed-forward {kind!r}")
        layers.append(HybridLayer(ParallelMixer(left, right, 0.5, 0.5, True), mlp))
    e = _take(d["embedding"], "embedding", ("bigram",))
    cfg = HybridConfig(d["vocab"], d["width"], tuple(layers), _take(d["norm"], "norm", ("eps",))["eps"], 1.0, dtype,
                       architecture="Fogizen", block="shifted",
                       bigram=BigramTable(**_take(e["bigram"], "embedding.bigram", ("buckets", "mul_prev", "mul_cur"))))
    cfg.validate()
    return cfg


def fogizen_config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    """The inverse of `fogizen_config_from_json` (the decay's rank is the checkpoint's)."""
    layers = []
    for l in cfg.layers:
        a, r, p = l.mixer.left, l.mixer.right, l.mlp
        left = {k: getattr(a, k) for k in ("heads", "kv_heads", "dim", "vdim", "scale")}
        left["mask"] = {"size": a.chunk}
        left["rot"] = {"base": a.rotary.base, "dims": a.rotary.dims}
        if a.rotary.scaling is not None:
            left["rot"]["scaling"] = dataclasses.asdict(a.rotary.scaling)
        if p is None:
            mlp = None
        elif p.kind == "dense":
            mlp = {"kind": "dense", "ff": p.ff}
        else:
            mlp = {"kind": "moe", "expert": {"ff": p.ff}, "router": {"experts": p.experts, "top": p.top, "scale": p.scale,
                                                                     "groups": {"count": p.groups, "keep": p.keep}}}
        layers.append({"type": "parallel", "mixer": {"left": left, "right": {"heads": r.heads, "dim": r.dim}}, "mlp": mlp})
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "layers": layers,
            "norm": {"eps": cfg.norm_eps}, "embedding": {"bigram": dataclasses.asdict(cfg.bigram)}}


def _mixer_from_dict(d: Mapping[str, Any]) -> Mixer:
    m = dict(d)
    if "left" in m:
        return ParallelMixer(**{**m, "left": _mixer_from_dict(m["left"]), "right": _mixer_from_dict(m["right"])})
    r = m.pop("rotary", None)
    if r is not None:
        r = dict(r)
        sc = r.pop("scaling", None)
        if sc is not None:
            sc = YarnScaling(**sc) if "original" in sc else LinearScaling(**sc)
        r = RotaryConfig(**r, scaling=sc)
    if "q_temp" in m:
        return GroupedAttentionMixer(**{**m, "q_temp": QueryTemperature(**m["q_temp"]) if m["q_temp"] is not None else None})
    if "chunk" in m:
        return TalkingAttentionMixer(**m, rotary=r)
    if "rank" in m:
        return TimeMixMixer(**m)
    if "decay" in m:
        return RetentionMixer(**{**m, "decay": tuple(m["decay"])}, rotary=r)
    if "state" in m:
        return Mamba2Mixer(**m)
    if "kv_heads" in m:
        return AttentionMixer(**m, rotary=r)
    if "kv_rank" in m:
        return LatentAttentionMixer(**m, rotary=r)
    return MlstmMixer(**m)


def hybrid_config_from_dict(d: Mapping[str, Any]) -> HybridConfig:
    """The inverse of `dataclasses.asdict(HybridConfig)` (the "model" section of an EngineConfig dictionary)."""
    d = dict(d)
    layers = []
    for l in d.pop("layers"):
        p = l.get("mlp")
        mlp: Optional[Mlp] = None if p is None else MoeMlp(**p) if "experts" in p else DenseMlp(**p)
        layers.append(HybridLayer(_mixer_from_dict(l["mixer"]), mlp, l.get("weights_of")))
    if d.get("bigram") is not None:
        d["bigram"] = BigramTable(**d["bigram"])
    cfg = HybridConfig(layers=tuple(layers), **d)
    cfg.validate()
    return cfg


def hybrid_stack(n_layers: int, width: int, heads: int, kv_heads: int, dim: int, window: int, ff: int, vocab: int,
                 mlstm_heads: int, mlstm_dim: int, mlstm_vdim: int, attention_every: int = 2, dtype: str = "bfloat16",
                 yarn: Optional[YarnScaling] = None, rot_dims: Optional[int] = None) -> HybridConfig:
    """A Timalorn-shaped decoder of `n_layers` with one attention layer in every `attention_every` (the rest mLSTM)."""
    att = AttentionMixer(heads, kv_heads, dim, window, dim ** -0.5, RotaryConfig(10000.0, rot_dims or dim // 2, yarn), 50.0)
    rec = MlstmMixer(mlstm_heads, mlstm_dim, mlstm_vdim, 15.0)
    layers = tuple(HybridLayer(att if i % attention_every == attention_every - 1 else rec, DenseMlp(ff))
                   for i in range(n_layers))
    cfg = HybridConfig(vocab, width, layers, 1e-6, math.sqrt(width), dtype)
    cfg.validate()
    return cfg


def latent_stack(n_layers: int, width: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, ff: int,
                 experts: int, top: int, expert_ff: int, vocab: int, share_from: Optional[int] = None,
                 dtype: str = "bfloat16") -> HybridConfig:
    """A Domilix-shaped decoder: the first layer's feed-forward is dense, the others' are mixtures of experts (experts 0: all
    dense); layers after `share_from` attend over that layer's latents."""
    rot = RotaryConfig(10000.0, rot_dim, interleaved=True) if rot_dim else None
    layers = []
    for i in range(n_layers):
        src = share_from if share_from is not None and i > share_from else None
        mixer = LatentAttentionMixer(heads, dim, rot_dim, vdim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, rot, src)
        layers.append(HybridLayer(mixer, DenseMlp(ff, "relu") if i == 0 or experts == 0 else MoeMlp(experts, top, expert_ff)))
    cfg = HybridConfig(vocab, width, tuple(layers), 1e-5, 1.0, dtype, architecture="Domilix", block="post_norm")
    cfg.validate()
    return cfg


def streams_stack(n_layers: int, width: int, streams: int, heads: int, kv_heads: int, dim: int, vdim: int, ret_heads: int,
                  ret_dim: int, ret_vdim: int, ssm_heads: int, ssm_vdim: int, ssm_state: int, ssm_groups: int, experts: int, top: int,
                  expert_ff: int, shared_ff: int, vocab: int, conv: int = 4, parallel_every: int = 2,
                  dtype: str = "bfloat16") -> HybridConfig:
    """A Fanulix-shaped decoder: one layer of attention beside retention in every `parallel_every` (the rest Mamba-2), a mixture of
    experts in each."""
    decay = tuple(1.0 - 2.0 ** (-5.0 - 7.0 * i / max(1, ret_heads - 1)) for i in range(ret_heads))
    both = ParallelMixer(GroupedAttentionMixer(heads, kv_heads, dim, vdim, dim ** -0.5, QueryTemperature(0.1, 4096)),
                         RetentionMixer(ret_heads, ret_dim, ret_vdim, decay, RotaryConfig(10000.0, ret_dim)), 0.7, 0.6)
    ssm = Mamba2Mixer(ssm_heads, ssm_vdim, ssm_state, ssm_groups, conv, ssm_groups)
    mlp = MoeMlp(experts, top, expert_ff, "gelu", False, shared_ff)
    layers = tuple(HybridLayer(both if i % parallel_every == parallel_every - 1 else ssm, mlp) for i in range(n_layers))
    cfg = HybridConfig(vocab, width, layers, 1e-6, 1.0, dtype, architecture="Fanulix", block="streams", streams=streams, tied_head=True,
                       logit_scale=0.5)
    cfg.validate()
    return cfg


def shifted_stack(n_layers: int, width: int, heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, mix_heads: int, mix_dim: int,
                  rank: int, ff: int, experts: int, top: int, groups: int, keep: int, expert_ff: int, vocab: int,
                  dtype: str = "bfloat16") -> HybridConfig:
    """A Fogizen-shaped decoder: the first layer's feed-forward is dense, the others' are mixtures of experts (experts 0: all dense)."""
    both = ParallelMixer(TalkingAttentionMixer(heads, kv_heads, dim, vdim, dim ** -0.5, chunk,
                                               RotaryConfig(10000.0, dim, LinearScaling(4.0), interleaved=True)),
                         TimeMixMixer(mix_heads, mix_dim, rank), 0.5, 0.5, True)
    moe = MoeMlp(experts, top, expert_ff, "silu", False, scoring="sigmoid", groups=groups, keep=keep, scale=1.5) if experts else None
    layers = tuple(HybridLayer(both, DenseMlp(ff, "xielu") if i == 0 or moe is None else moe) for i in range(n_layers))
    cfg = HybridConfig(vocab, width, layers, 1e-5, 1.0, dtype, architecture="Fogizen", block="shifted", bigram=BigramTable(vocab - 1, 31, 7))
    cfg.validate()
    return cfg


def tiny_shifted_config(**over: Any) -> HybridConfig:
    """CPU-sized Fogizen-shaped decoder: a dense layer, a mixture of experts in groups, and a layer without feed-forward."""
    both = ParallelMixer(TalkingAttentionMixer(4, 2, 20, 28, 0.21, 24, RotaryConfig(3000.0, 12, LinearScaling(2.5), interleaved=True)),
                         TimeMixMixer(3, 20), 0.5, 0.5, True)
    moe = MoeMlp(6, 2, 40, "silu", False, scoring="sigmoid", groups=3, keep=2, scale=1.3)
    kw: Dict[str, Any] = dict(vocab_size=300, hidden_size=88, norm_eps=2e-5, architecture="Fogizen", block="shifted",
                              bigram=BigramTable(97, 13, 5),
                              layers=(HybridLayer(both, DenseMlp(104, "xielu")), HybridLayer(both, moe), HybridLayer(both, None)))
    kw.update(over)
    cfg = HybridConfig(**kw)
    cfg.validate()
    return cfg


def tiny_streams_config(**over: Any) -> HybridConfig:
    """CPU-sized Fanulix-shaped decoder: attention beside retention, Mamba-2, and a Mamba-2 layer without feed-forward."""
    both = ParallelMixer(GroupedAttentionMixer(4, 2, 20, 28, 0.21, QueryTemperature(0.25, 24)),
                         RetentionMixer(3, 16, 20, (0.9, 0.97, 0.995), RotaryConfig(3000.0, 12)), 0.8, 0.45)
    kw: Dict[str, Any] = dict(vocab_size=300, hidden_size=88, norm_eps=2e-5, architecture="Fanulix", block="streams", streams=2,
                              tied_head=True, logit_scale=0.6,
                              layers=(HybridLayer(both, MoeMlp(6, 2, 40, "gelu", False, 72)),
                                      HybridLayer(Mamba2Mixer(4, 24, 20, 2, 4, 2), MoeMlp(5, 3, 24, "gelu", False, 24)),
                                      HybridLayer(Mamba2Mixer(3, 16, 12, 1, 3, 1), None)))
    kw.update(over)
    cfg = HybridConfig(**kw)
    cfg.validate()
    return cfg


def tiny_latent_config(**over: Any) -> HybridConfig:
    """CPU-sized Domilix-shaped decoder: dense, mixture of experts over the first layer's latents, and a layer without
    feed-forward."""
    rot = RotaryConfig(3000.0, 12, interleaved=True)
    own = LatentAttentionMixer(3, 20, 12, 28, 40, 36, 0.21, rot)
    kw: Dict[str, Any] = dict(vocab_size=300, hidden_size=88, norm_eps=2e-5, embedding_scale=1.5, architecture="Domilix",
                              block="post_norm",
                              layers=(HybridLayer(own, DenseMlp(104, "relu")),
                                      HybridLayer(dataclasses.replace(own, heads=2, kv_from=0), MoeMlp(6, 2, 40)),
                                      HybridLayer(own, None)))
    kw.update(over)
    cfg = HybridConfig(**kw)
    cfg.validate()
    return cfg


def tiny_hybrid_config(**over: Any) -> HybridConfig:
    """CPU-sized Timalorn-shaped decoder: mLSTM, attention, a second attention layer with the first one's weights, and an
    mLSTM layer without feed-forward."""
    att = AttentionMixer(4, 2, 24, 40, 0.2, RotaryConfig(5000.0, 8, YarnScaling(4.0, 64, 8.0, 1.0)), 30.0)
    rec = MlstmMixer(3, 16, 24, 9.0)
    kw: Dict[str, Any] = dict(vocab_size=300, hidden_size=88, norm_eps=1e-5, embedding_scale=7.5,
                              layers=(HybridLayer(rec, DenseMlp(104)), HybridLayer(att, DenseMlp(104)),
                                      HybridLayer(att, DenseMlp(104), 1), HybridLayer(rec, None)))
    kw.update(over)
    cfg = HybridConfig(**kw)
    cfg.validate()
    return cfg


@dataclass(frozen=True)
class ParallelConfig:
    tp_size: int = 1
    ep_size: int = 1             # experts partitioned over ep ranks (== tp group)
    pp_size: int = 1
    dcp_size: int = 1            # decode context parallel (KV interleave)
    indexer_sp: bool = True      # sequence-parallel indexer scoring for prefill chunks
    indexer_sp_min_rows: int = 256
    fused_collectives: bool = True   # False => NCCL-after-GEMM baseline paths
    eplb_redundant: int = 0          # spare physical expert slots per layer for replicas of hot experts (EPLB)
    eplb_record: bool = False        # count routed tokens per logical expert and layer (input of a rebalance)
    use_multimem: bool = False       # NVLS multimem loads/stores in the all-reduce

    def validate(self) -> None:
        for name in ("tp_size", "ep_size", "pp_size", "dcp_size"):
            if getattr(self, name) < 1:
                raise ConfigError(f"{name} must be >= 1")
        if self.ep_size not in (1, self.tp_size):
            raise ConfigError("ep_size must be 1 or equal tp_size")
        if self.eplb_redundant < 0 or self.eplb_redundant % self.tp_size:
            raise ConfigError("eplb_redundant must be a non-negative multiple of tp_size")


@dataclass(frozen=True)
class CacheConfig:
    page_tokens: int = 64            # rows per page in every cache group
    engine_block_tokens: int = 256   # scheduler-visible block (4 SWA pages, 1 C4A page)
    gpu_memory_utilization: float = 0.60
    num_pages: Optional[int] = None  # explicit pool size (tests / bench)
    enable_prefix_caching: bool = True
    # Context tokens the compressed-KV pools hold over all requests together.  None: room for max_num_seqs requests of
    # max_model_len each (nothing ever waits for pages).  With `size_by_memory` the engine derives it on a GPU from
    # gpu_memory_utilization x device memory minus what is allocated when it starts (the weights).
    kv_pool_tokens: Optional[int] = None
    size_by_memory: bool = False

    def validate(self) -> None:
        if self.page_tokens != 64:
            raise ConfigError("page_tokens must be 64")
        if self.engine_block_tokens % self.page_tokens:
            raise ConfigError("engine block must be a whole number of pages")
        if not (0.0 < self.gpu_memory_utilization <= 0.98):
            raise ConfigError("gpu_memory_utilization out of range")


@dataclass(frozen=True)
class SchedulerConfig:
    max_model_len: int = 430000
    max_num_seqs: int = 32
    max_num_batched_tokens: int = 4096
    graph_cap: int = 256             # largest decode batch captured as a CUDA graph
    decode_first: bool = True
    # Schedule and launch step k+1 before the tokens of step k are read: a decode row's input token is copied on the
    # device from the previous step's samples, the host reads them while the next step runs, and a request that turns
    # out to have ended (EOS) has one surplus row computed and dropped.  Off by default; not with speculative decoding.
    async_scheduling: bool = False

    def validate(self) -> None:
        if self.max_num_seqs < 1 or self.max_num_batched_tokens < 1:
            raise ConfigError("scheduler limits must be positive")
        if self.graph_cap < 0:
            raise ConfigError("graph_cap must be >= 0")


@dataclass(frozen=True)
class SpecConfig:
    method: str = "none"             # "none" | "dspark"
    num_speculative_tokens: int = 5
    markov_topk: int = 512           # 0 => dense Markov bias over the whole vocab
    temperature: float = 0.6
    markov_sideload: str = ""
    replicate_markov: bool = True

    def validate(self) -> None:
        if self.method not in ("none", "dspark"):
            raise ConfigError(f"unknown speculative method {self.method!r}")
        if self.method == "dspark" and not (1 <= self.num_speculative_tokens <= 15):
            raise ConfigError("num_speculative_tokens must be in [1, 15]")
        if self.markov_topk < 0:
            raise ConfigError("markov_topk must be >= 0")


@dataclass(frozen=True)
class KernelConfig:
    compressor_fp8: bool = True
    target_lm_head_fp8: bool = True
    fused_gate: bool = True
    oneshot_max_bytes: int = 512 * 1024   # one-shot all-reduce up to here, two-shot above
    wait_budget_iters: int = 4_000_000    # bound of every device-side spin
    multi_stream: bool = True

    def validate(self) -> None:
        if self.oneshot_max_bytes < 0 or self.wait_budget_iters < 1:
            raise ConfigError("kernel limits must be positive")


@dataclass(frozen=True)
class EngineConfig:
    model: Union[ModelConfig, "HybridConfig"] = field(default_factory=ModelConfig)
    parallel: ParallelConfig = field(default_factory=ParallelConfig)
    cache: CacheConfig = field(default_factory=CacheConfig)
    sched: SchedulerConfig = field(default_factory=SchedulerConfig)
    spec: SpecConfig = field(default_factory=SpecConfig)
    kernels: KernelConfig = field(default_factory=KernelConfig)
    seed: int = 0

    def validate(self) -> "EngineConfig":
        for part in (self.model, self.parallel, self.cache, self.sched, self.spec, self.kernels):
            part.validate()
        self.model.check_engine(self)
        if self.spec.method == "dspark" and self.parallel.pp_size > 1:
            # The reference refuses DSpark under pipeline parallelism
            # (overlay/dspark_utils_v2.py:158-159).
            raise ConfigError("dspark speculative decoding does not support pp_size > 1")
        return self

    # ---- (de)serialisation --------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)

    def resolved(self) -> str:
        """The resolved configuration as printed at start-up."""
        return json.dumps(self.to_dict(), indent=1, sort_keys=True)

    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "EngineConfig":
        def build(cls, sub):
            sub = dict(sub or {})
            names = {f.name for f in dataclasses.fields(cls)}
            unknown = set(sub) - names
            if unknown:
                raise ConfigError(f"unknown {cls.__name__} keys: {sorted(unknown)}")
            for k, v in list(sub.items()):
                if isinstance(v, list):
                    sub[k] = tuple(v)
            return cls(**sub)

        known = {"model", "parallel", "cache", "sched", "spec", "kernels", "seed"}
        unknown = set(d) - known
        if unknown:
            raise ConfigError(f"unknown EngineConfig sections: {sorted(unknown)}")
        m = d.get("model")
        return EngineConfig(
            model=hybrid_config_from_dict(m) if isinstance(m, Mapping) and "layers" in m else build(ModelConfig, m),
            parallel=build(ParallelConfig, d.get("parallel")),
            cache=build(CacheConfig, d.get("cache")),
            sched=build(SchedulerConfig, d.get("sched")),
            spec=build(SpecConfig, d.get("spec")),
            kernels=build(KernelConfig, d.get("kernels")),
            seed=int(d.get("seed", 0)),
        ).validate()


def model_config_from_hf(hf: Dict[str, Any]) -> ModelConfig:
    """Build a ModelConfig from a DeepSeek-V4 ``config.json`` dictionary."""
    names = {f.name for f in dataclasses.fields(ModelConfig)}
    kw = {k: (tuple(v) if isinstance(v, list) else v) for k, v in hf.items() if k in names}
    if "expert_dtype" in hf and hf["expert_dtype"] == "fp4":
        kw["expert_dtype"] = "mxfp4"    # checkpoint layout: e2m1 + ue8m0 per 32
    cfg = ModelConfig(**kw)
    cfg.validate()
    return cfg
