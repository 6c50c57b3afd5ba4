"""Model geometry for the supported decoder families.

One dataclass covers plain dense decoders, the Qwen3.5-family hybrid
(Gated-DeltaNet linear attention + gated full attention, dense or MoE FFN) and
Gemma 4 (sliding-window/global attention + MoE).  The three pinned Qwen3.5
geometries mirror the identities the reference pins in
``hipengine/kernels/policy.py:103-153``; the Gemma 4 26B-A4B numbers come from
``docs/model-cards/MODEL-GEMMA4.md:128-155`` of the reference.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import Dict, Optional, Tuple, Union

# head widths the attention kernels are built for; narrower heads are zero-padded to the next one at load
HEAD_WIDTHS = (64, 128, 256, 512)


def padded_head_width(d: int) -> int:
    for w in HEAD_WIDTHS:
        if d <= w:
            return w
    raise ValueError(f"head width {d} is above the widest supported one ({HEAD_WIDTHS[-1]})")


@dataclass(frozen=True)
class YarnSpec:
    """Context extension of a rotary table: slow pairs are slowed down by ``factor``, fast ones are kept."""
    factor: float
    original: float                      # context the unscaled table was made for
    fast: float                          # turns over that context from which a pair counts as fast ...
    slow: float                          # ... and below which as slow


@dataclass(frozen=True)
class BandSpec:
    """Context extension by wave length (Llama 3.1): waves that fit ``high`` times into the original context are kept, those
    that fit less than ``low`` times are slowed down by ``factor``, those between are mixed."""
    factor: float
    low: float
    high: float
    original: float

    def scaled(self, freq: float) -> float:
        turns = self.original * freq / (2 * math.pi)
        if turns >= self.high:
            return freq
        if turns <= self.low:
            return freq / self.factor
        keep = (turns - self.low) / (self.high - self.low)
        return (1.0 - keep) * freq / self.factor + keep * freq


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of pairs by position * base^(-2i / dims): of neighbours (2i, 2i + 1), or with ``halves`` of (i, i + dims / 2)."""
    dims: int
    base: float
    scaling: Optional[Union[YarnSpec, BandSpec]] = None
    halves: bool = False

    def table(self) -> Tuple[Tuple[float, ...], float]:
        """(angular frequency per pair, amplitude of sine and cosine)."""
        freq = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        y = self.scaling
        if y is None:
            return tuple(freq), 1.0
        if isinstance(y, BandSpec):
            return tuple(y.scaled(f) for f in freq), 1.0
        at = lambda turns: self.dims * math.log(y.original / (2 * math.pi * turns)) / (2 * math.log(self.base))
        lo, hi = max(math.floor(at(y.fast)), 0), min(math.ceil(at(y.slow)), self.dims - 1)
        for i, f in enumerate(freq):
            slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            freq[i] = f * (slow / y.factor + 1.0 - slow)
        return tuple(freq), 0.1 * math.log(y.factor) + 1.0


# how queries and keys are normalised
QK_NORM_NONE = "none"
QK_NORM_HEAD = "head"                    # every head over its own width, gains per dimension, before the rotation
QK_NORM_ROWS = "rows"                    # the whole projection at once, gains per column, before the rotation
QK_NORM_UNIT = "unit"                    # every head over its own width, no gains, after the rotation


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention of one layer, for designs whose layers are listed one by one."""
    heads: int
    kv_heads: int
    dim: int                             # query / key width per head
    vdim: int                            # value width per head
    scale: float
    softcap: float = 0.0                 # > 0: score <- softcap * tanh(score / softcap)
    rot: Optional[RotarySpec] = None     # of the first ``rot.dims`` dimensions of queries and keys
    window: int = 0                      # > 0: only the last ``window`` positions are visible ...
    keep_first: int = 0                  # ... and the sequence's first ``keep_first`` ones
    sink_score: Optional[float] = None   # score of a term in the softmax denominator that has no value
    qk_norm: str = QK_NORM_HEAD
    bias: bool = False                   # of the query, key and value projections
    keys_as_values: bool = False         # the values are the projected keys, before norm and rotation
    head_gate: bool = False              # sigmoid(w_g . h) per head on the output
    kv_from: Optional[int] = None        # attends to the keys and values of this earlier layer and has none of its own
    head_scale: bool = False             # a learned factor per head on the scores
    out_bias: bool = False               # of the output projection

    @property
    def width(self) -> int:
        """Width a head takes in the KV pages (both planes)."""
        return padded_head_width(max(self.dim, self.vdim))

    @property
    def cache_elems(self) -> int:
        """Elements a token takes in the layer's cache plane."""
        return 0 if self.kv_from is not None else 2 * self.kv_heads * self.width

    @property
    def state_elems(self) -> int:
        return 0

    def check(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads over {self.kv_heads} key/value heads, {self.dim} / {self.vdim} wide")
        if self.rot is not None and not (self.rot.dims % 2 == 0 and 2 <= self.rot.dims <= self.dim):
            raise ValueError(f"rotation of {self.rot.dims} of {self.dim} dimensions")
        if self.keys_as_values and self.vdim != self.dim:
            raise ValueError(f"keys of {self.dim} dimensions as values of {self.vdim}")
        if self.window < 0 or self.keep_first < 0:
            raise ValueError(f"window of {self.window}, {self.keep_first} first tokens kept")
        padded_head_width(max(self.dim, self.vdim))


# bounds of the latent attention kernels: padded latent columns, and those plus the padded rotated part
LATENT_MAX_RANK = 1024
LATENT_MAX_ROW = 1280


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are linear maps of one latent row per token (plus a rotated key part shared by
    all heads); only the latent and the rotated part are cached."""
    heads: int
    dim: int                             # unrotated query / key width per head
    rot_dim: int                         # rotated query / key width per head
    vdim: int
    kv_rank: int                         # latent width
    scale: float
    rot: RotarySpec
    q_rank: int = 0                      # > 0: queries go through a normalised latent of this width
    window: int = 0                      # > 0: only the last ``window`` positions are visible
    sink: bool = False                   # a learned term per head in the softmax denominator

    @property
    def rank_cols(self) -> int:
        """Columns of the latent in a cache row (zero-padded)."""
        return round_up(self.kv_rank, 16)

    @property
    def row_cols(self) -> int:
        """Columns of a cache row: latent, then the rotated part, zero-padded."""
        return round_up(self.rank_cols + self.rot_dim, 32)

    @property
    def cache_elems(self) -> int:
        return self.row_cols

    @property
    def state_elems(self) -> int:
        return 0

    def check(self) -> None:
        if min(self.heads, self.dim, self.vdim, self.kv_rank) < 1 or self.rot_dim < 2 or self.rot_dim % 2:
            raise ValueError(f"latent attention of {self.heads} heads, {self.dim} + {self.rot_dim} / {self.vdim} wide, "
                             f"latent {self.kv_rank}")
        if self.rot.dims != self.rot_dim:
            raise ValueError(f"rotary table over {self.rot.dims} dimensions for a rotated part of {self.rot_dim}")
        if self.rank_cols > LATENT_MAX_RANK or self.row_cols > LATENT_MAX_ROW:
            raise ValueError(f"latent of {self.kv_rank} + {self.rot_dim} columns is above the widest supported one "
                             f"({LATENT_MAX_RANK}, {LATENT_MAX_ROW} with the rotated part)")


@dataclass(frozen=True)
class RecurrentSpec:
    """Real-gated linear recurrence (RG-LRU) over a short causal convolution, gated by a GELU branch of the same width."""
    width: int
    blocks: int                          # the gates are block-diagonal maps of the convolution's output
    taps: int                            # of the convolution

    @property
    def block_cols(self) -> int:
        """Channels of a block, zero-padded."""
        return round_up(self.width // self.blocks, 8)

    @property
    def cols(self) -> int:
        return self.blocks * self.block_cols

    @property
    def state_elems(self) -> int:
        """fp32 numbers a request carries: one per channel, and the convolution's last inputs."""
        return self.cols * self.taps

    def check(self) -> None:
        if min(self.width, self.blocks, self.taps) < 1 or self.width % self.blocks:
            raise ValueError(f"recurrence of {self.width} channels in {self.blocks} blocks, {self.taps} taps")


@dataclass(frozen=True)
class SideBySideSpec:
    """Attention and a recurrence reading the same row; their outputs are added with a factor each."""
    left: AttentionSpec
    right: RecurrentSpec
    left_scale: float = 1.0
    right_scale: float = 1.0

    @property
    def window(self) -> int:
        return self.left.window

    @property
    def cache_elems(self) -> int:
        return self.left.cache_elems

    @property
    def state_elems(self) -> int:
        return self.right.state_elems

    def check(self) -> None:
        self.left.check()
        self.right.check()


# bounds of the linear attention kernels: key and value columns per head, taps of a convolution
LINEAR_MAX_DIM = 512
CONV_MAX_TAPS = 16
NORM_CONV_MAX_ROWS = 50 * 1024           # channels of a norm group times rows that its kernel keeps in shared memory


@dataclass(frozen=True)
class LinearAttentionSpec:
    """Linear attention with a matrix state per head: S <- g S + k w^T, o = S^T q, o normalised per head and gated by silu.

    ``decay`` given (retention): g is that constant per head, w the value, queries and keys are rotated.  Without it (gated
    delta rule): g and a step size b come from the row, w = b (v - g S^T k), queries, keys and values pass a short causal
    convolution and silu, queries and keys are unit vectors, the norm has gains."""
    heads: int
    kv_heads: int                        # query and key heads; head h uses number h // (heads / kv_heads)
    dim: int
    vdim: int
    decay: Optional[Tuple[float, ...]] = None
    rot: Optional[RotarySpec] = None
    taps: int = 1                        # of the convolution

    window = 0

    @property
    def delta(self) -> bool:
        return self.decay is None

    @property
    def vcols(self) -> int:
        """Value columns of a head, zero-padded."""
        return round_up(self.vdim, 8)

    @property
    def conv_cols(self) -> int:
        """Columns of the convolution: query, key and value rows, each zero-padded."""
        return 2 * round_up(self.kv_heads * self.dim, 8) + round_up(self.heads * self.vdim, 8)

    @property
    def cache_elems(self) -> int:
        return 0

    @property
    def state_elems(self) -> int:
        """fp32 numbers a request carries: the matrices, and a ring of the convolution's last inputs."""
        return self.heads * self.dim * self.vcols + (self.conv_cols * self.taps if self.delta and self.taps > 1 else 0)

    def check(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads over {self.kv_heads} query/key heads, {self.dim} / {self.vdim} wide")
        if max(self.dim, self.vdim) > LINEAR_MAX_DIM:
            raise ValueError(f"heads of {self.dim} / {self.vdim} columns are above the widest supported one ({LINEAR_MAX_DIM})")
        if not 1 <= self.taps <= CONV_MAX_TAPS:
            raise ValueError(f"convolution of {self.taps} taps")
        if self.decay is not None and (len(self.decay) != self.heads or min(self.decay) <= 0 or max(self.decay) > 1):
            raise ValueError(f"decays {self.decay} of {self.heads} heads")
        if self.rot is not None and not (self.rot.dims % 2 == 0 and 2 <= self.rot.dims <= self.dim):
            raise ValueError(f"rotation of {self.rot.dims} of {self.dim} dimensions")


@dataclass(frozen=True)
class DenseMlpSpec:
    ff: int
    act: str = "silu"                    # gated: "silu" | "gelu_tanh" | "clamped_glu"; ungated: "relu2"
    limit: float = 0.0                   # clamped_glu: bound of the gate (above) and of the up branch (both sides)


@dataclass(frozen=True)
class MoeMlpSpec:
    experts: int
    top: int
    ff: int
    groups: int = 1                      # groups of neighbouring experts ...
    groups_kept: int = 1                 # ... of which only the best ones may be chosen from
    scale: float = 1.0                   # factor on the normalised routing weights
    shared_ff: int = 0                   # > 0: shared expert, scaled per token by sigmoid(w_sg . h)
    score: str = "sigmoid"               # "sigmoid", normalised over the chosen experts | "softmax" over all, as it is
    act: str = "silu"                    # of the experts, as in DenseMlpSpec
    limit: float = 0.0

    def check(self) -> None:
        if min(self.experts, self.top, self.ff) < 1 or self.top > min(self.experts, 32) or self.experts > 512:
            raise ValueError(f"top {self.top} of {self.experts} experts of {self.ff} columns (up to 32 of 512 are supported)")


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, LatentAttentionSpec, SideBySideSpec, LinearAttentionSpec]
    mlp: Optional[Union[DenseMlpSpec, MoeMlpSpec]] = None
    parallel: bool = False               # both sublayers read one norm and are added together
    token_shift: bool = False            # the mixer reads a mix of this token's and the previous token's normalised row
    input_taps: int = 1                  # > 1: a causal convolution of the normalised rows is added to what the mixer reads

    @property
    def attention(self) -> Optional[Union[AttentionSpec, LatentAttentionSpec]]:
        """The part of the mixer that keeps a cache, if there is one."""
        if isinstance(self.mixer, LinearAttentionSpec):
            return None
        return self.mixer.left if isinstance(self.mixer, SideBySideSpec) else self.mixer

    def state_elems(self, hidden: int) -> int:
        """fp32 numbers a request carries for one run of this layer besides its cache rows."""
        return self.mixer.state_elems + round_up(hidden, 8) * (int(self.token_shift) + self.input_taps - 1)


@dataclass(frozen=True)
class LoopSpec:
    """Layers [start, stop) run ``times`` times in a row with the same weights, every pass with its own cache."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class ModelConfig:
    arch: str = "qwen35"                 # general.architecture of the GGUF file
    n_layers: int = 4
    hidden: int = 256
    vocab: int = 4096
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 64
    ffn: int = 768
    rms_eps: float = 1e-6
    rope_theta: float = 1e6
    rope_dim: int = 64                   # rotated dims per head (partial rotary when < head_dim)
    # attention flavour
    gated_attention: bool = False        # attn_q projects [Q | gate] per head; out *= sigmoid(gate)
    qk_norm: bool = False
    attn_scale: Optional[float] = None   # None -> head_dim ** -0.5
    # hybrid schedule: layer i is full attention iff (i + 1) % full_attention_interval == 0
    full_attention_interval: int = 0     # 0 -> every layer is full attention
    # Gated DeltaNet (linear attention) geometry
    ssm_groups: int = 0                  # number of K heads
    ssm_v_heads: int = 0                 # number of V heads (= time_step_rank)
    ssm_state: int = 128                 # Dk = Dv
    conv_kernel: int = 4
    # MoE
    n_experts: int = 0
    n_experts_used: int = 0
    expert_ffn: int = 0
    shared_ffn: int = 0
    # Gemma-style extras
    sliding_window: int = 0
    swa_pattern: int = 0                 # every swa_pattern-th layer is global, the rest sliding
    global_head_dim: int = 0
    global_kv_heads: int = 0
    final_softcap: float = 0.0
    embed_scale: float = 1.0
    act: str = "silu"                    # "silu" | "gelu_tanh"
    tie_embeddings: bool = False
    # MTP / NextN draft blocks appended after the main stack
    nextn_layers: int = 0
    max_context: int = 8192

    swa_rope_theta: float = 10000.0      # Gemma: sliding layers rotate the whole head with this base
    global_rope_fraction: float = 0.25   # Gemma: global layers rotate this fraction of the head ("proportional")

    # designs whose layers are listed one by one (``layer_specs``), some of them run repeatedly (``loop``)
    layer_specs: Tuple[LayerSpec, ...] = ()
    loop: Optional[LoopSpec] = None
    residual_mult: float = 1.0           # factor on what a layer adds to the residual
    norm_groups: int = 1                 # equal runs of channels that the norms of the residual are taken over

    # ---- derived
    def is_global_layer(self, i: int) -> bool:
        """Gemma-style schedule: every ``swa_pattern``-th layer attends globally, the rest use a sliding window."""
        return self.swa_pattern > 0 and (i + 1) % self.swa_pattern == 0

    def layer_head_dim(self, i: int) -> int:
        return self.global_head_dim if (self.is_global_layer(i) and self.global_head_dim) else self.head_dim

    def layer_kv_heads(self, i: int) -> int:
        return self.global_kv_heads if (self.is_global_layer(i) and self.global_kv_heads) else self.n_kv_heads

    def layer_window(self, i: int) -> int:
        return 0 if (self.swa_pattern == 0 or self.is_global_layer(i)) else self.sliding_window

    @property
    def is_hybrid(self) -> bool:
        return self.full_attention_interval > 0

    @property
    def has_recurrent_state(self) -> bool:
        """Does a request carry state besides its cache pages (prefix reuse then needs snapshots of it)?"""
        return self.is_hybrid or any(l.state_elems(self.hidden) for l in self.layer_specs)

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    @property
    def ssm_inner(self) -> int:
        return self.ssm_v_heads * self.ssm_state

    @property
    def linear_qkv_width(self) -> int:
        return 2 * self.ssm_groups * self.ssm_state + self.ssm_inner

    @property
    def q_width(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_width(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def q_proj_width(self) -> int:
        return self.q_width * (2 if self.gated_attention else 1)

    def is_full_attention_layer(self, i: int) -> bool:
        if not self.is_hybrid:
            return True
        return (i + 1) % self.full_attention_interval == 0

    def layer_kinds(self) -> Tuple[str, ...]:
        return tuple("full" if self.is_full_attention_layer(i) else "linear" for i in range(self.n_layers))

    @property
    def n_full_layers(self) -> int:
        return sum(1 for k in self.layer_kinds() if k == "full")

    @property
    def n_linear_layers(self) -> int:
        return self.n_layers - self.n_full_layers

    def scale(self) -> float:
        return self.attn_scale if self.attn_scale is not None else self.head_dim ** -0.5

    def layer_runs(self) -> Tuple[Tuple[int, int], ...]:
        """(layer, pass) in the order of execution; pass is -1 for a layer outside the loop.  A layer run, not a layer,
        owns a KV plane."""
        lp = self.loop
        if lp is None:
            return tuple((i, -1) for i in range(self.n_layers))
        runs = [(i, -1) for i in range(lp.start)]
        for t in range(lp.times):
            runs += [(i, t) for i in range(lp.start, lp.stop)]
        return tuple(runs + [(i, -1) for i in range(lp.stop, self.n_layers)])

    def kv_bytes_per_token(self, elem_bytes: int = 2) -> int:
        if self.layer_specs:
            return sum(self.layer_specs[i].mixer.cache_elems * elem_bytes for i, _ in self.layer_runs())
        return self.n_full_layers * 2 * self.n_kv_heads * self.head_dim * elem_bytes

    def recurrent_state_bytes(self) -> int:
        if self.layer_specs:
            return sum(4 * self.layer_specs[i].state_elems(self.hidden) for i, _ in self.layer_runs())
        gdn = self.n_linear_layers * self.ssm_v_heads * self.ssm_state * self.ssm_state * 4
        conv = self.n_linear_layers * self.linear_qkv_width * self.conv_kernel * 4
        return gdn + conv

    def with_layers(self, n_layers: int) -> "ModelConfig":
        if not self.layer_specs:
            return replace(self, n_layers=n_layers)
        lp = self.loop
        if lp is not None:
            stop = min(lp.stop, n_layers)
            lp = LoopSpec(lp.start, stop, lp.times) if lp.start < stop else None
        return replace(self, n_layers=n_layers, layer_specs=self.layer_specs[:n_layers], loop=lp)


# Tiny dense decoder of the CPU reference backend benchmark (4 layers, hidden 256, Q4_K weights).
TINY_DENSE = ModelConfig(arch="qwen3", n_layers=4, hidden=256, vocab=4096, n_heads=4, n_kv_heads=2,
                         head_dim=64, ffn=768, rms_eps=1e-6, rope_theta=1e6, rope_dim=64)

# Dense hybrid 27B: 64 layers [3 GDN + 1 gated full attention] x 16.
QWEN35_27B = ModelConfig(arch="qwen35", n_layers=64, hidden=5120, vocab=248320, n_heads=24, n_kv_heads=4,
                         head_dim=256, ffn=17408, rms_eps=1e-6, rope_theta=1e7, rope_dim=64,
                         gated_attention=True, qk_norm=True, full_attention_interval=4,
                         ssm_groups=16, ssm_v_heads=48, ssm_state=128, conv_kernel=4,
                         max_context=262144)

# MoE hybrid 35B-A3B: 40 layers, 256 experts top-8 + shared expert.
QWEN35_35B_A3B = ModelConfig(arch="qwen35moe", n_layers=40, hidden=2048, vocab=248320, n_heads=16, n_kv_heads=2,
                             head_dim=256, ffn=0, rms_eps=1e-6, rope_theta=1e7, rope_dim=64,
                             gated_attention=True, qk_norm=True, full_attention_interval=4,
                             ssm_groups=16, ssm_v_heads=32, ssm_state=128, conv_kernel=4,
                             n_experts=256, n_experts_used=8, expert_ffn=512, shared_ffn=512,
                             max_context=262144)

# Small hybrid used by tests and the smoke entry (same structure, toy widths).
TINY_HYBRID = ModelConfig(arch="qwen35", n_layers=4, hidden=512, vocab=2048, n_heads=4, n_kv_heads=2,
                          head_dim=256, ffn=1024, rope_theta=1e7, rope_dim=64, gated_attention=True,
                          qk_norm=True, full_attention_interval=4, ssm_groups=2, ssm_v_heads=4,
                          ssm_state=128, conv_kernel=4, max_context=4096)

# Small hybrid geometry whose heads / K-head groups / FFN blocks split evenly over 2 ranks.
TINY_HYBRID_TP = ModelConfig(arch="qwen35", n_layers=4, hidden=512, vocab=2048, n_heads=4, n_kv_heads=2,
                             head_dim=256, ffn=1024, rope_theta=1e7, rope_dim=64, gated_attention=True,
                             qk_norm=True, full_attention_interval=4, ssm_groups=4, ssm_v_heads=8,
                             ssm_state=128, conv_kernel=4, max_context=4096)

# The same at a geometry that splits over 2, 4 and 8 ranks (16 K-head groups -> 2 per rank at 8; 8 heads; 8 FFN blocks).
SMALL_HYBRID_TP8 = ModelConfig(arch="qwen35", n_layers=4, hidden=512, vocab=2048, n_heads=8, n_kv_heads=2,
                               head_dim=256, ffn=2048, rope_theta=1e7, rope_dim=64, gated_attention=True,
                               qk_norm=True, full_attention_interval=4, ssm_groups=16, ssm_v_heads=32,
                               ssm_state=128, conv_kernel=4, max_context=4096)

TINY_HYBRID_MOE_TP = ModelConfig(arch="qwen35moe", n_layers=4, hidden=512, vocab=2048, n_heads=4, n_kv_heads=2,
                                 head_dim=256, ffn=0, rope_theta=1e7, rope_dim=64, gated_attention=True,
                                 qk_norm=True, full_attention_interval=4, ssm_groups=4, ssm_v_heads=8,
                                 ssm_state=128, conv_kernel=4, n_experts=16, n_experts_used=4,
                                 expert_ffn=256, shared_ffn=256, max_context=4096)

TINY_HYBRID_MOE = ModelConfig(arch="qwen35moe", n_layers=4, hidden=512, vocab=2048, n_heads=4, n_kv_heads=2,
                              head_dim=256, ffn=0, rope_theta=1e7, rope_dim=64, gated_attention=True,
                              qk_norm=True, full_attention_interval=4, ssm_groups=2, ssm_v_heads=4,
                              ssm_state=128, conv_kernel=4, n_experts=16, n_experts_used=4,
                              expert_ffn=256, shared_ffn=256, max_context=4096)

# Gemma 4 26B-A4B: 30 layers, 5 sliding (window 1024) : 1 global.
GEMMA4_26B_A4B = ModelConfig(arch="gemma4", n_layers=30, hidden=2816, vocab=262144, n_heads=16, n_kv_heads=8,
                             head_dim=256, ffn=2112, rms_eps=1e-6, rope_theta=1e6, rope_dim=256,
                             qk_norm=True, attn_scale=1.0, sliding_window=1024, swa_pattern=6,
                             global_head_dim=512, global_kv_heads=2, n_experts=128, n_experts_used=8,
                             expert_ffn=704, final_softcap=30.0, embed_scale=2816 ** 0.5,
                             act="gelu_tanh", tie_embeddings=True, max_context=262144)

TINY_GEMMA4 = ModelConfig(arch="gemma4", n_layers=6, hidden=256, vocab=2048, n_heads=4, n_kv_heads=2,
                          head_dim=64, ffn=288, rope_theta=1e6, rope_dim=64, qk_norm=True, attn_scale=1.0,
                          sliding_window=32, swa_pattern=6, global_head_dim=128, global_kv_heads=1,
                          n_experts=8, n_experts_used=2, expert_ffn=128, final_softcap=30.0,
                          embed_scale=16.0, act="gelu_tanh", tie_embeddings=True, max_context=2048)


def sisisun_config(hidden: int, vocab: int, layers: Tuple[LayerSpec, ...], loop: Optional[LoopSpec] = None,
                   rms_eps: float = 1e-6, max_context: int = 262144) -> ModelConfig:
    """``ModelConfig`` of a Sisisun model: listed layers without rotation, sinusoidal position vector at the embedding,
    norm weights stored around zero, optional looped range.  The per-model fields of the other families are filled in
    from the layers for reports."""
    a = layers[0].mixer
    moe = [l.mlp for l in layers if isinstance(l.mlp, MoeMlpSpec)]
    dense = [l.mlp for l in layers if isinstance(l.mlp, DenseMlpSpec)]
    for i, l in enumerate(layers):
        if l.mixer.heads % l.mixer.kv_heads:
            raise ValueError(f"layer {i}: {l.mixer.heads} query heads over {l.mixer.kv_heads} key/value heads")
        if isinstance(l.mlp, MoeMlpSpec):
            m = l.mlp
            if m.experts % m.groups or not 1 <= m.groups_kept <= m.groups:
                raise ValueError(f"layer {i}: {m.experts} experts in {m.groups} groups, {m.groups_kept} kept")
            if not 1 <= m.top <= m.groups_kept * (m.experts // m.groups):
                raise ValueError(f"layer {i}: top {m.top} of {m.groups_kept} groups of {m.experts // m.groups}")
    if loop is not None and not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
        raise ValueError(f"loop {loop} over {len(layers)} layers")
    return ModelConfig(
        arch="sisisun", n_layers=len(layers), hidden=hidden, vocab=vocab, n_heads=a.heads, n_kv_heads=a.kv_heads,
        head_dim=a.dim, ffn=max([d.ff for d in dense], default=0), rms_eps=rms_eps, rope_dim=0, qk_norm=True,
        attn_scale=a.scale, n_experts=max([m.experts for m in moe], default=0),
        n_experts_used=max([m.top for m in moe], default=0), expert_ffn=max([m.ff for m in moe], default=0),
        shared_ffn=max([m.shared_ff for m in moe], default=0), layer_specs=tuple(layers), loop=loop,
        max_context=max_context)


# Small Sisisun geometry of the tests and the command line: unequal head widths, one layer without a feed-forward, a
# loop that neither starts nor stops with the stack.
_SISISUN_A = AttentionSpec(heads=4, kv_heads=2, dim=48, vdim=64, scale=0.15, softcap=20.0)
TINY_SISISUN = sisisun_config(
    192, 1024, (LayerSpec(_SISISUN_A, DenseMlpSpec(256, "clamped_glu", 1.5)),
                LayerSpec(_SISISUN_A, MoeMlpSpec(12, 3, 72, groups=3, groups_kept=2, scale=1.7, shared_ff=40)),
                LayerSpec(_SISISUN_A, None),
                LayerSpec(_SISISUN_A, DenseMlpSpec(160, "clamped_glu", 1.5))),
    loop=LoopSpec(1, 3, 2), max_context=8192)

# Geometries at the layer sizes of deployed models, for throughput: an 8B-class dense stack and a 30B-A3B-class
# mixture, both with a looped range.
_SISISUN_8B_A = AttentionSpec(heads=32, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0)
_SISISUN_30B_A = AttentionSpec(heads=32, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0)
SISISUN_8B = sisisun_config(4096, 128256, tuple(LayerSpec(_SISISUN_8B_A, DenseMlpSpec(14336, "clamped_glu", 7.0))
                                                for _ in range(32)), loop=LoopSpec(8, 16, 2))
SISISUN_30B_MOE = sisisun_config(2048, 151936, tuple(
    LayerSpec(_SISISUN_30B_A, MoeMlpSpec(128, 8, 768, groups=8, groups_kept=4, scale=2.5, shared_ff=768))
    for _ in range(48)), loop=LoopSpec(12, 24, 2))


def milutar_config(hidden: int, vocab: int, layers: Tuple[LayerSpec, ...], loop: Optional[LoopSpec] = None,
                   rms_eps: float = 1e-6, residual_mult: float = 1.0, max_context: int = 262144) -> ModelConfig:
    """``ModelConfig`` of a Milutar model: parallel layers with token shift and layer scale over latent attention, norms
    with a single gain, optional looped range."""
    if not layers:
        raise ValueError("a model needs layers")
    for i, l in enumerate(layers):
        try:
            l.mixer.check()
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    if loop is not None and not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
        raise ValueError(f"loop {loop} over {len(layers)} layers")
    a = layers[0].mixer
    return ModelConfig(
        arch="milutar", n_layers=len(layers), hidden=hidden, vocab=vocab, n_heads=a.heads, n_kv_heads=1,
        head_dim=a.dim + a.rot_dim, ffn=max([l.mlp.ff for l in layers if l.mlp is not None], default=0), rms_eps=rms_eps,
        rope_theta=a.rot.base, rope_dim=a.rot_dim, attn_scale=a.scale, layer_specs=tuple(layers), loop=loop,
        residual_mult=residual_mult, max_context=max_context)


def _milutar_layer(mixer: LatentAttentionSpec, ff: int) -> LayerSpec:
    return LayerSpec(mixer, DenseMlpSpec(ff, "relu2") if ff else None, parallel=True, token_shift=True)


# Small Milutar geometry of the tests and the command line: both kinds of attention, unequal widths, a layer without a
# feed-forward, a loop inside the stack.
_MILUTAR_W = LatentAttentionSpec(heads=3, dim=40, rot_dim=24, vdim=48, kv_rank=72, scale=0.125, window=50,
                                 rot=RotarySpec(24, 5000.0, YarnSpec(4.0, 512.0, 20.0, 1.5)))
_MILUTAR_F = LatentAttentionSpec(heads=5, dim=24, rot_dim=8, vdim=32, kv_rank=48, scale=0.18, q_rank=56, sink=True,
                                 rot=RotarySpec(8, 100000.0))
TINY_MILUTAR = milutar_config(
    200, 1024, (_milutar_layer(_MILUTAR_W, 232), _milutar_layer(_MILUTAR_F, 184), _milutar_layer(_MILUTAR_W, 0),
                _milutar_layer(_MILUTAR_F, 184)), loop=LoopSpec(1, 3, 2), residual_mult=0.6, max_context=8192)

# Geometry at the layer sizes of a deployed model, for throughput: an 8B-class width with 512-wide latents.
_MILUTAR_8B_W = LatentAttentionSpec(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, window=4096,
                                    rot=RotarySpec(64, 50000.0, YarnSpec(16.0, 8192.0, 24.0, 2.0)))
_MILUTAR_8B_F = LatentAttentionSpec(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, q_rank=1536,
                                    sink=True, rot=RotarySpec(64, 2e6))
MILUTAR_8B = milutar_config(4096, 128256, tuple(_milutar_layer(_MILUTAR_8B_F if i % 4 == 3 else _MILUTAR_8B_W, 20480)
                                                for i in range(28)), loop=LoopSpec(8, 16, 2), residual_mult=0.5)


def banelix_config(hidden: int, vocab: int, layers: Tuple[LayerSpec, ...], rms_eps: float = 1e-6, residual_mult: float = 1.0,
                   embed_scale: float = 1.0, max_context: int = 262144) -> ModelConfig:
    """``ModelConfig`` of a Banelix model: windowed attention layers (some on an earlier layer's keys and values) and layers
    of attention beside a gated linear recurrence, dense SiLU feed-forwards."""
    if not layers:
        raise ValueError("a model needs layers")
    for i, l in enumerate(layers):
        a = l.attention
        try:
            l.mixer.check()
            if a.kv_from is not None:
                if not 0 <= a.kv_from < i:
                    raise ValueError(f"keys and values of layer {a.kv_from}")
                src = layers[a.kv_from].mixer
                if not isinstance(src, AttentionSpec) or src.kv_from is not None:
                    raise ValueError(f"layer {a.kv_from} has no keys and values to share")
                if (src.kv_heads, src.dim, src.vdim) != (a.kv_heads, a.dim, a.vdim):
                    raise ValueError(f"layer {a.kv_from} has other key/value heads")
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    a = layers[0].attention
    return ModelConfig(
        arch="banelix", n_layers=len(layers), hidden=hidden, vocab=vocab, n_heads=a.heads, n_kv_heads=a.kv_heads,
        head_dim=a.dim, ffn=max([l.mlp.ff for l in layers if l.mlp is not None], default=0), rms_eps=rms_eps,
        rope_theta=a.rot.base, rope_dim=a.rot.dims, attn_scale=a.scale, embed_scale=embed_scale, layer_specs=tuple(layers),
        residual_mult=residual_mult, max_context=max_context)


def _banelix_attention(heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, rot: RotarySpec,
                       kv_from: Optional[int] = None) -> AttentionSpec:
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, rot=rot, window=window, sink_score=0.0, qk_norm=QK_NORM_ROWS,
                         bias=True, kv_from=kv_from)


def _banelix_side_by_side(heads: int, kv_heads: int, dim: int, scale: float, rot: RotarySpec, right: RecurrentSpec,
                          left_scale: float, right_scale: float) -> SideBySideSpec:
    left = AttentionSpec(heads, kv_heads, dim, dim, scale, rot=rot, qk_norm=QK_NORM_UNIT, bias=True, keys_as_values=True,
                         head_gate=True)
    return SideBySideSpec(left, right, left_scale, right_scale)


# Small Banelix geometry of the tests and the command line: unequal widths, a layer without a feed-forward, a layer on the
# keys and values of an earlier one with a window of its own.
_BANELIX_ROT = RotarySpec(40, 8000.0, YarnSpec(4.0, 512.0, 20.0, 1.5), halves=True)
_BANELIX_P = _banelix_side_by_side(6, 2, 40, 0.15, RotarySpec(24, 90000.0, BandSpec(6.0, 1.0, 3.0, 400.0), halves=True),
                                   RecurrentSpec(120, 3, 4), 0.9, 0.7)
TINY_BANELIX = banelix_config(
    216, 1024, (LayerSpec(_banelix_attention(4, 2, 48, 56, 0.14, 50, _BANELIX_ROT), DenseMlpSpec(232)),
                LayerSpec(_BANELIX_P, DenseMlpSpec(184)), LayerSpec(_BANELIX_P, None),
                LayerSpec(_banelix_attention(4, 2, 48, 56, 0.12, 33, _BANELIX_ROT, kv_from=0), DenseMlpSpec(184))),
    residual_mult=0.8, embed_scale=6.0, max_context=8192)

# Geometry at the layer sizes of a deployed model, for throughput: an 8B-class width, one windowed layer in four.
_BANELIX_8B_ROT = RotarySpec(128, 50000.0, YarnSpec(16.0, 8192.0, 32.0, 1.0), halves=True)
_BANELIX_8B_P = _banelix_side_by_side(32, 8, 128, 128 ** -0.5, RotarySpec(64, 500000.0, BandSpec(8.0, 1.0, 4.0, 8192.0), halves=True),
                                      RecurrentSpec(4096, 16, 4), 1.0, 1.0)
BANELIX_8B = banelix_config(4096, 128256, tuple(
    LayerSpec(_banelix_attention(32, 8, 128, 128, 128 ** -0.5, 4096, _BANELIX_8B_ROT, kv_from=i - 4 if i % 8 == 7 else None)
              if i % 4 == 3 else _BANELIX_8B_P, DenseMlpSpec(14336)) for i in range(24)), residual_mult=0.5, embed_scale=64.0)


def mepatar_config(hidden: int, vocab: int, layers: Tuple[LayerSpec, ...], rms_eps: float = 1e-6, norm_groups: int = 1,
                   embed_scale: float = 1.0, max_context: int = 262144) -> ModelConfig:
    """``ModelConfig`` of a Mepatar model: parallel layers of two norms over groups of channels with an input convolution;
    mixers are attention over a window and the first tokens, retention, or the gated delta rule."""
    if not layers:
        raise ValueError("a model needs layers")
    if norm_groups < 1 or hidden % norm_groups:
        raise ValueError(f"norm over {norm_groups} groups of {hidden} channels")
    for i, l in enumerate(layers):
        try:
            l.mixer.check()
            if not 1 <= l.input_taps <= CONV_MAX_TAPS:
                raise ValueError(f"input convolution of {l.input_taps} taps")
            if hidden // norm_groups * max(1, 2 * (l.input_taps - 1)) > NORM_CONV_MAX_ROWS:
                raise ValueError(f"norms over {hidden // norm_groups} channels with an input convolution of {l.input_taps} taps")
            if isinstance(l.mlp, MoeMlpSpec):
                l.mlp.check()
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    att = next((l.attention for l in layers if l.attention is not None), None)
    m, rot = att or layers[0].mixer, next((l.mixer.rot for l in layers if l.mixer.rot is not None), None)
    moe = [l.mlp for l in layers if isinstance(l.mlp, MoeMlpSpec)]
    return ModelConfig(
        arch="mepatar", n_layers=len(layers), hidden=hidden, vocab=vocab, n_heads=m.heads, n_kv_heads=m.kv_heads,
        head_dim=m.dim, ffn=max([l.mlp.ff for l in layers if isinstance(l.mlp, DenseMlpSpec)], default=0), rms_eps=rms_eps,
        rope_theta=rot.base if rot else 0.0, rope_dim=rot.dims if rot else 0, attn_scale=att.scale if att else None,
        n_experts=max([e.experts for e in moe], default=0), n_experts_used=max([e.top for e in moe], default=0),
        expert_ffn=max([e.ff for e in moe], default=0), embed_scale=embed_scale, layer_specs=tuple(layers),
        norm_groups=norm_groups, max_context=max_context)


def mepatar_attention(heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, keep_first: int,
                      rot: RotarySpec) -> AttentionSpec:
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, rot=rot, window=window, keep_first=keep_first, bias=True,
                         head_scale=True, out_bias=True)


def mepatar_layer(mixer: Union[AttentionSpec, LinearAttentionSpec], mlp: Optional[Union[DenseMlpSpec, MoeMlpSpec]],
                  taps: int) -> LayerSpec:
    return LayerSpec(mixer, mlp, parallel=True, input_taps=taps)


def mepatar_experts(experts: int, top: int, ff: int, limit: float) -> MoeMlpSpec:
    return MoeMlpSpec(experts, top, ff, score="softmax", act="clamped_glu", limit=limit)


# Small Mepatar geometry of the tests and the command line: every kind of layer, unequal widths, a layer without a
# feed-forward.
TINY_MEPATAR = mepatar_config(
    208, 1024, (mepatar_layer(LinearAttentionSpec(4, 2, 40, 48, taps=4), DenseMlpSpec(232, "gelu_tanh"), 3),
                mepatar_layer(mepatar_attention(6, 2, 48, 56, 0.14, 50, 6, RotarySpec(32, 20000.0)), mepatar_experts(12, 3, 72, 2.0), 3),
                mepatar_layer(LinearAttentionSpec(3, 3, 56, 40, (0.97, 0.99, 0.998), RotarySpec(24, 5000.0, halves=True)),
                              mepatar_experts(12, 3, 72, 2.0), 3),
                mepatar_layer(LinearAttentionSpec(4, 2, 40, 48, taps=4), None, 3)),
    rms_eps=1e-5, norm_groups=4, embed_scale=8.0, max_context=8192)

# Geometry at the layer sizes of a deployed model, for throughput: an 8B-class width, a period of three delta, three retention
# and two attention layers.
_MEPATAR_8B_D = LinearAttentionSpec(32, 16, 128, 128, taps=4)
_MEPATAR_8B_R = LinearAttentionSpec(32, 32, 128, 128, tuple(1.0 - 2.0 ** (-5 - 5 * h / 31) for h in range(32)),
                                    RotarySpec(128, 1e6, halves=True))
_MEPATAR_8B_A = mepatar_attention(32, 8, 128, 128, 128 ** -0.5, 4096, 128, RotarySpec(64, 50000.0))
_MEPATAR_8B_PERIOD = (_MEPATAR_8B_D, _MEPATAR_8B_R, _MEPATAR_8B_D, _MEPATAR_8B_A, _MEPATAR_8B_D, _MEPATAR_8B_R, _MEPATAR_8B_R,
                      _MEPATAR_8B_A)
MEPATAR_8B = mepatar_config(4096, 128256, tuple(mepatar_layer(m, DenseMlpSpec(14336, "gelu_tanh"), 4)
                                                for m in _MEPATAR_8B_PERIOD * 3), norm_groups=8, embed_scale=64.0)
# ... and a 30B-A3B-class mixture
MEPATAR_30B_MOE = mepatar_config(2048, 151936, tuple(
    mepatar_layer(m, mepatar_experts(128, 8, 768, 7.0), 4) for m in (
        LinearAttentionSpec(32, 16, 128, 128, taps=4), _MEPATAR_8B_R, LinearAttentionSpec(32, 16, 128, 128, taps=4),
        mepatar_attention(32, 4, 128, 128, 128 ** -0.5, 4096, 128, RotarySpec(64, 50000.0))) * 12), norm_groups=4, embed_scale=45.0)


@dataclass(frozen=True)
class AssistantConfig:
    """Gemma 4 assistant (MTP) head: a separate four-block draft model with no K/V projections of its own.  Every
    block attends against the backbone's KV of one of its last two layers (a sliding block reads layer ``n - 2``, a
    full-attention block layer ``n - 1``), so head count, KV heads, head width, window and RoPE of a block are those
    of the backbone layer it reads.  Contract: the reference's ``docs/reference/GEMMA4-ASSISTANT-MTP.md:36-60``
    (hyperparameters) and ``:62-80`` (tensor layout)."""
    arch: str = "gemma4-assistant"
    n_blocks: int = 4
    hidden: int = 1024                   # the head's own width
    backbone_hidden: int = 2816          # the target's width (``embedding_length_out``)
    ffn: int = 8192
    n_heads: int = 16
    vocab: int = 262144
    swa_blocks: Tuple[bool, ...] = (True, True, True, False)
    rms_eps: float = 1e-6

    def backbone_layer(self, il: int, backbone: ModelConfig) -> int:
        return backbone.n_layers - 2 if self.swa_blocks[il] else backbone.n_layers - 1

    def check_pairing(self, backbone: ModelConfig) -> None:
        """The head is only meaningful against the backbone it was trained with: refuse a mismatch before loading."""
        errs = []
        if backbone.arch != "gemma4":
            errs.append(f"backbone arch {backbone.arch!r} is not gemma4")
        if self.backbone_hidden != backbone.hidden:
            errs.append(f"embedding_length_out {self.backbone_hidden} != backbone width {backbone.hidden}")
        if self.n_heads != backbone.n_heads:
            errs.append(f"head count {self.n_heads} != backbone's {backbone.n_heads}")
        if self.vocab != backbone.vocab:
            errs.append(f"vocabulary {self.vocab} != backbone's {backbone.vocab}")
        if len(self.swa_blocks) != self.n_blocks:
            errs.append("sliding-window pattern length != block count")
        if backbone.n_layers >= 2 and backbone.arch == "gemma4":
            if backbone.is_global_layer(backbone.n_layers - 2) or not backbone.is_global_layer(backbone.n_layers - 1):
                errs.append("backbone's last two layers are not (sliding, global)")
        if (2 * self.backbone_hidden) % 256 or self.hidden % 256 or self.ffn % 256:
            errs.append("widths must be multiples of the 256-element block")
        if errs:
            raise ValueError("assistant head does not pair with this backbone: " + "; ".join(errs))


GEMMA4_26B_ASSISTANT = AssistantConfig()
TINY_GEMMA4_ASSISTANT = AssistantConfig(hidden=256, backbone_hidden=256, ffn=512, n_heads=4, vocab=2048)

NAMED_ASSISTANTS: Dict[str, AssistantConfig] = {
    "gemma4-26b-a4b": GEMMA4_26B_ASSISTANT,
    "tiny-gemma4": TINY_GEMMA4_ASSISTANT,
}

NAMED_CONFIGS: Dict[str, ModelConfig] = {
    "tiny-dense": TINY_DENSE,
    "tiny-hybrid": TINY_HYBRID,
    "tiny-hybrid-moe": TINY_HYBRID_MOE,
    "tiny-hybrid-tp": TINY_HYBRID_TP,
    "small-hybrid-tp8": SMALL_HYBRID_TP8,
    "tiny-hybrid-moe-tp": TINY_HYBRID_MOE_TP,
    "tiny-gemma4": TINY_GEMMA4,
    "qwen35-27b": QWEN35_27B,
    # the same geometries with the checkpoint's trailing NextN (MTP) block, for speculative serving runs
    "qwen35-27b-mtp": replace(QWEN35_27B, nextn_layers=1),
    "tiny-hybrid-mtp": replace(TINY_HYBRID, nextn_layers=1),
    "qwen35-35b-a3b": QWEN35_35B_A3B,
    "gemma4-26b-a4b": GEMMA4_26B_A4B,
    "tiny-sisisun": TINY_SISISUN,
    "sisisun-8b": SISISUN_8B,
    "sisisun-30b-moe": SISISUN_30B_MOE,
    "tiny-milutar": TINY_MILUTAR,
    "milutar-8b": MILUTAR_8B,
    "tiny-banelix": TINY_BANELIX,
    "banelix-8b": BANELIX_8B,
    "tiny-mepatar": TINY_MEPATAR,
    "mepatar-8b": MEPATAR_8B,
    "mepatar-30b-moe": MEPATAR_30B_MOE,
}
