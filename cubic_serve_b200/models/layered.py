"""Layered decoders: every layer names its own token mixer, the residual stream is fp32.

``config.json`` of such a checkpoint has ``architecture``, ``vocab``, ``width``, ``norm.eps`` and the list ``layers``.  What
the layers of an architecture have in common is its entry in ``DESIGNS``:

* ``Bumodra``: parallel layers (mixer and feed-forward read the same norm and are added to the residual together); ``loop`` =
  {start, stop, times} runs the layers ``start .. stop - 1`` ``times`` times with the same weights, each pass with its own
  cache and state; a pass starts with a projection of [residual ; embedding output];
* ``Loduzen``: sequential layers (mixer, then feed-forward, each behind a norm of its own), tied output head; ``token_side`` =
  {dim} adds, after the feed-forward, what the layer takes from its part of a second embedding of the token;
* ``Vimelorn``: sequential sublayers on ``streams`` residual streams (hyper-connections: every sublayer reads a weighted sum of
  them, its result is added to all of them while they are mixed), scaled embedding; feed-forwards are dense or routed: experts
  chosen by score plus correction, some of which return the token itself, and a gated shared expert;
* ``Fovunex``: sequential layers whose results pass a gate per channel that reads the same normed input, norms with one number,
  scaled embedding, clamped gated feed-forward; a loop, before whose later passes the embedding output is added again.

Mixers (another one is a spec, a reader in ``_MIXER_READERS``, an inventory entry, a ``_pack_*`` function and a method of
``models/layered_runner.py``):

* ``delta`` / ``channel_delta``: short convolution, gated delta rule with one decay per head / per (head, key channel);
* ``latent_attention``: attention over cached latents, with a sliding window, low-rank queries and a gate per head (``Bumodra``), or
  with a rotated key part that all heads share (``Fovunex``);
* ``mamba2``: short convolution, scalar-decay linear recurrence (state-space duality), gated norm in equal parts;
* ``parallel``: two mixers that read the same norm, each scaled: sliding-window grouped-query attention with head norms,
  rotary pairs, a softmax sink and values that are the raw keys; and gated linear attention with a decay per key channel;
* ``attention``: short convolutions of q, k and v, rotary halves, unit root mean squares, a window beside kept first tokens
  (``Vimelorn``); or the difference of two attention maps over the same values inside chunks of positions, heads normed and gated
  (``Fovunex``);
* ``attention_2``: q and k normed over their whole projections, queries warmer with their position, a bias per distance and head;
* ``mingru``: an element-wise recurrence whose gate and candidate read the current token only.

ONE matrix holds all projections that read a layer's norm and ONE the output projections side by side, whatever the mixer is:
with parallel layers the first also has the feed-forward's up rows and the second its down columns ([o | down]); with gated
residuals the matrices that read a norm end with the rows of the gate.  Rows and columns are padded with zeros to what the GEMM
asks for.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, replace
from pathlib import Path

import torch

from ..ops import wq_pack
from ..ops.eager import rope_inv_freq
from .config import QuantSpec

MAX_CONV_TAPS, MAX_DELTA_DIM, MAX_LATENT, MAX_HEAD = 16, 256, 1024, 256      # limits of the kernels
MAX_STREAMS, MAX_ROUTER, MAX_TOP = 8, 256, 32
LATENT_WIDTHS = ((64, 64), (128, 128), (192, 128), (256, 256), (320, 256), (512, 512), (576, 512))   # of latent_attn.cu


@dataclass(frozen=True)
class Design:
    """What the layers of an architecture have in common."""
    mixers: dict[str, str]       # type in ``config.json`` -> entry of ``_MIXER_READERS``
    sequential: bool             # mixer and feed-forward one after the other, each with a norm; else in parallel behind one
    norm_offset: float           # a norm's factor is this plus its stored weight
    embed_norm: bool             # the embedding is normed before the first layer
    tied_head: bool              # the output head is the embedding table
    ff: str                      # "squared_relu" (up, down) or gated (gate, up, down): "gelu_glu", "silu_glu", "clamped_glu"
    streams: bool = False        # several residual streams, routed feed-forwards
    embed_scale: bool = False    # the embedding is scaled
    scalar_norm: bool = False    # a norm of the residual has one number for all channels
    gated: bool = False          # a sublayer's result passes a sigmoid gate per channel that reads the sublayer's input
    loop: str = ""               # a loop of layers: passes start with a projection of [residual ; embedding output] ("project"),
                                 # or later passes with their sum ("add"); "": none


DESIGNS = {
    "Bumodra": Design({"delta": "delta", "channel_delta": "channel_delta", "latent_attention": "latent"}, False, 1.0, True, False,
                      "squared_relu", loop="project"),
    "Loduzen": Design({"parallel": "parallel", "mamba2": "mamba2"}, True, 0.0, False, True, "gelu_glu"),
    "Vimelorn": Design({"attention": "conv_attention", "attention_2": "biased_attention"}, True, 0.0, False, False, "silu_glu",
                       streams=True, embed_scale=True),
    "Fovunex": Design({"latent_attention": "rotated_latent", "attention": "differential", "mingru": "mingru"}, True, 0.0, False, False,
                      "clamped_glu", embed_scale=True, scalar_norm=True, gated=True, loop="add"),
}
ARCHITECTURES = tuple(DESIGNS)


class LayeredConfigError(ValueError):
    pass


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


# ------------------------------------------------------------------ configuration
class MixerSpec:
    """A layer's token mixer: sizes and constants.  ``parts``: the mixers it consists of (itself, unless it is a pair)."""

    @property
    def parts(self) -> tuple["MixerSpec", ...]:
        return (self,)

    def page_bytes(self, act_bytes: int) -> int:
        """One 16-token page of its cache."""
        return 0

    def state_bytes(self, act_bytes: int) -> int:
        """Recurrent state of a request."""
        return 0


@dataclass(frozen=True)
class DeltaSpec(MixerSpec):
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    per_channel: bool = False
    decay_rank: int = 0          # per_channel: inner sizes of the low-rank decay and output-gate projections
    gate_rank: int = 0

    @property
    def channels(self) -> int:
        """Convolved channels: q | k of the key heads, v of the value heads."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def conv_width(self) -> int:
        return round_up(self.channels, 8)

    @property
    def state_stride(self) -> int:
        return round_up(self.dim, 4)

    @property
    def label(self) -> str:
        return "channel_delta" if self.per_channel else "delta"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def state_bytes(self, act_bytes: int) -> int:
        return self.heads * self.vdim * self.state_stride * 4 + round_up((self.conv - 1) * self.conv_width * act_bytes, 16)

    def validate(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.conv) <= 0 or self.heads % self.kv_heads:
            raise LayeredConfigError("delta heads are grouped evenly over positive key head counts and sizes")
        if self.conv > MAX_CONV_TAPS or self.dim > MAX_DELTA_DIM:
            raise LayeredConfigError(f"delta layers take up to {MAX_CONV_TAPS} convolution taps and key width {MAX_DELTA_DIM}")


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` channels.  ``scaling``: as ``ModelConfig.rope_scaling``; the attention factor of
    ``yarn`` multiplies cosine and sine here."""
    dims: int
    base: float
    scaling: tuple | None = None

    def validate(self, width: int) -> None:
        if self.dims % 2 or not 0 <= self.dims <= width or self.base <= 0:
            raise LayeredConfigError("rotary channels come in pairs inside a head")

    def _exact(self) -> torch.Tensor:
        return rope_inv_freq(self.dims, self.base, scaling=self.scaling, dtype=torch.float64)

    @property
    def factor(self) -> float:
        """On cosine and sine."""
        return float(self.scaling[5]) if self.scaling and self.scaling[0] == "yarn" else 1.0

    def table(self) -> tuple[torch.Tensor, float]:
        """(fp32 radians per position of every pair, factor on cosine and sine)."""
        return self._exact().float(), self.factor

    def split_table(self) -> torch.Tensor:
        """fp32 ``[2, pairs]``: radians per position, and what rounding took from them."""
        exact = self._exact()
        return torch.stack([exact.float(), (exact - exact.float().double()).float()])


@dataclass(frozen=True)
class LatentSpec(MixerSpec):
    heads: int
    dim: int
    vdim: int
    q_rank: int                  # inner size of the low-rank query projection; 0: one full matrix
    kv_rank: int
    scale: float
    window: int = 0              # 0: every earlier token
    rot_dim: int = 0             # rotated channels of a query head, beside ``dim``; the rotated key is shared by all heads
    rotary: RotarySpec | None = None
    gated: bool = True           # a sigmoid gate per head
    label = "latent"

    def page_bytes(self, act_bytes: int) -> int:
        return 16 * self.row_padded * act_bytes

    @property
    def rot_col(self) -> int:
        """Column of the rotated part in a cached row, behind the latent."""
        return round_up(self.kv_rank, 8) if self.rot_dim else self.kv_rank

    @property
    def _padded(self) -> tuple[int, int]:
        """Columns of (a cached row, its latent part read as values): pairs the attention kernels are built for."""
        for row, rank in LATENT_WIDTHS:
            if self.rot_col + self.rot_dim <= row and self.kv_rank <= rank:
                return row, rank
        return MAX_LATENT, MAX_LATENT

    @property
    def row_padded(self) -> int:
        return self._padded[0]

    @property
    def rank_padded(self) -> int:
        return self._padded[1]

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def validate(self) -> None:
        if min(self.heads, self.dim, self.vdim, self.kv_rank) <= 0 or min(self.q_rank, self.window, self.rot_dim) < 0:
            raise LayeredConfigError("latent attention sizes are positive")
        if self.rot_col + self.rot_dim > MAX_LATENT or self.rot_dim > MAX_HEAD:
            raise LayeredConfigError(f"latents of up to {MAX_LATENT} channels with their rotated part are served")
        if bool(self.rot_dim) != (self.rotary is not None):
            raise LayeredConfigError("rotated channels and their frequencies come together")
        if self.rotary is not None:
            self.rotary.validate(self.rot_dim)
            if self.rotary.dims != self.rot_dim:
                raise LayeredConfigError("the rotated part of latent attention is rotated as a whole")


@dataclass(frozen=True)
class AttentionSpec(MixerSpec):
    """Grouped-query attention with head norms and rotary pairs; a value is the raw key of its token."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rotary: RotarySpec
    window: int = 0              # 0: every earlier token
    sink: float | None = 0.0     # score of a softmax entry without a value (None: none)
    label = "attention"

    @property
    def width_padded(self) -> int:
        """Columns of a cached key or value: the widths the attention kernels are built for."""
        return round_up(self.dim, 64)

    @property
    def out_width(self) -> int:
        return self.heads * self.dim

    def page_bytes(self, act_bytes: int) -> int:
        return 16 * self.kv_heads * 2 * self.width_padded * act_bytes

    def validate(self) -> None:
        if min(self.heads, self.kv_heads, self.dim) <= 0 or self.heads % self.kv_heads or self.window < 0:
            raise LayeredConfigError("attention heads are grouped evenly over positive key head counts and sizes")
        if self.dim > MAX_HEAD:
            raise LayeredConfigError(f"attention heads of up to {MAX_HEAD} channels are served")
        self.rotary.validate(self.dim)


@dataclass(frozen=True)
class GatedLinearSpec(MixerSpec):
    """Gated linear attention: decay per key channel, a state of [key channel, value channel] per head."""
    heads: int
    dim: int
    vdim: int
    tau: float                   # the decay is a sigmoid to the power 1 / tau
    decay_rank: int = 0          # inner size of the low-rank decay projection
    label = "gated_linear"

    @property
    def state_stride(self) -> int:
        return round_up(self.dim, 4)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def state_bytes(self, act_bytes: int) -> int:
        return self.heads * self.vdim * self.state_stride * 4

    def validate(self) -> None:
        if min(self.heads, self.dim, self.vdim) <= 0 or self.tau <= 0:
            raise LayeredConfigError("gated linear attention sizes and tau are positive")
        if self.dim > MAX_DELTA_DIM:
            raise LayeredConfigError(f"gated linear attention takes key widths of up to {MAX_DELTA_DIM}")


@dataclass(frozen=True)
class SsdSpec(MixerSpec):
    """State-space duality layer (Mamba-2): ``heads`` of ``vdim`` channels, B and C of ``state`` channels per group."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int
    label = "mamba2"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Convolved channels: x of the heads, B and C of the groups."""
        return self.out_width + 2 * self.groups * self.state

    @property
    def conv_width(self) -> int:
        return round_up(self.channels, 8)

    @property
    def state_stride(self) -> int:
        return round_up(self.state, 4)

    def state_bytes(self, act_bytes: int) -> int:
        return self.heads * self.vdim * self.state_stride * 4 + round_up((self.conv - 1) * self.conv_width * act_bytes, 16)

    def validate(self) -> None:
        if min(self.heads, self.vdim, self.state, self.groups, self.conv, self.norm_groups) <= 0 or self.heads % self.groups \
                or self.out_width % self.norm_groups:
            raise LayeredConfigError("mamba2 heads are grouped evenly and the normed width is cut evenly")
        if self.conv > MAX_CONV_TAPS or self.state > MAX_DELTA_DIM:
            raise LayeredConfigError(f"mamba2 layers take up to {MAX_CONV_TAPS} convolution taps and state width {MAX_DELTA_DIM}")


@dataclass(frozen=True)
class PairSpec(MixerSpec):
    """Two mixers side by side on the same input: ``left_scale * left + right_scale * right``."""
    left: MixerSpec
    right: MixerSpec
    left_scale: float
    right_scale: float

    @property
    def label(self) -> str:
        return f"{self.left.label}+{self.right.label}"

    @property
    def parts(self) -> tuple[MixerSpec, ...]:
        return (self.left, self.right)

    @property
    def right_off(self) -> int:
        """Column of the right outputs in the operand of the joint output product."""
        return round_up(self.left.out_width, 8)

    @property
    def out_width(self) -> int:
        return self.right_off + self.right.out_width

    def page_bytes(self, act_bytes: int) -> int:
        return sum(p.page_bytes(act_bytes) for p in self.parts)

    def state_bytes(self, act_bytes: int) -> int:
        return sum(p.state_bytes(act_bytes) for p in self.parts)

    def validate(self) -> None:
        for p in self.parts:
            p.validate()


class _QkvSpec(MixerSpec):
    """Grouped-query attention with keys and values of their own (columns [q | k | v] of the projection)."""

    @property
    def width_padded(self) -> int:
        """Columns of a cached key or value: the widths the attention kernels are built for."""
        return round_up(max(self.dim, self.vdim), 64)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def offsets(self) -> tuple[int, int, int]:
        """First columns of q, k and v from the first of them on."""
        k = round_up(self.heads * self.dim, 8)
        return 0, k, k + round_up(self.kv_heads * self.dim, 8)

    def page_bytes(self, act_bytes: int) -> int:
        return 16 * self.kv_heads * 2 * self.width_padded * act_bytes

    def validate(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) <= 0 or self.heads % self.kv_heads:
            raise LayeredConfigError("attention heads are grouped evenly over positive key head counts and sizes")
        if max(self.dim, self.vdim) > MAX_HEAD:
            raise LayeredConfigError(f"attention heads of up to {MAX_HEAD} channels are served")


@dataclass(frozen=True)
class ConvAttentionSpec(_QkvSpec):
    """Short convolutions of q, k and v, rotary halves, heads over their root mean square, a window beside kept first tokens."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    rotary: "RotarySpec"
    window: int = 0              # 0: every earlier token
    keep: int = 0                # first tokens that stay visible behind the window
    label = "conv_attention"

    @property
    def conv_width(self) -> int:
        """Convolved columns of the projection."""
        return round_up(self.offsets[2] + self.kv_heads * self.vdim, 8)

    def state_bytes(self, act_bytes: int) -> int:
        return round_up((self.conv - 1) * self.conv_width * act_bytes, 16)

    def validate(self) -> None:
        super().validate()
        if not 1 <= self.conv <= MAX_CONV_TAPS:
            raise LayeredConfigError(f"attention takes 1 to {MAX_CONV_TAPS} convolution taps")
        self.rotary.validate(self.dim)
        if self.window < 0 or self.keep < 0:
            raise LayeredConfigError("an attention window and the tokens kept before it are not negative")


@dataclass(frozen=True)
class BiasedAttentionSpec(_QkvSpec):
    """q and k normed over their whole projections, queries times ``1 + coef ln(floor((position + 1) / every) + 1)``, a learned
    bias by bucket of distance and head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    buckets: int                 # rows of the bias table
    bias_max: int                # distance at which the last bucket's steps end
    temp_coef: float = 0.0
    temp_every: int = 0          # 0: no factor
    window = 0
    label = "biased_attention"

    def bucket(self, n: int) -> int:
        """Row of distance n: a row each for the first half, equal steps of the logarithm up to ``bias_max`` for the rest.  In
        integers, so that no rounding moves a border."""
        B = self.buckets
        half = B // 2
        if n < half:
            return n
        k = 0
        while k < B - half and n ** (B - half) * half ** (k + 1) >= self.bias_max ** (k + 1) * half ** (B - half):
            k += 1
        return min(B - 1, half + k)

    def bucket_of_distance(self) -> torch.Tensor:
        """Rows of the distances 0 .. ``bias_max``; farther ones share the last."""
        return torch.tensor([self.bucket(n) for n in range(self.bias_max + 1)])

    def validate(self) -> None:
        super().validate()
        if self.buckets < 2 or self.bias_max <= self.buckets // 2:
            raise LayeredConfigError("distance biases have two rows or more and a largest distance behind their first half")
        if self.temp_every < 0:
            raise LayeredConfigError("the query factor grows every positive number of positions")


@dataclass(frozen=True)
class DifferentialSpec(_QkvSpec):
    """Two attention maps per head over the same values: the second's output times a learned factor is taken from the first's, the
    difference normed per head and gated per channel.  Head norms and rotary halves on every map; ``chunk``: a token sees its own
    chunk of positions only."""
    heads: int
    kv_heads: int
    dim: int                     # of a map
    vdim: int
    scale: float
    rotary: RotarySpec
    diff: float                  # constant part of the factor
    chunk: int = 0               # 0: every earlier token
    label = "differential"

    @property
    def width_padded(self) -> int:
        """Columns of a cached key (both maps, half of them each) or value: the widths the kernels are built for."""
        return next((p for p in (64, 128) if max(2 * self.dim, self.vdim) <= p), 256)

    @property
    def offsets(self) -> tuple[int, int, int]:
        k = round_up(self.heads * 2 * self.dim, 8)
        return 0, k, k + round_up(self.kv_heads * 2 * self.dim, 8)

    def validate(self) -> None:
        super().validate()
        if 2 * self.dim > MAX_HEAD:
            raise LayeredConfigError(f"maps of up to {MAX_HEAD // 2} channels are served")
        self.rotary.validate(self.dim)
        if self.chunk < 0:
            raise LayeredConfigError("a chunk holds a positive number of positions")


@dataclass(frozen=True)
class MinGruSpec(MixerSpec):
    """Element-wise recurrence of ``width`` channels: ``S <- (1 - z) S + z candidate``, gate and candidate from the current token."""
    width: int
    label = "mingru"

    @property
    def out_width(self) -> int:
        return self.width

    @property
    def padded(self) -> int:
        """Channels of the state: whole 16-byte rows."""
        return round_up(self.width, 4)

    def state_bytes(self, act_bytes: int) -> int:
        return self.padded * 4

    def validate(self) -> None:
        if self.width <= 0:
            raise LayeredConfigError("a recurrence has a positive width")


ATTENTION_SPECS = (LatentSpec, AttentionSpec, ConvAttentionSpec, BiasedAttentionSpec, DifferentialSpec)


@dataclass(frozen=True)
class RoutedSpec:
    """Squared-relu experts of which a token uses ``top``, ``identity`` more that return the token itself, and a gated shared
    expert.  Scores are a softmax over all; the choice adds a correction, the weights do not and sum to one."""
    experts: int
    top: int
    ff: int
    identity: int = 0
    shared_ff: int = 0           # 0: no shared expert

    @property
    def outputs(self) -> int:
        """Outputs of the router."""
        return self.experts + self.identity

    def validate(self) -> None:
        if min(self.experts, self.top, self.ff) <= 0 or min(self.identity, self.shared_ff) < 0 or self.top > self.outputs:
            raise LayeredConfigError("experts, their widths and routes of a token are positive, with no more routes than outputs")
        if self.outputs > MAX_ROUTER or self.top > MAX_TOP:
            raise LayeredConfigError(f"routers of up to {MAX_ROUTER} outputs and {MAX_TOP} routes are served")


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    ff: int = 0                  # feed-forward width; 0 = none
    routed: RoutedSpec | None = None     # instead of a dense feed-forward
    limit: float = 0.0           # of a clamped feed-forward

    @property
    def has_ff(self) -> bool:
        return self.ff > 0 or self.routed is not None


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    rms_eps: float
    loop: tuple[int, int, int] | None = None      # (start, stop, times)
    dtype: str = "bfloat16"                       # activations and products: bfloat16 | float32
    architecture: str = ARCHITECTURES[0]
    side_dim: int = 0                             # width of a layer's part of the token's side embedding; 0 = none
    streams: int = 1                              # residual streams
    embed_scale: float = 1.0
    family: str = "layered"
    max_position: int = 1 << 20                   # positions are rotary or none: only memory limits the context
    quant: QuantSpec = field(default_factory=lambda: QuantSpec("none", 16, 0))
    eos_token_id: int | None = None

    is_moe = False
    qkv_bias = False
    mrope_section = None
    mtp_layers = 0

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def is_hybrid(self) -> bool:
        """Some layer keeps recurrent state per request."""
        return any(l.mixer.state_bytes(4) for l in self.layers)

    @property
    def act_bytes(self) -> int:
        return 4 if self.dtype == "float32" else 2

    @property
    def runs(self) -> tuple[tuple[int, bool], ...]:
        """Layer runs in order: (layer, whether a loop pass starts right before it)."""
        n = self.num_layers
        if self.loop is None:
            return tuple((i, False) for i in range(n))
        a, b, times = self.loop
        return (tuple((i, False) for i in range(a)) + tuple((i, i == a) for _ in range(times) for i in range(a, b))
                + tuple((i, False) for i in range(b, n)))

    def reenters(self, run: int) -> bool:
        """Whether a later pass of the loop, one that adds the embedding output, starts right before this layer run."""
        return self.design.loop == "add" and self.runs[run][1] and run > self.loop[0]

    @property
    def page_bytes(self) -> int:
        """One 16-token page of every attention run."""
        return sum(self.layers[i].mixer.page_bytes(self.act_bytes) for i, _ in self.runs)

    @property
    def state_bytes_per_request(self) -> int:
        return sum(self.layers[i].mixer.state_bytes(self.act_bytes) for i, _ in self.runs)

    @property
    def state_runs(self) -> int:
        """Mixers of the layer runs that keep state per request."""
        return sum(p.state_bytes(self.act_bytes) > 0 for i, _ in self.runs for p in self.layers[i].mixer.parts)

    def run_parts(self, kind: type | tuple[type, ...]) -> int:
        """How many mixers of a kind the layer runs have (each with a cache or state of its own)."""
        return sum(isinstance(p, kind) for i, _ in self.runs for p in self.layers[i].mixer.parts)

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers)) <= 0 or self.rms_eps < 0:
            raise LayeredConfigError("vocab, width and the layer list are positive")
        if self.dtype not in ("bfloat16", "float32"):
            raise LayeredConfigError(f"dtype {self.dtype!r} is not bfloat16 or float32")
        for l in self.layers:
            l.mixer.validate()
            if l.ff < 0 or l.ff and l.routed:
                raise LayeredConfigError("feed-forward widths are positive")
            if l.ff and self.design.ff == "clamped_glu" and l.limit <= 0:
                raise LayeredConfigError("a clamped feed-forward has a positive limit")
            if l.routed is not None:
                if not self.design.streams:
                    raise LayeredConfigError(f"{self.architecture} layers have dense feed-forwards")
                l.routed.validate()
        if not 1 <= self.streams <= MAX_STREAMS or self.streams > 1 and not self.design.streams:
            raise LayeredConfigError(f"1 to {MAX_STREAMS} residual streams are served, more than one in designs that mix them")
        if self.side_dim < 0 or (self.side_dim or not self.design.loop) and self.loop is not None:
            raise LayeredConfigError("layers of this design are run once, and the side input of a layer has a positive width")
        if self.loop is not None:
            a, b, times = self.loop
            if not 0 <= a < b <= self.num_layers or times < 1:
                raise LayeredConfigError("loop needs 0 <= start < stop <= layers and times >= 1")

    def to_config(self) -> dict:
        """The ``config.json`` object of this configuration."""
        layers = [{**dict(zip(("type", "mixer"), _mixer_config(l.mixer))), "mlp": _ff_config(l)} for l in self.layers]
        loop = None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop))
        out = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
               "norm": {"eps": self.rms_eps}, "layers": layers}
        if self.design.embed_scale:
            out["embedding"] = {"scale": self.embed_scale}
        if self.design.streams:
            out["streams"] = self.streams
        elif self.design.loop:
            out["loop"] = loop
        else:
            out["token_side"] = {"dim": self.side_dim} if self.side_dim else None
        return out


def _rotary_config(r: RotarySpec) -> dict:
    scaling = {"scaling": dict(zip(("factor", "original", "fast", "slow"), r.scaling[1:5]))} if r.scaling else {}
    return {"dims": r.dims, "base": r.base, **scaling}


def _mask_config(window: int) -> dict | None:
    return {"size": window} if window else None


def _ff_config(l: LayerSpec) -> dict | None:
    """Feed-forward object of a layer's entry in ``config.json``."""
    if l.routed is None:
        limit = {"limit": l.limit} if l.limit else {}
        return {"kind": "dense", "ff": l.ff, **limit} if l.ff else None
    r = l.routed
    return {"kind": "moe", "expert": {"ff": r.ff}, "router": {"experts": r.experts, "identity": r.identity, "top": r.top},
            "shared": {"ff": r.shared_ff} if r.shared_ff else None}


def _mixer_config(m: MixerSpec) -> tuple[str, dict]:
    """(type, mixer object) of a layer's entry in ``config.json``."""
    if isinstance(m, DeltaSpec):
        return m.label, {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
    if isinstance(m, LatentSpec) and m.rot_dim:
        return "latent_attention", {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                                    "scale": m.scale, "rot": _rotary_config(m.rotary)}
    if isinstance(m, LatentSpec):
        return "latent_attention", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                                    "scale": m.scale, "mask": _mask_config(m.window)}
    if isinstance(m, SsdSpec):
        return "mamba2", {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv,
                          "norm_groups": m.norm_groups}
    if isinstance(m, ConvAttentionSpec):
        return "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv, "scale": m.scale,
                             "rot": {"dims": m.rotary.dims, "base": m.rotary.base},
                             "mask": {"size": m.window, "keep_first": m.keep} if m.window else None}
    if isinstance(m, BiasedAttentionSpec):
        return "attention_2", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                               "bias_max": m.bias_max,
                               "q_temp": {"coef": m.temp_coef, "every": m.temp_every} if m.temp_every else None}
    if isinstance(m, DifferentialSpec):
        return "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff,
                             "rot": _rotary_config(m.rotary), "mask": _mask_config(m.chunk)}
    if isinstance(m, MinGruSpec):
        return "mingru", {"width": m.width}
    a, g = m.left, m.right
    rot = {"scaling": None, **_rotary_config(a.rotary)}
    return "parallel", {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale,
                                 "mask": _mask_config(a.window), "rot": rot},
                        "right": {"heads": g.heads, "dim": g.dim, "vdim": g.vdim, "tau": g.tau},
                        "left_scale": m.left_scale, "right_scale": m.right_scale}


def architecture_of(raw: dict) -> str | None:
    """Architecture a configuration names when it is one of this family's, else None."""
    arch = raw.get("architecture")
    return arch if arch in ARCHITECTURES else None


def _window(m: dict) -> int:
    mask = m.get("mask")
    if not mask:
        return 0
    if int(mask["size"]) < 1:
        raise LayeredConfigError("an attention window holds at least the token itself")
    return int(mask["size"])


def _read_rotary(rot: dict | None) -> RotarySpec:
    if not rot:
        return RotarySpec(0, 1.0)
    sc = rot.get("scaling")
    if sc:
        factor = float(sc["factor"])
        sc = ("yarn", factor, float(sc["original"]), float(sc["fast"]), float(sc["slow"]), 0.1 * math.log(factor) + 1.0)
    return RotarySpec(int(rot["dims"]), float(rot["base"]), sc or None)


def _read_delta(m: dict, p: str, rank, per_channel: bool = False) -> DeltaSpec:
    return DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), per_channel,
                     rank(f"{p}.a1") if per_channel else 0, rank(f"{p}.g1") if per_channel else 0)


def _read_latent(m: dict, p: str, rank) -> LatentSpec:
    return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]),
                      _window(m))


def _read_rotated_latent(m: dict, p: str, rank) -> LatentSpec:
    return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), 0, int(m["kv_rank"]), float(m["scale"]), 0, int(m["rot_dim"]),
                      _read_rotary(m["rot"]), False)


def _read_differential(m: dict, p: str, rank) -> DifferentialSpec:
    return DifferentialSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                            _read_rotary(m.get("rot")), float(m["diff"]), _window(m))


def _read_mingru(m: dict, p: str, rank) -> MinGruSpec:
    return MinGruSpec(int(m["width"]))


def _read_mamba2(m: dict, p: str, rank) -> SsdSpec:
    return SsdSpec(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m["norm_groups"]))


def _read_parallel(m: dict, p: str, rank) -> PairSpec:
    a, g = m["left"], m["right"]
    if int(a.get("vdim", a["dim"])) != int(a["dim"]):
        raise LayeredConfigError("the values of this attention are its keys: vdim equals dim")
    left = AttentionSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), float(a["scale"]), _read_rotary(a.get("rot")), _window(a))
    right = GatedLinearSpec(int(g["heads"]), int(g["dim"]), int(g["vdim"]), float(g["tau"]), rank(f"{p}.right.a1"))
    return PairSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _read_conv_attention(m: dict, p: str, rank) -> ConvAttentionSpec:
    mask = m.get("mask") or {}
    return ConvAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m.get("conv") or 1),
                             float(m["scale"]), _read_rotary(m.get("rot")), _window(m), int(mask.get("keep_first") or 0))


def _read_biased_attention(m: dict, p: str, rank) -> BiasedAttentionSpec:
    temp = m.get("q_temp") or {}
    if temp and int(temp["every"]) < 1:
        raise LayeredConfigError("the query factor grows every positive number of positions")
    return BiasedAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), rank(f"{p}.rel"),
                               int(m["bias_max"]), float(temp.get("coef", 0.0)), int(temp.get("every", 0)))


def _read_ff(mlp: dict | None, i: int, d: Design) -> dict:
    """Feed-forward fields of a ``LayerSpec``."""
    if not mlp:
        return {}
    kind = mlp.get("kind")
    if kind == "dense":
        return {"ff": int(mlp["ff"]), **({"limit": float(mlp["limit"])} if d.ff == "clamped_glu" else {})}
    if kind != "moe" or not d.streams:
        raise LayeredConfigError(f"layer {i}: unknown feed-forward {kind!r}")
    r, shared = mlp["router"], mlp.get("shared")
    return {"routed": RoutedSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(r.get("identity") or 0),
                                 int(shared["ff"]) if shared else 0)}


_MIXER_READERS = {"delta": _read_delta, "channel_delta": lambda m, p, rank: _read_delta(m, p, rank, True),
                  "latent": _read_latent, "rotated_latent": _read_rotated_latent, "mamba2": _read_mamba2, "parallel": _read_parallel,
                  "conv_attention": _read_conv_attention, "biased_attention": _read_biased_attention,
                  "differential": _read_differential, "mingru": _read_mingru}


def parse_layered_config(raw: dict, shapes: dict[str, tuple[int, ...]] | None = None, name: str = "") -> LayeredConfig:
    """``config.json`` -> configuration.  Sizes that only a tensor's shape states (the inner sizes of the low-rank decay and
    gate projections) come from ``shapes``."""
    arch = architecture_of(raw)
    if arch is None:
        raise LayeredConfigError(f"architecture {raw.get('architecture')!r} is not one of {ARCHITECTURES}")
    shapes = shapes or {}

    def rank(tensor: str) -> int:
        if tensor not in shapes:
            raise LayeredConfigError(f"the size of {tensor} is stated by the checkpoint's tensors only")
        return int(shapes[tensor][0])

    layers = []
    for i, l in enumerate(raw["layers"]):
        if l["type"] not in DESIGNS[arch].mixers:
            raise LayeredConfigError(f"layer {i}: unknown mixer {l['type']!r}")
        mixer = _MIXER_READERS[DESIGNS[arch].mixers[l["type"]]](l["mixer"], f"l{i}.mix", rank)
        layers.append(LayerSpec(mixer, **_read_ff(l.get("mlp"), i, DESIGNS[arch])))
    loop, side = raw.get("loop"), raw.get("token_side")
    more = {}
    if DESIGNS[arch].streams:
        more["streams"] = int(raw.get("streams") or 1)
    if DESIGNS[arch].embed_scale:
        more["embed_scale"] = float((raw.get("embedding") or {}).get("scale", 1.0))
    cfg = LayeredConfig(name or arch, int(raw["vocab"]), int(raw["width"]), tuple(layers), float(raw["norm"]["eps"]),
                        (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None, architecture=arch,
                        side_dim=int(side["dim"]) if side else 0, **more)
    cfg.validate()
    return cfg


# ------------------------------------------------------------------ tensor inventory
def _mixer_shapes(m: MixerSpec, p: str, W: int) -> dict[str, tuple[int, ...]]:
    out: dict[str, tuple[int, ...]] = {}
    if isinstance(m, PairSpec):
        return {**_mixer_shapes(m.left, f"{p}.left", W), **_mixer_shapes(m.right, f"{p}.right", W)}
    if isinstance(m, DeltaSpec):
        for t, c in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
            out[f"{p}.{t}"] = (c, W)
            out[f"{p}.{t}.conv"] = (c, m.conv)
        out[f"{p}.b"] = (m.heads, W)
        out[f"{p}.A_log"] = (m.heads,)
        out[f"{p}.norm"] = (m.vdim,)
        if m.per_channel:
            out.update({f"{p}.a1": (m.decay_rank, W), f"{p}.a2": (m.heads * m.dim, m.decay_rank),
                        f"{p}.dt_bias": (m.heads * m.dim,),
                        f"{p}.g1": (m.gate_rank, W), f"{p}.g2": (m.heads * m.vdim, m.gate_rank)})
        else:
            out.update({f"{p}.a": (m.heads, W), f"{p}.dt_bias": (m.heads,), f"{p}.g": (m.heads * m.vdim, W)})
    elif isinstance(m, LatentSpec) and m.rot_dim:
        out.update({f"{p}.q": (m.heads * (m.dim + m.rot_dim), W), f"{p}.dkv": (m.kv_rank + m.rot_dim, W), f"{p}.dkv.norm": (m.kv_rank,),
                    f"{p}.uk": (m.heads * m.dim, m.kv_rank), f"{p}.uv": (m.heads * m.vdim, m.kv_rank)})
    elif isinstance(m, DifferentialSpec):
        out.update({f"{p}.q": (m.heads * 2 * m.dim, W), f"{p}.k": (m.kv_heads * 2 * m.dim, W), f"{p}.v": (m.kv_heads * m.vdim, W),
                    f"{p}.g": (m.out_width, W)})
        out.update({f"{p}.{t}": (m.dim,) for t in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
    elif isinstance(m, MinGruSpec):
        out.update({f"{p}.{t}": (m.width, W) for t in "zxg"})
        out.update({f"{p}.{t}.b": (m.width,) for t in "zx"})
    elif isinstance(m, LatentSpec):
        out.update({f"{p}.dq": (m.q_rank, W), f"{p}.dq.norm": (m.q_rank,), f"{p}.uq": (m.heads * m.dim, m.q_rank),
                    f"{p}.dkv": (m.kv_rank, W), f"{p}.dkv.norm": (m.kv_rank,), f"{p}.uk": (m.heads * m.dim, m.kv_rank),
                    f"{p}.uv": (m.heads * m.vdim, m.kv_rank), f"{p}.g": (m.heads, W)})
    elif isinstance(m, AttentionSpec):
        out.update({f"{p}.q": (m.heads * m.dim, W), f"{p}.k": (m.kv_heads * m.dim, W), f"{p}.q.norm": (m.dim,),
                    f"{p}.k.norm": (m.dim,)})
    elif isinstance(m, _QkvSpec):
        sizes = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        out.update({f"{p}.{t}": (n, W) for t, n in sizes.items()})
        if isinstance(m, ConvAttentionSpec):
            out.update({f"{p}.{t}.conv": (n, m.conv) for t, n in sizes.items()})
        else:
            out.update({f"{p}.q.norm": (sizes["q"],), f"{p}.k.norm": (sizes["k"],), f"{p}.rel": (m.buckets, m.heads)})
    elif isinstance(m, GatedLinearSpec):
        out.update({f"{p}.{t}": (m.heads * c, W) for t, c in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim))})
        out.update({f"{p}.norm": (m.vdim,), f"{p}.a1": (m.decay_rank, W), f"{p}.a2": (m.heads * m.dim, m.decay_rank),
                    f"{p}.a2.b": (m.heads * m.dim,)})
    else:
        out.update({f"{p}.in": (m.out_width + m.channels + m.heads, W), f"{p}.conv": (m.channels, m.conv),
                    f"{p}.conv.b": (m.channels,), f"{p}.dt_bias": (m.heads,), f"{p}.A_log": (m.heads,), f"{p}.D": (m.heads,),
                    f"{p}.norm": (m.out_width,)})
    out[f"{p}.o"] = (W, m.out_width)
    return out


def tensor_shapes(cfg: LayeredConfig) -> dict[str, tuple[int, ...]]:
    """Every tensor of a checkpoint of this configuration."""
    W, d = cfg.hidden_size, cfg.design
    norm = () if d.scalar_norm else (W,)
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab_size, W), "final.norm": norm}
    if d.embed_norm:
        out["embed.norm"] = (W,)
    if not d.tied_head:
        out["head"] = (cfg.vocab_size, W)
    if cfg.loop is not None and d.loop == "project":
        out["loop.in"] = (W, 2 * W)
    if cfg.side_dim:
        out["side.embed"] = (cfg.vocab_size, cfg.num_layers * cfg.side_dim)
    for i, l in enumerate(cfg.layers):
        out[f"l{i}.norm1"] = norm
        out.update(_mixer_shapes(l.mixer, f"l{i}.mix", W))
        if d.sequential and l.has_ff:
            out[f"l{i}.norm2"] = norm
        if d.gated:
            for q in (1, 2) if l.has_ff else (1,):
                out.update({f"l{i}.rg{q}": (W, W), f"l{i}.rg{q}.b": (W,)})
        if d.streams:
            for q in (1, 2) if l.has_ff else (1,):
                out.update({f"l{i}.hc{q}.in": (cfg.streams,), f"l{i}.hc{q}.out": (cfg.streams,),
                            f"l{i}.hc{q}.mix": (cfg.streams, cfg.streams)})
        if l.routed is not None:
            r, p = l.routed, f"l{i}.mlp"
            for e in range(r.experts):
                out.update({f"{p}.e{e}.up": (r.ff, W), f"{p}.e{e}.down": (W, r.ff)})
            out.update({f"{p}.router": (r.outputs, W), f"{p}.correction": (r.outputs,)})
            if r.shared_ff:
                out.update({f"{p}.shared.up": (r.shared_ff, W), f"{p}.shared.down": (W, r.shared_ff), f"{p}.shared.sg": (1, W)})
        if l.ff:
            if d.ff.endswith("_glu"):
                out[f"l{i}.mlp.gate"] = (l.ff, W)
            out[f"l{i}.mlp.up"] = (l.ff, W)
            out[f"l{i}.mlp.down"] = (W, l.ff)
        if cfg.side_dim:
            out.update({f"l{i}.side.gate": (cfg.side_dim, W), f"l{i}.side.proj": (W, cfg.side_dim), f"l{i}.side.norm": (W,)})
    return out


def check_inventory(cfg: LayeredConfig, shapes: dict[str, tuple[int, ...]]) -> None:
    """The checkpoint's tensors are exactly the configuration's (what a missing feed-forward would need is ignored)."""
    want = tensor_shapes(cfg)
    for n, s in want.items():
        if n not in shapes:
            raise LayeredConfigError(f"missing tensor {n}")
        if tuple(shapes[n]) != s:
            raise LayeredConfigError(f"{n}: shape {tuple(shapes[n])}, expected {s}")
    idle = {f"l{i}.{t}" for i, l in enumerate(cfg.layers) if cfg.design.sequential and not l.has_ff
            for t in ("norm2", "hc2.in", "hc2.out", "hc2.mix", "rg2", "rg2.b")}
    extra = sorted(set(shapes) - set(want) - idle)
    if extra:
        raise LayeredConfigError(f"checkpoint has {len(extra)} tensors this configuration does not own, e.g. {extra[:3]}")


def random_tensors(cfg: LayeredConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights with the magnitudes of a trained model: unit-variance activations through every product."""
    g = torch.Generator(device=device).manual_seed(seed)
    stream = ("norm", "norm1", "norm2")              # norms of the residual stream; the others are plain factors
    out = {}
    for n, s in tensor_shapes(cfg).items():
        z = torch.randn(s, generator=g, device=device)
        last = n.rsplit(".", 1)[-1]
        if last in stream:
            of_stream = n in ("embed.norm", "final.norm") or n.count(".") == 1
            t = (1.0 - cfg.design.norm_offset if of_stream else 1.0) + 0.1 * z
        elif ".hc" in n:                             # streams that stay alike, each sublayer's input and result of about their size
            t = 0.1 * z + {"in": 1.0 / cfg.streams, "out": 1.0}.get(last, torch.eye(cfg.streams, device=device) if last == "mix" else 0.0)
        elif last == "rel":
            t = 0.5 * z
        elif last == "correction":
            t = 0.02 * z
        elif n == "embed" and cfg.design.embed_scale:
            t = z / cfg.embed_scale
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.3 * z / s[0] ** 0.25
        elif last == "A_log":
            t = 0.5 * z - 2.0
        elif last in ("dt_bias", "b") and len(s) == 1:
            t = 0.5 * z
        elif last == "D":
            t = 1.0 + 0.1 * z
        elif n == "embed" and not cfg.design.tied_head or n == "side.embed":
            t = z
        else:
            t = z / math.sqrt(s[1])
        out[n] = t.to(torch.bfloat16)
    return out


def write_checkpoint(path: str | Path, cfg: LayeredConfig, tensors: dict[str, torch.Tensor]) -> Path:
    from safetensors.torch import save_file
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    save_file({n: t.contiguous() for n, t in tensors.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(cfg.to_config(), indent=1))
    return path


# ------------------------------------------------------------------ packed weights
def _pad(t: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    out = torch.zeros(rows, cols, dtype=torch.bfloat16, device=t.device)
    out[:t.shape[0], :t.shape[1]] = t
    return out


def _matrix(t: torch.Tensor) -> wq_pack.PackedWeight:
    """A bf16 matrix with zero columns up to the GEMM's K block (both arithmetic modes read it as stored)."""
    return wq_pack.pack_bf16(_pad(t, t.shape[0], round_up(t.shape[1], wq_pack.BLOCK_K)))


@dataclass
class BlockDiagonal:
    """Per-head matrices ``[H, n, k]`` as one block-diagonal operand: groups of ``heads`` consecutive heads share a block of
    ``rows`` output rows (a multiple of the GEMM's 128-row tile) and ``w.k`` input columns, zero off its own diagonal.
    ``rows`` 0: one ordinary matrix (all heads in one group)."""
    w: wq_pack.PackedWeight
    heads: int
    rows: int

    @staticmethod
    def group(n: int, total: int) -> int:
        return min(total, wq_pack.TILE_N // math.gcd(n, wq_pack.TILE_N))

    @staticmethod
    def pack(per_head: torch.Tensor) -> "BlockDiagonal":
        H, n, k = per_head.shape
        hp = BlockDiagonal.group(n, H)
        kg = round_up(hp * k, wq_pack.BLOCK_K)
        out = torch.zeros(H * n, kg, dtype=torch.bfloat16, device=per_head.device)
        for h in range(H):
            c = (h % hp) * k
            out[h * n:(h + 1) * n, c:c + k] = per_head[h]
        return BlockDiagonal(wq_pack.pack_bf16(out), hp, hp * n if hp < H else 0)


@dataclass
class DeltaWeights:
    spec: DeltaSpec
    conv_w: torch.Tensor             # fp32 [taps, conv_width]
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm_w: torch.Tensor
    b_off: int                       # columns of the projection's output
    a_off: int                       # per head: decay logits; per channel: inner columns of the low-rank projections
    z_off: int                       # per head: output gate
    low: wq_pack.PackedWeight | None = None    # per channel: [decay logits | output gate] from the inner columns
    low_z: int = 0                   # first gate column of its output


@dataclass
class LatentWeights:
    spec: LatentSpec
    q_norm: torch.Tensor | None      # low-rank queries
    c_norm: torch.Tensor
    uq: wq_pack.PackedWeight | None  # rows in the column layout of ``absorb``'s input; None: the projection writes them at ``q_off``
    absorb: BlockDiagonal            # queries -> latent space
    value: BlockDiagonal             # latent outputs -> head outputs
    c_off: int
    g_off: int = -1                  # gates of the heads (< 0: none)
    q_off: int = 0                   # low-rank queries, or full ones
    qr_off: int = 0                  # rotated part of the queries [H, rot_dim]
    r_off: int = 0                   # ... of the shared key
    freq: torch.Tensor | None = None # fp32 [2, pairs] radians per position, and what rounding took from them
    rot_mult: float = 1.0


@dataclass
class AttentionWeights:
    spec: AttentionSpec
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    freq: torch.Tensor               # fp32 [pairs] radians per position
    rot_mult: float                  # factor on cosine and sine
    q_off: int
    k_off: int
    out_scale: float = 1.0


@dataclass
class GatedLinearWeights:
    spec: GatedLinearSpec
    low: wq_pack.PackedWeight        # decay logits from the inner columns
    bias: torch.Tensor
    norm_w: torch.Tensor             # times what the mixer's output is scaled by
    q_off: int
    k_off: int
    v_off: int
    g_off: int
    a_off: int


@dataclass
class SsdWeights:
    spec: SsdSpec
    conv_w: torch.Tensor             # fp32 [taps, conv_width], channels x | B | C
    conv_b: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    d: torch.Tensor
    norm_w: torch.Tensor
    z_off: int
    x_off: int
    dt_off: int


@dataclass
class PairWeights:
    spec: PairSpec
    left: object
    right: object


@dataclass
class ConvAttentionWeights:
    spec: ConvAttentionSpec
    conv_w: torch.Tensor             # fp32 [taps, conv_width]
    freq: torch.Tensor               # fp32 [2, pairs] radians per position, and what rounding took from them
    q_off: int


@dataclass
class BiasedAttentionWeights:
    spec: BiasedAttentionSpec
    q_norm: torch.Tensor             # fp32 [H d]
    k_norm: torch.Tensor             # fp32 [G d]
    bias: torch.Tensor               # fp32 [bias_max + 1, H] by distance
    q_off: int


@dataclass
class DifferentialWeights:
    spec: DifferentialSpec
    q_norm: torch.Tensor             # fp32 [d]
    k_norm: torch.Tensor
    freq: torch.Tensor               # fp32 [2, pairs]
    less: float                      # what the second map is multiplied by before it is taken away
    q_off: int
    g_off: int


@dataclass
class MinGruWeights:
    spec: MinGruSpec
    bias: torch.Tensor               # fp32 [2, width] of gate and candidate
    z_off: int
    x_off: int
    g_off: int


@dataclass
class StreamWeights:
    """How a sublayer reads and writes the residual streams (fp32)."""
    read: torch.Tensor               # [streams]
    write: torch.Tensor              # [streams]
    mix: torch.Tensor                # [streams, streams] from, to


@dataclass
class RoutedWeights:
    """ONE matrix reads the feed-forward's norm for everybody: [router | shared expert's gate] in fp32, then the shared expert's
    up rows behind the squared relu."""
    spec: RoutedSpec
    head: wq_pack.PackedWeight
    split: int                       # fp32 columns of its output
    correction: torch.Tensor
    up: wq_pack.PackedWeight         # experts stacked
    down: wq_pack.PackedWeight
    shared_down: wq_pack.PackedWeight | None


@dataclass
class SideWeights:
    """A layer's input from the token's side embedding."""
    gate: torch.Tensor               # bf16 [dim, W rounded up]
    proj: wq_pack.PackedWeight
    norm_w: torch.Tensor
    col: int                         # first column of the layer's part of the side embedding


@dataclass
class LayerWeights:
    norm: torch.Tensor               # fp32 factor of the norm
    proj: wq_pack.PackedWeight       # mixer inputs; parallel layers: [mixer inputs | feed-forward up]
    split: int                       # mixer columns
    ff: int
    mixer: object                    # DeltaWeights | LatentWeights | SsdWeights | PairWeights
    out: wq_pack.PackedWeight        # mixer output; parallel layers: [o | down]
    out_off: int                     # parallel layers: first feed-forward column of ``out``'s input
    norm2: torch.Tensor | None = None            # sequential layers: the feed-forward's norm, products and width of its activation
    gate_up: wq_pack.PackedWeight | None = None  # rows in the order of the fused gated activation
    down: wq_pack.PackedWeight | None = None
    side: SideWeights | None = None
    streams: tuple[StreamWeights, ...] = ()      # of the mixer and of the feed-forward
    routed: RoutedWeights | None = None
    rg_off: int = 0                  # gated residuals: columns of the gate's logits in the output of ``proj``,
    rg: tuple[torch.Tensor, ...] = ()            # biases (fp32 [W]) of the mixer's and of the feed-forward's gate; the latter's
    ff_rows: int = 0                 # logits follow these rows of ``gate_up``
    limit: float = 0.0               # of a clamped feed-forward

    def matrices(self) -> list[wq_pack.PackedWeight]:
        """Every packed matrix of the layer."""
        out = [self.proj, self.out]
        for part in ((self.mixer.left, self.mixer.right) if isinstance(self.mixer, PairWeights) else (self.mixer,)):
            if isinstance(part, LatentWeights):
                out += [m for m in (part.uq, part.absorb.w, part.value.w) if m is not None]
            elif getattr(part, "low", None) is not None:
                out.append(part.low)
        out += [m for m in (self.gate_up, self.down) if m is not None]
        if self.routed is not None:
            out += [m for m in (self.routed.head, self.routed.up, self.routed.down, self.routed.shared_down) if m is not None]
        return out + ([self.side.proj] if self.side is not None else [])


@dataclass
class LayeredWeights:
    embed: torch.Tensor
    embed_norm: torch.Tensor | None
    loop_in: wq_pack.PackedWeight | None
    layers: list[LayerWeights]
    final_norm: torch.Tensor
    lm_head: wq_pack.PackedWeight
    side_embed: torch.Tensor | None = None
    vocab_start: int = 0

    def nbytes(self) -> int:
        total = self.embed.numel() * 2 + self.lm_head.nbytes + (self.loop_in.nbytes if self.loop_in else 0)
        if self.side_embed is not None:
            total += self.side_embed.numel() * 2 + sum(l.side.gate.numel() * 2 for l in self.layers)
        return total + sum(m.nbytes for l in self.layers for m in l.matrices())


class _Rows:
    """Stacks row sections of a projection, each starting at a multiple of ``align`` columns of its output."""

    def __init__(self, k: int) -> None:
        self.k, self.parts, self.n = k, [], 0

    def add(self, *mats: torch.Tensor, align: int = 8, size: int = 0) -> int:
        self._fill(round_up(self.n, align) - self.n, mats[0])
        off = self.n
        for m in mats:
            self.parts.append(m.to(torch.bfloat16))
            self.n += m.shape[0]
        self._fill(max(0, off + size - self.n), mats[0])
        return off

    def _fill(self, n: int, like: torch.Tensor) -> None:
        if n:
            self.parts.append(torch.zeros(n, self.k, dtype=torch.bfloat16, device=like.device))
            self.n += n

    def end(self, align: int = 8) -> torch.Tensor:
        self._fill(round_up(self.n, align) - self.n, self.parts[0])
        return torch.cat(self.parts)


def _f32(get, n: str) -> torch.Tensor:
    return get(n).float().contiguous()


def _pack_delta(m: DeltaSpec, p: str, rows: _Rows, get) -> DeltaWeights:
    rows.add(get(f"{p}.q"), get(f"{p}.k"), get(f"{p}.v"))
    b_off = rows.add(get(f"{p}.b"))
    conv = torch.cat([get(f"{p}.{t}.conv") for t in "qkv"]).float()
    conv_w = torch.zeros(m.conv, m.conv_width, device=conv.device)
    conv_w[:, :m.channels] = conv.t()
    common = dict(spec=m, conv_w=conv_w.contiguous(), a_log=_f32(get, f"{p}.A_log"), dt_bias=_f32(get, f"{p}.dt_bias"),
                  norm_w=_f32(get, f"{p}.norm"), b_off=b_off)
    if not m.per_channel:
        a_off = rows.add(get(f"{p}.a"))
        return DeltaWeights(**common, a_off=a_off, z_off=rows.add(get(f"{p}.g")))
    inner = round_up(m.decay_rank + m.gate_rank, 64)
    a_off = rows.add(get(f"{p}.a1"), get(f"{p}.g1"), align=64, size=inner)
    low_z = round_up(m.heads * m.dim, 8)
    low = torch.zeros(low_z + m.heads * m.vdim, inner, dtype=torch.bfloat16, device=conv.device)
    low[:m.heads * m.dim, :m.decay_rank] = get(f"{p}.a2")
    low[low_z:, m.decay_rank:m.decay_rank + m.gate_rank] = get(f"{p}.g2")
    return DeltaWeights(**common, a_off=a_off, z_off=0, low=wq_pack.pack_bf16(low), low_z=low_z)


def _pack_latent(m: LatentSpec, p: str, rows: _Rows, get) -> LatentWeights:
    H, d, e, r, R, Rp = m.heads, m.dim, m.vdim, m.rot_dim, m.kv_rank, m.row_padded
    uk = torch.zeros(H, Rp, d, dtype=torch.bfloat16, device=get(f"{p}.uk").device)
    uk[:, :R] = get(f"{p}.uk").view(H, d, R).transpose(1, 2)
    absorb = BlockDiagonal.pack(uk)
    uv = torch.zeros(H, e, m.rank_padded, dtype=torch.bfloat16, device=uk.device)
    uv[:, :, :R] = get(f"{p}.uv").view(H, e, R)
    value = BlockDiagonal.pack(uv)
    # the query projection writes every head where its block of ``absorb`` reads it
    hp, kg = absorb.heads, absorb.w.k

    def spread(src: torch.Tensor) -> torch.Tensor:
        out = torch.zeros(-(-H // hp) * kg, src.shape[-1], dtype=torch.bfloat16, device=uk.device)
        for h in range(H):
            c = (h // hp) * kg + (h % hp) * d
            out[c:c + d] = src[h]
        return out
    c_norm = _f32(get, f"{p}.dkv.norm")
    if m.rot_dim:
        q = get(f"{p}.q").view(H, d + r, -1)
        q_off = rows.add(spread(q[:, :d]))
        qr_off = rows.add(q[:, d:].flatten(0, 1))
        down = get(f"{p}.dkv")
        c_off, r_off = rows.add(down[:R]), rows.add(down[R:])
        return LatentWeights(m, None, c_norm, None, absorb, value, c_off, q_off=q_off, qr_off=qr_off, r_off=r_off,
                             freq=m.rotary.split_table().to(uk.device).contiguous(), rot_mult=m.rotary.factor)
    q_off = rows.add(get(f"{p}.dq"))
    c_off = rows.add(get(f"{p}.dkv"))
    g_off = rows.add(get(f"{p}.g"))
    uq = spread(get(f"{p}.uq").view(H, d, m.q_rank))
    return LatentWeights(m, _f32(get, f"{p}.dq.norm"), c_norm, _matrix(uq), absorb, value, c_off, g_off, q_off)


def _pack_attention(m: AttentionSpec, p: str, rows: _Rows, get, out_scale: float = 1.0) -> AttentionWeights:
    q_off = rows.add(get(f"{p}.q"))
    k_off = rows.add(get(f"{p}.k"))
    freq, mult = m.rotary.table()
    q_norm = _f32(get, f"{p}.q.norm")
    return AttentionWeights(m, q_norm, _f32(get, f"{p}.k.norm"), freq.to(q_norm.device).contiguous(), mult, q_off, k_off, out_scale)


def _add_qkv(m: _QkvSpec, p: str, rows: _Rows, get) -> int:
    q_off = rows.add(get(f"{p}.q"))
    offs = q_off, rows.add(get(f"{p}.k")), rows.add(get(f"{p}.v"))
    assert tuple(o - q_off for o in offs) == m.offsets
    return q_off


def _pack_conv_attention(m: ConvAttentionSpec, p: str, rows: _Rows, get) -> ConvAttentionWeights:
    q_off = _add_qkv(m, p, rows, get)
    dev = get(f"{p}.q").device
    conv_w = torch.zeros(m.conv, m.conv_width, device=dev)
    for t, off in zip("qkv", m.offsets):
        w = get(f"{p}.{t}.conv").float()
        conv_w[:, off:off + w.shape[0]] = w.t()
    return ConvAttentionWeights(m, conv_w, m.rotary.split_table().to(dev).contiguous(), q_off)


def _pack_biased_attention(m: BiasedAttentionSpec, p: str, rows: _Rows, get) -> BiasedAttentionWeights:
    q_off = _add_qkv(m, p, rows, get)
    rel = _f32(get, f"{p}.rel")
    return BiasedAttentionWeights(m, _f32(get, f"{p}.q.norm"), _f32(get, f"{p}.k.norm"),
                                  rel[m.bucket_of_distance().to(rel.device)].contiguous(), q_off)


def _pack_differential(m: DifferentialSpec, p: str, rows: _Rows, get) -> DifferentialWeights:
    q_off = _add_qkv(m, p, rows, get)
    g_off = rows.add(get(f"{p}.g"))
    dot = [float((get(f"{p}.lq{i}").double() * get(f"{p}.lk{i}").double()).sum()) for i in (1, 2)]
    q_norm = _f32(get, f"{p}.q.norm")
    return DifferentialWeights(m, q_norm, _f32(get, f"{p}.k.norm"), m.rotary.split_table().to(q_norm.device).contiguous(),
                               math.exp(dot[0]) - math.exp(dot[1]) + m.diff, q_off, g_off)


def _pack_mingru(m: MinGruSpec, p: str, rows: _Rows, get) -> MinGruWeights:
    z_off, x_off, g_off = (rows.add(get(f"{p}.{t}")) for t in "zxg")
    return MinGruWeights(m, torch.stack([_f32(get, f"{p}.{t}.b") for t in "zx"]).contiguous(), z_off, x_off, g_off)


def _pack_gated_linear(m: GatedLinearSpec, p: str, rows: _Rows, get, out_scale: float = 1.0) -> GatedLinearWeights:
    q_off, k_off, v_off, g_off = (rows.add(get(f"{p}.{t}")) for t in "qkvg")
    inner = round_up(m.decay_rank, 64)
    a_off = rows.add(get(f"{p}.a1"), align=64, size=inner)
    return GatedLinearWeights(m, _matrix(get(f"{p}.a2").to(torch.bfloat16)), _f32(get, f"{p}.a2.b"),
                              out_scale * _f32(get, f"{p}.norm"), q_off, k_off, v_off, g_off, a_off)


def _pack_ssd(m: SsdSpec, p: str, rows: _Rows, get) -> SsdWeights:
    z, x, dt = get(f"{p}.in").split([m.out_width, m.channels, m.heads])
    z_off, x_off, dt_off = rows.add(z), rows.add(x), rows.add(dt)
    conv_w = torch.zeros(m.conv, m.conv_width, device=x.device)
    conv_w[:, :m.channels] = get(f"{p}.conv").float().t()
    conv_b = torch.zeros(m.conv_width, device=x.device)
    conv_b[:m.channels] = get(f"{p}.conv.b").float()
    return SsdWeights(m, conv_w, conv_b, *(_f32(get, f"{p}.{t}") for t in ("A_log", "dt_bias", "D", "norm")), z_off, x_off, dt_off)


def _pack_pair(m: PairSpec, p: str, rows: _Rows, get) -> PairWeights:
    return PairWeights(m, _PACKERS[type(m.left)](m.left, f"{p}.left", rows, get, out_scale=m.left_scale),
                       _PACKERS[type(m.right)](m.right, f"{p}.right", rows, get, out_scale=m.right_scale))


_PACKERS = {DeltaSpec: _pack_delta, LatentSpec: _pack_latent, AttentionSpec: _pack_attention, GatedLinearSpec: _pack_gated_linear,
            SsdSpec: _pack_ssd, PairSpec: _pack_pair, ConvAttentionSpec: _pack_conv_attention,
            BiasedAttentionSpec: _pack_biased_attention, DifferentialSpec: _pack_differential, MinGruSpec: _pack_mingru}


def _pack_output(m: MixerSpec, p: str, get, ff: int, W: int) -> tuple[torch.Tensor, int]:
    """Output projections side by side, with room for ``ff`` feed-forward columns: (matrix, first of those columns)."""
    off = round_up(m.out_width, 8)
    parts = ((m.left, f"{p}.left", 0), (m.right, f"{p}.right", m.right_off)) if isinstance(m, PairSpec) else ((m, p, 0),)
    out = torch.zeros(W, round_up(off + ff, 64), dtype=torch.bfloat16, device=get(f"{parts[0][1]}.o").device)
    for part, prefix, col in parts:
        out[:, col:col + part.out_width] = get(f"{prefix}.o")
    return out, off


def _pack_glu(gate: torch.Tensor, up: torch.Tensor, rest: torch.Tensor | None = None) -> tuple[wq_pack.PackedWeight, int]:
    """[gate ; up] in the row order of the GEMM's gated activation, the width padded to whole blocks of it, or, with ``rest`` rows
    behind them, to whole tiles: (matrix, rows of the gated activation)."""
    ff, k = gate.shape
    both = torch.zeros(2, round_up(ff, 16 if rest is None else wq_pack.TILE_N // 2), k, dtype=torch.bfloat16, device=gate.device)
    both[0, :ff], both[1, :ff] = gate, up
    w = wq_pack.swiglu_interleave(_matrix(both.flatten(0, 1)))
    if rest is None:
        return w, w.n
    codes = torch.cat([w.codes, _pad(rest, rest.shape[0], w.k)])
    return replace(w, n=codes.shape[0], codes=codes), w.n


def _stack(mats) -> wq_pack.PackedWeight:
    """Equal matrices along a leading axis, each as ``_matrix`` packs it."""
    packed = [_matrix(t.to(torch.bfloat16)) for t in mats]
    return replace(packed[0], codes=torch.stack([w.codes for w in packed]))


def _pack_routed(r: RoutedSpec, p: str, W: int, get) -> RoutedWeights:
    rows = _Rows(W)
    rows.add(get(f"{p}.router"))
    if r.shared_ff:
        rows.add(get(f"{p}.shared.sg"), align=1)
    rows.end()
    split = rows.n
    if r.shared_ff:
        rows.add(get(f"{p}.shared.up"))
    return RoutedWeights(r, _matrix(rows.end(1)), split, _f32(get, f"{p}.correction"),
                         _stack(get(f"{p}.e{e}.up") for e in range(r.experts)), _stack(get(f"{p}.e{e}.down") for e in range(r.experts)),
                         _matrix(get(f"{p}.shared.down").to(torch.bfloat16)) if r.shared_ff else None)


def _pack_streams(p: str, get) -> StreamWeights:
    return StreamWeights(*(_f32(get, f"{p}.{t}") for t in ("in", "out", "mix")))


def _norm_factor(cfg: LayeredConfig, get, name: str) -> torch.Tensor:
    """fp32 factor per channel of a norm of the residual."""
    return (cfg.design.norm_offset + _f32(get, name)).expand(cfg.hidden_size).contiguous()


def pack_layer(cfg: LayeredConfig, i: int, get) -> LayerWeights:
    """``get(name)`` -> tensor on the target device."""
    l, p, W, d = cfg.layers[i], f"l{i}", cfg.hidden_size, cfg.design
    rows = _Rows(W)
    mixer = _PACKERS[type(l.mixer)](l.mixer, f"{p}.mix", rows, get)
    rg_off = rows.add(get(f"{p}.rg1")) if d.gated else 0
    proj = rows.end()
    split = proj.shape[0]
    joint = 0 if d.sequential else l.ff
    out, out_off = _pack_output(l.mixer, f"{p}.mix", get, joint, W)
    if joint:
        proj = torch.cat([proj, get(f"{p}.mlp.up").to(torch.bfloat16)])
        out[:, out_off:out_off + l.ff] = get(f"{p}.mlp.down")
    lw = LayerWeights(_norm_factor(cfg, get, f"{p}.norm1"), _matrix(proj), split, joint, mixer, wq_pack.pack_bf16(out), out_off)
    if d.streams:
        lw.streams = tuple(_pack_streams(f"{p}.hc{q}", get) for q in ((1, 2) if l.has_ff else (1,)))
    if d.sequential and l.has_ff:
        lw.norm2 = _norm_factor(cfg, get, f"{p}.norm2")
    if d.gated:
        lw.rg_off, lw.rg, lw.limit = rg_off, tuple(_f32(get, f"{p}.rg{q}.b") for q in ((1, 2) if l.has_ff else (1,))), l.limit
    if l.routed is not None:
        lw.routed = _pack_routed(l.routed, f"{p}.mlp", W, get)
    if d.sequential and l.ff:
        lw.gate_up, lw.ff_rows = _pack_glu(get(f"{p}.mlp.gate"), get(f"{p}.mlp.up"),
                                           get(f"{p}.rg2").to(torch.bfloat16) if d.gated else None)
        lw.down = _matrix(get(f"{p}.mlp.down").to(torch.bfloat16))
    if cfg.side_dim:
        gate = get(f"{p}.side.gate").to(torch.bfloat16)
        lw.side = SideWeights(_pad(gate, gate.shape[0], round_up(W, 64)), _matrix(get(f"{p}.side.proj").to(torch.bfloat16)),
                              _f32(get, f"{p}.side.norm"), i * cfg.side_dim)
    return lw


def pack_weights(cfg: LayeredConfig, get) -> LayeredWeights:
    d = cfg.design
    embed = get("embed").to(torch.bfloat16).contiguous()
    return LayeredWeights(
        embed=embed, embed_norm=_norm_factor(cfg, get, "embed.norm") if d.embed_norm else None,
        loop_in=_matrix(get("loop.in")) if cfg.loop is not None and d.loop == "project" else None,
        layers=[pack_layer(cfg, i, get) for i in range(cfg.num_layers)],
        final_norm=_norm_factor(cfg, get, "final.norm"), lm_head=_matrix(embed if d.tied_head else get("head")),
        side_embed=get("side.embed").to(torch.bfloat16).contiguous() if cfg.side_dim else None)


def random_layered_weights(cfg: LayeredConfig, device="cuda", seed: int = 0, *_, **__) -> LayeredWeights:
    t = random_tensors(cfg, seed, device)
    return pack_weights(cfg, t.__getitem__)


def load_layered_weights(ck, device="cuda", *_, **__) -> LayeredWeights:
    """Admitted checkpoint -> packed weights on ``device``."""
    def get(name: str) -> torch.Tensor:
        return ck.store.get(name).to(device)
    return pack_weights(ck.cfg, get)


# ------------------------------------------------------------------ named configurations
def tiny_layered_config() -> LayeredConfig:
    """A few small layers of every kind, with a loop (tests and demonstrations)."""
    return LayeredConfig(
        "layered-tiny", 384, 192,
        (LayerSpec(DeltaSpec(4, 2, 48, 40, 4), 160), LayerSpec(LatentSpec(5, 24, 40, 56, 72, 0.2, 37), 160),
         LayerSpec(DeltaSpec(3, 3, 40, 24, 2, True, 12, 20), 0), LayerSpec(LatentSpec(4, 32, 32, 64, 64, 0.17, 50), 128)),
        1e-5, (1, 3, 2))


def layered_8b_config() -> LayeredConfig:
    """Layers of the size of an 8B model: three delta layers (two with a decay per channel) and one windowed latent
    attention layer in turn."""
    delta = LayerSpec(DeltaSpec(32, 16, 128, 128, 4), 12288)
    channel = LayerSpec(DeltaSpec(32, 32, 128, 128, 4, True, 128, 128), 12288)
    latent = LayerSpec(LatentSpec(32, 128, 128, 1536, 512, 128 ** -0.5, 1024), 12288)
    return LayeredConfig("layered-8b", 151936, 4096, (delta, channel, channel, latent) * 9, 1e-6, None)


def tiny_sequential_config() -> LayeredConfig:
    """A few small sequential layers of both kinds (tests and demonstrations)."""
    pair = PairSpec(AttentionSpec(6, 2, 40, 0.2, RotarySpec(24, 10000.0, ("yarn", 4.0, 128.0, 16.0, 1.0, 0.1 * math.log(4.0) + 1.0)), 37),
                    GatedLinearSpec(3, 24, 32, 8.0, 12), 0.8, 1.1)
    ssd = SsdSpec(6, 24, 20, 2, 4, 3)
    return LayeredConfig("layered-seq-tiny", 384, 192, (LayerSpec(ssd, 160), LayerSpec(pair, 160), LayerSpec(ssd, 96), LayerSpec(pair, 0)),
                         1e-5, architecture="Loduzen", side_dim=20)


def sequential_8b_config() -> LayeredConfig:
    """Sequential layers of the size of an 8B model: one state-space layer in four, else windowed sink attention beside gated
    linear attention."""
    rotary = RotarySpec(64, 1e6, ("yarn", 8.0, 8192.0, 32.0, 1.0, 0.1 * math.log(8.0) + 1.0))
    pair = LayerSpec(PairSpec(AttentionSpec(32, 8, 128, 128 ** -0.5, rotary, 1024), GatedLinearSpec(16, 128, 128, 16.0, 64), 1.0, 1.0), 12288)
    ssd = LayerSpec(SsdSpec(128, 64, 128, 8, 4, 8), 12288)
    return LayeredConfig("layered-seq-8b", 151936, 4096, (ssd, pair, pair, pair) * 8, 1e-6, architecture="Loduzen", side_dim=64)


def tiny_streams_config() -> LayeredConfig:
    """A few small layers of both attentions and both feed-forwards on three residual streams (tests and demonstrations)."""
    near = ConvAttentionSpec(6, 2, 40, 24, 4, 0.2, RotarySpec(24, 10000.0), 37, 5)
    far = BiasedAttentionSpec(4, 4, 32, 48, 0.2, 12, 50, 0.3, 20)
    routed = RoutedSpec(6, 3, 80, 2, 96)
    return LayeredConfig("layered-streams-tiny", 384, 192, (LayerSpec(near, 160), LayerSpec(far, routed=routed), LayerSpec(near, routed=routed),
                                                            LayerSpec(far)), 1e-5, architecture="Vimelorn", streams=3, embed_scale=13.0)


def streams_moe_config() -> LayeredConfig:
    """Layers of the size of a mixture-of-experts model with 4 of 64 experts: three windowed attention layers and one of every
    earlier token in turn, every second feed-forward routed, two residual streams."""
    near = ConvAttentionSpec(32, 8, 128, 128, 4, 1.0, RotarySpec(128, 1e6), 1024, 8)
    far = BiasedAttentionSpec(32, 8, 128, 128, 128 ** -0.5, 32, 512, 0.1, 4096)
    routed = RoutedSpec(64, 4, 1024, 8, 1024)
    group = (LayerSpec(near, 8192), LayerSpec(near, routed=routed), LayerSpec(near, 8192), LayerSpec(far, routed=routed))
    return LayeredConfig("layered-streams-moe", 151936, 4096, group * 8, 1e-6, architecture="Vimelorn", streams=2, embed_scale=64.0)


def tiny_gated_config() -> LayeredConfig:
    """A few small layers of every kind with gated residuals and a loop (tests and demonstrations)."""
    latent = LatentSpec(5, 24, 40, 0, 72, 0.2, 0, 20, RotarySpec(20, 10000.0, ("yarn", 4.0, 128.0, 16.0, 1.0, 0.1 * math.log(4.0) + 1.0)), False)
    pair = DifferentialSpec(6, 2, 24, 40, 0.2, RotarySpec(16, 10000.0), 0.4, 37)
    return LayeredConfig("layered-gated-tiny", 384, 192, (LayerSpec(latent, 160, limit=2.0), LayerSpec(MinGruSpec(224), 128, limit=2.0),
                                                          LayerSpec(pair, 160, limit=2.0), LayerSpec(MinGruSpec(160))),
                         1e-5, (1, 3, 2), architecture="Fovunex", embed_scale=0.7)


def gated_8b_config() -> LayeredConfig:
    """Layers of the size of an 8B model with gated residuals: latent attention over every earlier token, differential attention in
    chunks and element-wise recurrences in turn."""
    yarn = ("yarn", 8.0, 8192.0, 32.0, 1.0, 0.1 * math.log(8.0) + 1.0)
    latent = LayerSpec(LatentSpec(32, 128, 128, 0, 512, 192 ** -0.5, 0, 64, RotarySpec(64, 1e6, yarn), False), 12288, limit=7.0)
    pair = LayerSpec(DifferentialSpec(32, 8, 64, 128, 64 ** -0.5, RotarySpec(64, 1e6), 0.6, 4096), 12288, limit=7.0)
    gru = LayerSpec(MinGruSpec(6144), 12288, limit=7.0)
    return LayeredConfig("layered-gated-8b", 151936, 4096, (pair, gru, pair, latent) * 8, 1e-6, architecture="Fovunex", embed_scale=1.0)


NAMED = {"layered-tiny": tiny_layered_config, "layered-8b": layered_8b_config, "layered-seq-tiny": tiny_sequential_config,
         "layered-seq-8b": sequential_8b_config, "layered-streams-tiny": tiny_streams_config, "layered-streams-moe": streams_moe_config,
         "layered-gated-tiny": tiny_gated_config, "layered-gated-8b": gated_8b_config}


_MIXER_SOURCES = {DeltaSpec: ("delta_rule.cu",), LatentSpec: ("latent_attn.cu",), AttentionSpec: ("gqa_attn.cu",),
                  GatedLinearSpec: ("linear_recurrence.cu",), SsdSpec: ("linear_recurrence.cu",),
                  ConvAttentionSpec: ("qkv_prepare.cu", "gqa_attn.cu"), BiasedAttentionSpec: ("qkv_prepare.cu", "gqa_attn.cu"),
                  DifferentialSpec: ("qkv_prepare.cu", "gqa_attn.cu"), MinGruSpec: ("mingru.cu",)}


def kernel_sources(cfg: LayeredConfig) -> set[str]:
    """Sources of ``csrc`` whose kernels a model of this configuration launches: products, rows, pages, sampling, and its mixers'."""
    out = {"wq_gemm.cu", "wq_gemm_sk.cu", "elementwise.cu", "kv_cache.cu", "sampling.cu", "guard.cu", "layered.cu"}
    for l in cfg.layers:
        for part in l.mixer.parts:
            out.update(_MIXER_SOURCES[type(part)])
        if l.routed is not None:
            out.add("moe.cu")
    if cfg.design.streams:
        out.add("streams.cu")
    return out


def with_dtype(cfg: LayeredConfig, dtype: str) -> LayeredConfig:
    return replace(cfg, dtype=dtype)
