"""Layered decoders: every layer names its own token mixer, a run of layers may be repeated, the residual stream is fp32.

``config.json`` of such a checkpoint has ``architecture`` (``Bumodra``), ``vocab``, ``width``, ``norm.eps``, the list
``layers`` and optionally ``loop``.  A layer is parallel: mixer and feed-forward read the same norm and their outputs are
added to the residual together.  ``loop`` = {start, stop, times} runs the layers ``start .. stop - 1`` ``times`` times with
the same weights, each pass with its own cache and state; a pass starts with a projection of [residual ; embedding output].

Mixers (``MIXERS``; another one is added there, in ``pack_layer`` and in ``models/layered_runner.py``):

* ``delta`` / ``channel_delta``: short convolution, gated delta rule with one decay per head / per (head, key channel);
* ``latent_attention``: attention over cached latents with a sliding window and a gate per head.

Weights are packed for the parallel layout: ONE matrix holds all projections that read the norm (mixer inputs, then the
feed-forward's up rows), ONE matrix holds both output projections side by side ([o | down]), so a layer has two large
products whatever its mixer is.  Rows and columns are padded with zeros to what the GEMM asks for.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, replace
from pathlib import Path

import torch

from ..ops import wq_pack
from .config import QuantSpec

ARCHITECTURES = ("Bumodra",)
MAX_CONV_TAPS, MAX_DELTA_DIM, MAX_LATENT = 16, 256, 1024      # limits of the kernels


class LayeredConfigError(ValueError):
    pass


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


# ------------------------------------------------------------------ configuration
@dataclass(frozen=True)
class DeltaSpec:
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
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0              # 0: every earlier token

    @property
    def rank_padded(self) -> int:
        """Columns of a cached latent: the widths the attention kernels are built for."""
        return next((p for p in (64, 128, 256, 512) if self.kv_rank <= p), MAX_LATENT)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def validate(self) -> None:
        if min(self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank) <= 0 or self.window < 0:
            raise LayeredConfigError("latent attention sizes are positive")
        if self.kv_rank > MAX_LATENT:
            raise LayeredConfigError(f"latents of up to {MAX_LATENT} channels are served")


@dataclass(frozen=True)
class LayerSpec:
    mixer: object                # DeltaSpec | LatentSpec
    ff: int = 0                  # feed-forward width (squared relu); 0 = none


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
    family: str = "layered"
    max_position: int = 1 << 20                   # no positions enter the model: only memory limits the context
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
    def is_hybrid(self) -> bool:
        """Some layer keeps recurrent state per request."""
        return any(isinstance(l.mixer, DeltaSpec) for l in self.layers)

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

    @property
    def page_bytes(self) -> int:
        """One 16-token page of every attention run."""
        return sum(16 * self.layers[i].mixer.rank_padded * self.act_bytes for i, _ in self.runs
                   if isinstance(self.layers[i].mixer, LatentSpec))

    @property
    def state_bytes_per_request(self) -> int:
        return sum(self.layers[i].mixer.state_bytes(self.act_bytes) for i, _ in self.runs
                   if isinstance(self.layers[i].mixer, DeltaSpec))

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers)) <= 0 or self.rms_eps < 0:
            raise LayeredConfigError("vocab, width and the layer list are positive")
        if self.dtype not in ("bfloat16", "float32"):
            raise LayeredConfigError(f"dtype {self.dtype!r} is not bfloat16 or float32")
        for l in self.layers:
            l.mixer.validate()
            if l.ff < 0:
                raise LayeredConfigError("feed-forward widths are positive")
        if self.loop is not None:
            a, b, times = self.loop
            if not 0 <= a < b <= self.num_layers or times < 1:
                raise LayeredConfigError("loop needs 0 <= start < stop <= layers and times >= 1")

    def to_config(self) -> dict:
        """The ``config.json`` object of this configuration."""
        layers = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, DeltaSpec):
                kind = "channel_delta" if m.per_channel else "delta"
                mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            else:
                kind = "latent_attention"
                mix = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                       "scale": m.scale, "mask": {"size": m.window} if m.window else None}
            layers.append({"type": kind, "mixer": mix, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        loop = None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop))
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.rms_eps}, "layers": layers, "loop": loop}


def architecture_of(raw: dict) -> str | None:
    """Architecture a configuration names when it is one of this family's, else None."""
    arch = raw.get("architecture")
    return arch if arch in ARCHITECTURES else None


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
        m, kind = l["mixer"], l["type"]
        if kind in ("delta", "channel_delta"):
            ch = kind == "channel_delta"
            mixer = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), ch,
                              rank(f"l{i}.mix.a1") if ch else 0, rank(f"l{i}.mix.g1") if ch else 0)
        elif kind == "latent_attention":
            mask = m.get("mask")
            mixer = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]),
                               float(m["scale"]), int(mask["size"]) if mask else 0)
            if mask and mixer.window < 1:
                raise LayeredConfigError("an attention window holds at least the token itself")
        else:
            raise LayeredConfigError(f"layer {i}: unknown mixer {kind!r}")
        mlp = l.get("mlp")
        if mlp and mlp.get("kind") != "dense":
            raise LayeredConfigError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        layers.append(LayerSpec(mixer, int(mlp["ff"]) if mlp else 0))
    loop = raw.get("loop")
    cfg = LayeredConfig(name or arch, int(raw["vocab"]), int(raw["width"]), tuple(layers), float(raw["norm"]["eps"]),
                        (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None, architecture=arch)
    cfg.validate()
    return cfg


# ------------------------------------------------------------------ tensor inventory
def tensor_shapes(cfg: LayeredConfig) -> dict[str, tuple[int, ...]]:
    """Every tensor of a checkpoint of this configuration."""
    W = cfg.hidden_size
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab_size, W), "embed.norm": (W,), "final.norm": (W,),
                                       "head": (cfg.vocab_size, W)}
    if cfg.loop is not None:
        out["loop.in"] = (W, 2 * W)
    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"l{i}.mix"
        out[f"l{i}.norm1"] = (W,)
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
        else:
            out.update({f"{p}.dq": (m.q_rank, W), f"{p}.dq.norm": (m.q_rank,), f"{p}.uq": (m.heads * m.dim, m.q_rank),
                        f"{p}.dkv": (m.kv_rank, W), f"{p}.dkv.norm": (m.kv_rank,), f"{p}.uk": (m.heads * m.dim, m.kv_rank),
                        f"{p}.uv": (m.heads * m.vdim, m.kv_rank), f"{p}.g": (m.heads, W)})
        out[f"{p}.o"] = (W, m.out_width)
        if l.ff:
            out[f"l{i}.mlp.up"] = (l.ff, W)
            out[f"l{i}.mlp.down"] = (W, l.ff)
    return out


def check_inventory(cfg: LayeredConfig, shapes: dict[str, tuple[int, ...]]) -> None:
    """The checkpoint's tensors are exactly the configuration's."""
    want = tensor_shapes(cfg)
    for n, s in want.items():
        if n not in shapes:
            raise LayeredConfigError(f"missing tensor {n}")
        if tuple(shapes[n]) != s:
            raise LayeredConfigError(f"{n}: shape {tuple(shapes[n])}, expected {s}")
    extra = sorted(set(shapes) - set(want))
    if extra:
        raise LayeredConfigError(f"checkpoint has {len(extra)} tensors this configuration does not own, e.g. {extra[:3]}")


def random_tensors(cfg: LayeredConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights with the magnitudes of a trained model: unit-variance activations through every product."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for n, s in tensor_shapes(cfg).items():
        z = torch.randn(s, generator=g, device=device)
        if n.endswith((".dq.norm", ".dkv.norm", ".mix.norm")):
            t = 1.0 + 0.1 * z                    # plain norm weights
        elif n.endswith("norm") or n.endswith("norm1"):
            t = 0.1 * z                          # stored around zero
        elif n.endswith(".A_log"):
            t = 0.5 * z - 2.0
        elif n.endswith(".dt_bias"):
            t = 0.5 * z
        elif n.endswith(".conv"):
            t = z / math.sqrt(s[1])
        elif n == "embed":
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
    q_norm: torch.Tensor
    c_norm: torch.Tensor
    uq: wq_pack.PackedWeight         # rows in the column layout of ``absorb``'s input
    absorb: BlockDiagonal            # queries -> latent space
    value: BlockDiagonal             # latent outputs -> head outputs
    c_off: int
    g_off: int


@dataclass
class LayerWeights:
    norm: torch.Tensor               # fp32 factor 1 + w
    proj: wq_pack.PackedWeight       # [mixer inputs | feed-forward up]
    split: int                       # mixer columns
    ff: int
    mixer: object                    # DeltaWeights | LatentWeights
    out: wq_pack.PackedWeight        # [o | down]
    out_off: int                     # first feed-forward column of ``out``'s input


@dataclass
class LayeredWeights:
    embed: torch.Tensor
    embed_norm: torch.Tensor
    loop_in: wq_pack.PackedWeight | None
    layers: list[LayerWeights]
    final_norm: torch.Tensor
    lm_head: wq_pack.PackedWeight
    vocab_start: int = 0

    def nbytes(self) -> int:
        total = self.embed.numel() * 2 + self.lm_head.nbytes + (self.loop_in.nbytes if self.loop_in else 0)
        for l in self.layers:
            total += l.proj.nbytes + l.out.nbytes
            m = l.mixer
            if isinstance(m, LatentWeights):
                total += m.uq.nbytes + m.absorb.w.nbytes + m.value.w.nbytes
            elif m.low is not None:
                total += m.low.nbytes
        return total


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


def pack_layer(cfg: LayeredConfig, i: int, get) -> LayerWeights:
    """``get(name)`` -> tensor on the target device."""
    l, p = cfg.layers[i], f"l{i}.mix"
    W, m = cfg.hidden_size, l.mixer

    def f32(n):
        return get(n).float().contiguous()

    rows = _Rows(W)
    if isinstance(m, DeltaSpec):
        rows.add(get(f"{p}.q"), get(f"{p}.k"), get(f"{p}.v"))
        b_off = rows.add(get(f"{p}.b"))
        conv = torch.cat([get(f"{p}.{t}.conv") for t in "qkv"]).float()
        conv_w = torch.zeros(m.conv, m.conv_width, device=conv.device)
        conv_w[:, :m.channels] = conv.t()
        common = dict(spec=m, conv_w=conv_w.contiguous(), a_log=f32(f"{p}.A_log"), dt_bias=f32(f"{p}.dt_bias"),
                      norm_w=f32(f"{p}.norm"), b_off=b_off)
        if m.per_channel:
            inner = round_up(m.decay_rank + m.gate_rank, 64)
            a_off = rows.add(get(f"{p}.a1"), get(f"{p}.g1"), align=64, size=inner)
            low_z = round_up(m.heads * m.dim, 8)
            low = torch.zeros(low_z + m.heads * m.vdim, inner, dtype=torch.bfloat16, device=conv.device)
            low[:m.heads * m.dim, :m.decay_rank] = get(f"{p}.a2")
            low[low_z:, m.decay_rank:m.decay_rank + m.gate_rank] = get(f"{p}.g2")
            mixer = DeltaWeights(**common, a_off=a_off, z_off=0, low=wq_pack.pack_bf16(low), low_z=low_z)
        else:
            a_off = rows.add(get(f"{p}.a"))
            z_off = rows.add(get(f"{p}.g"))
            mixer = DeltaWeights(**common, a_off=a_off, z_off=z_off)
    else:
        H, d, e, R, Rp = m.heads, m.dim, m.vdim, m.kv_rank, m.rank_padded
        rows.add(get(f"{p}.dq"))
        c_off = rows.add(get(f"{p}.dkv"))
        g_off = rows.add(get(f"{p}.g"))
        uk = torch.zeros(H, Rp, d, dtype=torch.bfloat16, device=get(f"{p}.uk").device)
        uk[:, :R] = get(f"{p}.uk").view(H, d, R).transpose(1, 2)
        absorb = BlockDiagonal.pack(uk)
        uv = torch.zeros(H, e, Rp, dtype=torch.bfloat16, device=uk.device)
        uv[:, :, :R] = get(f"{p}.uv").view(H, e, R)
        # the query projection writes every head where its block of ``absorb`` reads it
        hp, kg = absorb.heads, absorb.w.k
        uq = torch.zeros(-(-H // hp) * kg, m.q_rank, dtype=torch.bfloat16, device=uk.device)
        src = get(f"{p}.uq").view(H, d, m.q_rank)
        for h in range(H):
            c = (h // hp) * kg + (h % hp) * d
            uq[c:c + d] = src[h]
        mixer = LatentWeights(m, f32(f"{p}.dq.norm"), f32(f"{p}.dkv.norm"), _matrix(uq), absorb, BlockDiagonal.pack(uv),
                              c_off, g_off)
    mixer_rows = rows.end()
    split = mixer_rows.shape[0]
    out_off = round_up(m.out_width, 8)
    out = torch.zeros(W, round_up(out_off + l.ff, 64), dtype=torch.bfloat16, device=mixer_rows.device)
    out[:, :m.out_width] = get(f"{p}.o")
    if l.ff:
        mixer_rows = torch.cat([mixer_rows, get(f"l{i}.mlp.up").to(torch.bfloat16)])
        out[:, out_off:out_off + l.ff] = get(f"l{i}.mlp.down")
    return LayerWeights(1.0 + f32(f"l{i}.norm1"), _matrix(mixer_rows), split, l.ff, mixer, wq_pack.pack_bf16(out), out_off)


def pack_weights(cfg: LayeredConfig, get) -> LayeredWeights:
    return LayeredWeights(
        embed=get("embed").to(torch.bfloat16).contiguous(), embed_norm=1.0 + get("embed.norm").float(),
        loop_in=_matrix(get("loop.in")) if cfg.loop is not None else None,
        layers=[pack_layer(cfg, i, get) for i in range(cfg.num_layers)],
        final_norm=1.0 + get("final.norm").float(), lm_head=_matrix(get("head")))


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


NAMED = {"layered-tiny": tiny_layered_config, "layered-8b": layered_8b_config}


def with_dtype(cfg: LayeredConfig, dtype: str) -> LayeredConfig:
    return replace(cfg, dtype=dtype)
