"""Tensor-level wrappers over the native sm_100a kernels.

Every wrapper takes CUDA tensors, launches on the current stream and raises
``NativeLibraryError`` on a non-zero launch code.  There is deliberately no
PyTorch fallback on the GPU path: a missing library is an error.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import native
from .wq_pack import FMT_BF16, FMT_CUBIC4, FMT_FP8, FMT_FP8_BLOCK, PackedWeight

PAGE_TOKENS = 16


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


class Workspace:
    """Per-device scratch shared by split-K GEMMs and split-KV attention.

    ``counters`` must stay zero between launches (the kernels restore it);
    ``status`` collects device-side error codes and is polled by ``check_status``.
    """

    def __init__(self, device: torch.device, gemm_bytes: int = 64 << 20, attn_floats: int = 4 << 20,
                 counters: int = 1 << 16) -> None:
        self.device = device
        self.gemm = torch.empty(gemm_bytes, dtype=torch.uint8, device=device)
        self.attn = torch.empty(max(attn_floats, 1), dtype=torch.float32, device=device)
        self.gemm_counters = torch.zeros(counters, dtype=torch.int32, device=device)
        self.attn_counters = torch.zeros(counters, dtype=torch.int32, device=device)
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self._retired: list[torch.Tensor] = []
        # e4m3 activation operand of the fp8 GEMMs (codes and per-token scales), grown on demand
        self.fp8_q = torch.empty(0, dtype=torch.uint8, device=device)
        self.fp8_scale = torch.empty(0, dtype=torch.float32, device=device)

    def ensure_fp8(self, rows: int, k: int) -> None:
        if rows * k > self.fp8_q.numel():
            self._retired.append(self.fp8_q)          # captured graphs may hold the old address: retire, never free
            self.fp8_q = torch.empty(max(rows * k, 256 * 16384), dtype=torch.uint8, device=self.device)
        if rows > self.fp8_scale.numel():
            self._retired.append(self.fp8_scale)
            self.fp8_scale = torch.empty(max(rows, 8192), dtype=torch.float32, device=self.device)

    def ensure_attn(self, floats: int) -> None:
        if floats > self.attn.numel():
            # captured graphs may hold the old address: retire, never free
            self._retired.append(self.attn)
            self.attn = torch.empty(floats, dtype=torch.float32, device=self.device)

    def check_status(self) -> None:
        code = int(self.status.item())
        if code:
            self.status.zero_()
            raise native.NativeLibraryError(f"device kernel reported status {code} (bounded wait ran out)")


_workspaces: dict[int, Workspace] = {}


def workspace(device: torch.device) -> Workspace:
    idx = device.index if device.index is not None else torch.cuda.current_device()
    ws = _workspaces.get(idx)
    if ws is None:
        ws = _workspaces[idx] = Workspace(torch.device("cuda", idx))
    return ws


def sm_count(device: torch.device) -> int:
    return torch.cuda.get_device_properties(device).multi_processor_count


_CLUSTER_CAPACITY_GUESS = {2: 72, 3: 40, 4: 32, 5: 24, 6: 16, 7: 16, 8: 16}      # 8 GPCs of 16-18 usable SMs
_cluster_capacity: dict[tuple[int, int], int] = {}


def resident_clusters(fmt: int, size: int) -> int:
    """Clusters of ``size`` K splits of the per-tile GEMM that fit on the device at once (its CTAs share a GPC)."""
    key = (fmt, size)
    if key not in _cluster_capacity:
        n = 0
        if torch.cuda.is_available():
            n = native.lib().cb_wq_gemm_resident_clusters(fmt, size)
        _cluster_capacity[key] = n if n > 0 else _CLUSTER_CAPACITY_GUESS.get(size, 0)
    return _cluster_capacity[key]


# Measured launch plans (``ops/autotune.py``): "fmt:m:n:k:act" -> (use the persistent kernel, split-K factor of the
# per-tile kernel).  Consulted before the rules below when the caller forces nothing; empty unless a plan was installed.
TUNED_PLANS: dict[str, tuple[bool, int]] = {}


def choose_splits(m: int, n: int, k: int, sms: int = 148, fmt: int = FMT_CUBIC4, cluster: bool = True) -> int:
    """Split-K factor: fill the SMs when the (n-tile x m-tile) grid is small.

    The splits of a tile form a thread-block cluster and sum their partial tiles through distributed shared
    memory; that only works when all clusters of the launch are resident at once, so the largest factor whose
    clusters fit is taken (48 tiles: 2, because only ~40 clusters of 3 fit on 8 GPCs).  ``cluster`` False (partials
    through the workspace, the last split sums them) keeps the plain rule.  A split pays off while each CTA still
    has >= 8 k-blocks of work.
    """
    from .strategies import active
    g = active().gemm
    n_tiles = -(-n // 128)
    m_tiles = -(-m // 256)
    tiles = n_tiles * m_tiles
    k_blocks = k // 64
    if tiles * 2 > sms or k_blocks < 2 * g.split_k_min_blocks:
        return 1
    base = max(1, min(sms // tiles, k_blocks // g.split_k_min_blocks, g.split_k_max))
    if cluster:
        for s in range(min(base, 8), 1, -1):
            if tiles <= resident_clusters(fmt, s):
                return s
    return base


def use_stream_k(m: int, n: int, fmt: int, sms: int = 148, k: int = 4096) -> bool:
    """Which GEMM kernel serves a shape when the caller does not say.

    Measured on a B200 inside CUDA graphs (cubic4, K = 4096): the persistent stream-K kernel wins when there are
    more weight tiles than SMs, because it removes the second, partly empty wave: N = 24576 runs 69 -> 45 us at
    16-64 batch rows, 70 -> 54 us at 128 and 80 -> 69 us at 256 (the fix-up of a streamed tile is deferred to the
    end of its CTA and done by 640 threads), and the bf16 lm_head is 5 % faster.  With fewer tiles than SMs its
    fixed costs (start-up, fp32 partial tiles summed by the last CTA) make it 10-25 % slower than one CTA per
    (tile, split).  Above 256 rows (prefill chunks, several row tiles) the persistent kernel runs on CTA pairs
    (cta_group::2, half an activation tile per SM): 4096 x 24576 x 4096 takes 700 us against 778 us, 4096 x 4096 x
    12288 342 against 425; it is chosen when every pair gets enough k-blocks to amortise its start-up
    (512 x 6144 x 4096, 41 k-blocks per pair, is 48 us against 41 us on the per-tile kernel).
    The thresholds live in the operator configuration (``ops/strategies.py``).
    """
    from .strategies import active
    g = active().gemm
    n_tiles = -(-n // 128)
    m_tiles = -(-m // 256)
    if m > max(g.stream_k_max_rows, 256) and fmt != FMT_BF16:
        pairs = sms // 2
        return (g.cta_pairs and n_tiles % 2 == 0 and pairs > 0
                and (n_tiles // 2) * m_tiles * (k // 64) >= g.pair_min_blocks * pairs)
    if n_tiles * m_tiles <= g.stream_k_min_tile_ratio * sms:
        return False
    return m <= g.stream_k_max_rows or (fmt == FMT_BF16 and g.stream_k_bf16)


@dataclass
class Fp8Act:
    """Activations quantized per token for the fp8 GEMMs: e4m3 bytes ``q [M, K]`` and fp32 scales ``scale [M]``."""
    q: torch.Tensor
    scale: torch.Tensor

    @property
    def shape(self):
        return self.q.shape

    @property
    def device(self):
        return self.q.device


def fp8_quantize(x: torch.Tensor, ws: Workspace | None = None, out: Fp8Act | None = None, scale_max=None) -> Fp8Act:
    """Dynamic per-token e4m3 quantization of ``x [M, K]`` (bf16): ``scale = max(amax / 448, 1 / (448 * 512))``,
    ``q = e4m3(x / scale)`` (the reference's rule, ``quantization/extensions/fp8/reference.py:47-59`` there).  Without
    ``out`` the result lives in the workspace's fp8 buffers until the next quantization.

    ``scale_max``: a callable that reduces the fp32 scale vector in place with MAX over the tensor-parallel ranks; given
    for operands whose K dimension is sharded, so that every rank quantizes with the scale of the whole row."""
    m, k = x.shape
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1
    if out is None:
        ws = ws or workspace(x.device)
        ws.ensure_fp8(m, k)
        out = Fp8Act(ws.fp8_q[:m * k].view(m, k), ws.fp8_scale[:m])
    if scale_max is not None:
        for phase in (1, 2):
            code = native.lib().cb_fp8_quantize_rows_phase(x.data_ptr(), x.stride(0), out.q.data_ptr(), out.q.stride(0),
                                                           out.scale.data_ptr(), m, k, phase, _stream())
            native.check(code, "cb_fp8_quantize_rows_phase")
            if phase == 1:
                scale_max(out.scale)
        return out
    code = native.lib().cb_fp8_quantize_rows(x.data_ptr(), x.stride(0), out.q.data_ptr(), out.q.stride(0),
                                             out.scale.data_ptr(), m, k, _stream())
    native.check(code, "cb_fp8_quantize_rows")
    return out


def rmsnorm_fp8(x: torch.Tensor, weight: torch.Tensor, eps: float, residual: torch.Tensor | None = None,
                zero_centered: bool = False, ws: Workspace | None = None) -> Fp8Act:
    """RMSNorm whose output leaves as e4m3 + per-token scales (the bf16-rounded norm output is what gets quantized,
    so the result equals ``fp8_quantize(rmsnorm(...))``)."""
    m, h = x.shape
    ws = ws or workspace(x.device)
    ws.ensure_fp8(m, h)
    out = Fp8Act(ws.fp8_q[:m * h].view(m, h), ws.fp8_scale[:m])
    code = native.lib().cb_rmsnorm_fp8(x.data_ptr(), _ptr(residual), _ptr(residual), weight.data_ptr(), out.q.data_ptr(), h,
                                       out.scale.data_ptr(), m, h, float(eps), int(zero_centered), _stream())
    native.check(code, "cb_rmsnorm_fp8")
    return out


def swiglu_fp8(gate_up: torch.Tensor, ws: Workspace | None = None) -> Fp8Act:
    """SwiGLU of ``[gate | up]`` whose output leaves as e4m3 + per-token scales."""
    m, two_i = gate_up.shape
    i = two_i // 2
    ws = ws or workspace(gate_up.device)
    ws.ensure_fp8(m, i)
    out = Fp8Act(ws.fp8_q[:m * i].view(m, i), ws.fp8_scale[:m])
    code = native.lib().cb_swiglu_fp8(gate_up.data_ptr(), out.q.data_ptr(), i, out.scale.data_ptr(), m, i, _stream())
    native.check(code, "cb_swiglu_fp8")
    return out


def _wq_gemm_fp8(x, w: PackedWeight, out, residual, splits, ws: Workspace, link, swiglu: bool,
                 min_units: int | None = None) -> torch.Tensor:
    """The fp8 branch of ``wq_gemm`` / ``wq_gemm_act``: quantize the activations per token unless the caller already
    holds them as ``Fp8Act``, then e4m3 x e4m3 on the tensor cores with both scales applied in the epilogue."""
    if link is not None and (link.mode & 1) and not isinstance(x, Fp8Act):
        raise ValueError("an fp8 GEMM cannot wait for gathered rows: its quantizer would read them before they arrive")
    a = x if isinstance(x, Fp8Act) else fp8_quantize(x, ws)
    m, k = a.q.shape
    push = link is not None and (link.mode & 2)
    l = native.lib()
    # the persistent kernel (stream-K at decode sizes with more tiles than SMs, CTA pairs above 256 rows) serves row
    # scales; block scales and explicit split factors stay on the per-tile kernel
    # (measured: the fp8 loop is bound by the L2 -> SM operand feed in both kernels; CTA pairs pay off for deep K at
    # prefill sizes -- 4096 x 4096 x 12288: 153 us against 176 us -- and nowhere else, stream-K at decode sizes ties)
    stream_k = (splits is None and w.fmt == FMT_FP8 and link is None
                and (min_units is not None or (m >= 2048 and k >= 8192 and (-(-w.n // 128)) % 2 == 0)))
    if stream_k and min_units is None:
        from .strategies import active
        min_units = active().gemm.stream_k_min_units
    min_units = min_units or 0
    if not stream_k:
        if splits is None:
            splits = choose_splits(m, w.n, k, fmt=w.fmt)
        if splits > 1 and l.cb_wq_gemm_workspace_bytes(m, w.n, splits) > ws.gemm.numel():
            splits = 1
    code = l.cb_wq_gemm_fp8(a.q.data_ptr(), a.q.stride(0), a.scale.data_ptr(), w.codes.data_ptr(), w.meta.data_ptr(),
                            int(w.fmt == FMT_FP8_BLOCK), None if push else out.data_ptr(), w.n if push else out.stride(0),
                            _ptr(residual), m, w.n, k, int(splits or 1), int(swiglu), int(stream_k), int(min_units),
                            ws.gemm.data_ptr(), ws.gemm.numel(), ws.gemm_counters.data_ptr(), ws.status.data_ptr(),
                            _stream(), None if link is None else ctypes.byref(link))
    native.check(code, "cb_wq_gemm_fp8")
    return out


def wq_gemm(x: torch.Tensor, w: PackedWeight, out: torch.Tensor | None = None,
            residual: torch.Tensor | None = None, splits: int | None = None,
            ws: Workspace | None = None, link=None, min_units: int | None = None) -> torch.Tensor:
    """``out[M, N] = x[M, K] @ W[N, K]^T * alpha (+ residual)`` with W in packed form.

    Two kernels: one CTA per (weight tile, K split) (``csrc/wq_gemm.cu``) and the persistent stream-K kernel
    (``csrc/wq_gemm_sk.cu``).  With neither ``splits`` nor ``min_units`` given the faster one for the shape is
    used (``use_stream_k``).  ``splits`` forces the first with that split-K factor; ``min_units`` forces the
    second (0 = its own schedule, > 0 = the smallest run of k-blocks a CTA is dealt).
    """
    assert isinstance(x, Fp8Act) or (x.dtype == torch.bfloat16 and x.dim() == 2 and x.stride(1) == 1)
    m, k = x.shape
    assert k == w.k, (k, w.k)
    push = link is not None and (link.mode & 2)
    if out is None and not push:
        out = torch.empty((m, w.n), dtype=torch.bfloat16, device=x.device)
    assert push or (out.stride(1) == 1 and out.shape == (m, w.n))
    if residual is not None:
        assert residual.shape == out.shape and residual.stride(0) == out.stride(0)
    ws = ws or workspace(x.device)
    if w.fmt in (FMT_FP8, FMT_FP8_BLOCK):
        return _wq_gemm_fp8(x, w, out, residual, splits, ws, link, False, min_units)
    l = native.lib()
    if splits is None and min_units is None and link is None and TUNED_PLANS:
        tuned = TUNED_PLANS.get(f"{w.fmt}:{m}:{w.n}:{k}:0")
        if tuned is not None:
            splits, min_units = (None, 0) if tuned[0] else (tuned[1], None)
    if splits is None and min_units is None and use_stream_k(m, w.n, w.fmt, sm_count(x.device), k):
        from .strategies import active
        min_units = active().gemm.stream_k_min_units
    if splits is None and min_units is not None:
        code = l.cb_wq_gemm_sk(w.fmt, x.data_ptr(), x.stride(0), w.codes.data_ptr(), _ptr(w.meta),
                               None if push else out.data_ptr(), w.n if push else out.stride(0), _ptr(residual),
                               float(w.alpha), m, w.n, k, w.group_k, int(min_units), ws.gemm.data_ptr(),
                               ws.gemm.numel(), ws.gemm_counters.data_ptr(), ws.status.data_ptr(), _stream(),
                               None if link is None else ctypes.byref(link))
        native.check(code, "cb_wq_gemm_sk")
        return out
    if splits is None:
        splits = choose_splits(m, w.n, k, fmt=w.fmt)
    if splits > 1:
        need = l.cb_wq_gemm_workspace_bytes(m, w.n, splits)
        if need > ws.gemm.numel():
            splits = 1
    code = l.cb_wq_gemm_tp(w.fmt, x.data_ptr(), x.stride(0), w.codes.data_ptr(), _ptr(w.meta),
                           None if push else out.data_ptr(), w.n if push else out.stride(0), _ptr(residual),
                           float(w.alpha), m, w.n, k, w.group_k, splits, ws.gemm.data_ptr(),
                           ws.gemm_counters.data_ptr(), ws.status.data_ptr(), _stream(),
                           None if link is None else ctypes.byref(link))
    native.check(code, "cb_wq_gemm")
    return out


def wq_gemm_act(x: torch.Tensor, w: PackedWeight, out: torch.Tensor | None = None, splits: int | None = None,
                ws: Workspace | None = None, min_units: int | None = None, link=None) -> torch.Tensor:
    """Gate/up projection with SwiGLU in the GEMM epilogue: ``out[M, N/2] = silu(x Wg^T) * (x Wu^T)``.

    ``w`` is the ``[gate; up]`` matrix in the interleaved row order (``wq_pack.swiglu_interleave``).  The projection
    ``link`` (gather-wait only) as in ``wq_gemm``.  The projection is rounded to bf16 before the activation, as when ``wq_gemm`` and ``swiglu`` run as two kernels, so both paths
    give the same values; the ``[M, N]`` intermediate is never written.  Kernel choice as in ``wq_gemm``.
    """
    assert w.act_interleaved, "weight rows are not in the SwiGLU order"
    assert isinstance(x, Fp8Act) or (x.dtype == torch.bfloat16 and x.dim() == 2 and x.stride(1) == 1)
    m, k = x.shape
    assert k == w.k, (k, w.k)
    if out is None:
        out = torch.empty((m, w.n // 2), dtype=torch.bfloat16, device=x.device)
    assert out.stride(1) == 1 and out.shape == (m, w.n // 2)
    ws = ws or workspace(x.device)
    if w.fmt in (FMT_FP8, FMT_FP8_BLOCK):
        return _wq_gemm_fp8(x, w, out, None, splits, ws, link, True, min_units)
    l = native.lib()
    if splits is None and min_units is None and link is None and TUNED_PLANS:
        tuned = TUNED_PLANS.get(f"{w.fmt}:{m}:{w.n}:{k}:1")
        if tuned is not None:
            splits, min_units = (None, 0) if tuned[0] else (tuned[1], None)
    stream_k = splits is None and (min_units is not None or use_stream_k(m, w.n, w.fmt, sm_count(x.device), k))
    if stream_k and min_units is None:
        from .strategies import active
        min_units = active().gemm.stream_k_min_units
    if not stream_k:
        if splits is None:
            splits = choose_splits(m, w.n, k, fmt=w.fmt)
        if splits > 1 and l.cb_wq_gemm_workspace_bytes(m, w.n, splits) > ws.gemm.numel():
            splits = 1
    code = l.cb_wq_gemm_act(w.fmt, x.data_ptr(), x.stride(0), w.codes.data_ptr(), _ptr(w.meta), out.data_ptr(),
                            out.stride(0), float(w.alpha), m, w.n, k, w.group_k, int(stream_k), int(splits or 1),
                            int(min_units or 0), ws.gemm.data_ptr(), ws.gemm.numel(), ws.gemm_counters.data_ptr(),
                            ws.status.data_ptr(), _stream(), None if link is None else ctypes.byref(link))
    native.check(code, "cb_wq_gemm_act")
    return out


def gate_up_act(x: torch.Tensor, w: PackedWeight, gu: torch.Tensor, act: torch.Tensor, ws: Workspace | None = None,
                link=None) -> int:
    """``act = swiglu(x @ W^T)`` for a ``[gate; up]`` projection: one launch when the rows of ``w`` are interleaved
    for the fused epilogue, else the GEMM into ``gu`` followed by the activation kernel.  Returns the launch count."""
    if w.act_interleaved:
        wq_gemm_act(x, w, out=act, ws=ws, link=link)
        return 1
    wq_gemm(x, w, out=gu, ws=ws, link=link)
    swiglu(gu, out=act)
    return 2


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor | None = None,
            residual: torch.Tensor | None = None, zero_centered: bool = False) -> torch.Tensor:
    """RMSNorm; with ``residual`` the sum ``x + residual`` is written back into ``residual`` first."""
    rows, h = x.shape
    if out is None:
        out = torch.empty_like(x)
    code = native.lib().cb_rmsnorm(x.data_ptr(), _ptr(residual), _ptr(residual), weight.data_ptr(), out.data_ptr(),
                                   rows, h, float(eps), int(zero_centered), _stream())
    native.check(code, "cb_rmsnorm")
    return out


def rmsnorm_rows(x: torch.Tensor, rows: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor | None = None,
                 zero_centered: bool = False) -> torch.Tensor:
    """``out[i] = rmsnorm(x[rows[i]])`` (``rows`` int64): the final norm over the rows whose logits are wanted, with the
    row gather done by the kernel's own loads."""
    assert rows.dtype == torch.int64 and x.stride(1) == 1 and x.stride(0) == x.shape[1]
    n, h = rows.numel(), x.shape[1]
    if out is None:
        out = torch.empty((n, h), dtype=x.dtype, device=x.device)
    code = native.lib().cb_rmsnorm_rows(x.data_ptr(), rows.data_ptr(), weight.data_ptr(), out.data_ptr(), n, h,
                                        float(eps), int(zero_centered), _stream())
    native.check(code, "cb_rmsnorm_rows")
    return out


def swiglu(gate_up: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    rows, two_i = gate_up.shape
    i = two_i // 2
    if out is None:
        out = torch.empty((rows, i), dtype=gate_up.dtype, device=gate_up.device)
    native.check(native.lib().cb_swiglu(gate_up.data_ptr(), out.data_ptr(), rows, i, _stream()), "cb_swiglu")
    return out


def embedding(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None, vocab_start: int = 0) -> torch.Tensor:
    t = ids.numel()
    h = table.shape[1]
    if out is None:
        out = torch.empty((t, h), dtype=table.dtype, device=table.device)
    code = native.lib().cb_embedding(ids.data_ptr(), table.data_ptr(), out.data_ptr(), t, h, vocab_start,
                                     table.shape[0], _stream())
    native.check(code, "cb_embedding")
    return out


def kv_blob_bytes(head_dim: int, k_bits: int, v_bits: int) -> int:
    d = head_dim
    scale = PAGE_TOKENS * (d // 32) * 4
    return PAGE_TOKENS * d * k_bits // 8 + PAGE_TOKENS * d * v_bits // 8 + 2 * scale


def rope_kv_write(qkv: torch.Tensor, q_out: torch.Tensor, cache: torch.Tensor, positions: torch.Tensor,
                  slots: torch.Tensor, inv_freq: torch.Tensor, hq: int, hkv: int, head_dim: int,
                  k_bits: int, v_bits: int, q_norm: torch.Tensor | None = None,
                  k_norm: torch.Tensor | None = None, eps: float = 1e-6, rotary_dim: int | None = None,
                  rotate: bool = False, positions_hw: tuple[torch.Tensor, torch.Tensor] | None = None,
                  mrope_section: tuple[int, int, int] | None = None, qkv_bias: torch.Tensor | None = None) -> None:
    """``rotate``: every q / k / v head vector is Walsh-Hadamard transformed (after RoPE) before it is written, which
    spreads outlier channels over the 32-channel quantization groups; ``q . k`` is unchanged and the attention
    output is transformed back with ``hadamard`` (reference: ``ops/cuda/cache_rotation_native.cu:12``).
    ``positions_hw``: int32 row- and column-axis positions ``[T]`` each; with them ``positions`` is the temporal axis
    and ``mrope_section`` says how many frequency slots follow each axis (interleaved layout; reference:
    ``ops/cuda/position/qwen_mrope.py:25``).  ``qkv_bias``: bf16 ``[(hq + 2 hkv) head_dim]`` added to the rows as they
    are read (projection biases of the Qwen2 family)."""
    t = qkv.shape[0]
    rot = head_dim if rotary_dim is None else rotary_dim
    if qkv_bias is not None:
        assert qkv_bias.dtype == torch.bfloat16 and qkv_bias.numel() == (hq + 2 * hkv) * head_dim and qkv_bias.is_contiguous()
    if positions_hw is None and qkv_bias is None:
        code = native.lib().cb_rope_kv_write(qkv.data_ptr(), q_out.data_ptr(), cache.data_ptr(), positions.data_ptr(),
                                             slots.data_ptr(), _ptr(q_norm), _ptr(k_norm), inv_freq.data_ptr(), t, hq,
                                             hkv, head_dim, rot, float(eps), k_bits, v_bits, int(rotate), _stream())
        native.check(code, "cb_rope_kv_write")
        return
    ph = pw = None
    sec = (0, 0, 0)
    if positions_hw is not None:
        if mrope_section is None or sum(mrope_section) != rot // 2:
            raise ValueError("three-axis positions need the section counts of the rotary width")
        ph, pw = positions_hw
        sec = mrope_section
        assert ph.dtype == pw.dtype == torch.int32 and ph.numel() >= t and pw.numel() >= t
    code = native.lib().cb_rope_kv_write_axes(qkv.data_ptr(), q_out.data_ptr(), cache.data_ptr(), positions.data_ptr(),
                                              _ptr(ph), _ptr(pw), int(sec[1]), int(sec[2]), _ptr(qkv_bias),
                                              slots.data_ptr(), _ptr(q_norm), _ptr(k_norm), inv_freq.data_ptr(), t, hq,
                                              hkv, head_dim, rot, float(eps), k_bits, v_bits, int(rotate), _stream())
    native.check(code, "cb_rope_kv_write_axes")


def hadamard(x: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """Normalised Walsh-Hadamard transform of every consecutive 128-vector of the rows of ``x`` (bf16; its own inverse)."""
    rows, cols = x.shape
    assert cols % 128 == 0 and x.stride(1) == 1 and x.dtype == torch.bfloat16
    out = x if out is None else out
    native.check(native.lib().cb_hadamard(x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), cols // 128, rows,
                                          _stream()), "cb_hadamard")
    return out


def copy_pages(cache: torch.Tensor, src: torch.Tensor, dst: torch.Tensor) -> None:
    page_bytes = cache.stride(0) * cache.element_size()
    native.check(native.lib().cb_copy_pages(cache.data_ptr(), src.data_ptr(), dst.data_ptr(), src.numel(),
                                            page_bytes, _stream()), "cb_copy_pages")


def copy_rows(t: torch.Tensor, src: torch.Tensor, dst: torch.Tensor) -> None:
    """``t[dst[i]] = t[src[i]]`` for whole leading-axis rows of a contiguous tensor (bit-preserving; the page-copy
    kernel with a row as the page).  A row must be a multiple of 16 bytes."""
    if not t.is_contiguous() or (t.stride(0) * t.element_size()) % 16:
        raise ValueError("copy_rows: rows must be contiguous multiples of 16 bytes")
    copy_pages(t, src, dst)


def paged_attention(q: torch.Tensor, out: torch.Tensor, cache: torch.Tensor, page_table: torch.Tensor,
                    rb_req: torch.Tensor, rb_qstart: torch.Tensor, rb_qcount: torch.Tensor, rb_ctx: torch.Tensor,
                    hq: int, hkv: int, head_dim: int, k_bits: int, v_bits: int, scale: float | None = None,
                    splits: int = 1, ws: Workspace | None = None) -> torch.Tensor:
    """Attention of row blocks over the paged quantized cache (see ``csrc/paged_attn.cu``)."""
    rbs = rb_req.numel()
    ws = ws or workspace(q.device)
    l = native.lib()
    if splits > 1:
        ws.ensure_attn(l.cb_paged_attn_partial_floats(rbs, hkv, splits))
        assert rbs * hkv <= ws.attn_counters.numel()
    code = l.cb_paged_attn(q.data_ptr(), out.data_ptr(), cache.data_ptr(), page_table.data_ptr(), rb_req.data_ptr(),
                           rb_qstart.data_ptr(), rb_qcount.data_ptr(), rb_ctx.data_ptr(), rbs, hq, hkv, head_dim,
                           page_table.shape[1], k_bits, v_bits,
                           float(scale if scale is not None else 1.0 / math.sqrt(head_dim)), splits,
                           ws.attn.data_ptr(), ws.attn_counters.data_ptr(), ws.status.data_ptr(), _stream())
    native.check(code, "cb_paged_attn")
    return out


def sample(logits: torch.Tensor, out_ids: torch.Tensor, temperature: torch.Tensor | None = None,
           top_p: torch.Tensor | None = None, top_k: torch.Tensor | None = None,
           seeds: torch.Tensor | None = None, counters: torch.Tensor | None = None,
           mask: torch.Tensor | None = None, out_logprob: torch.Tensor | None = None,
           vocab: int | None = None, out_value: torch.Tensor | None = None, id_offset: int = 0) -> torch.Tensor:
    rows = logits.shape[0]
    code = native.lib().cb_sample(logits.data_ptr(), int(logits.dtype == torch.float32), logits.stride(0), _ptr(mask),
                                  0 if mask is None else mask.stride(0), _ptr(temperature), _ptr(top_p), _ptr(top_k),
                                  _ptr(seeds), _ptr(counters), out_ids.data_ptr(), _ptr(out_logprob),
                                  _ptr(out_value), int(id_offset), rows, vocab or logits.shape[1], _stream())
    native.check(code, "cb_sample")
    return out_ids


SAMPLE_CANDIDATES = 20      # candidate slots per row of vocab-sharded sampling (= the largest top-k)


def sample_candidates(logits: torch.Tensor, cand_val: torch.Tensor, cand_id: torch.Tensor,
                      temperature: torch.Tensor | None = None, top_k: torch.Tensor | None = None,
                      mask: torch.Tensor | None = None, vocab: int | None = None, id_offset: int = 0) -> None:
    """Rank-local half of vocab-sharded sampling: the best (logit, global id) pairs of every row, ``[rows, 20]``."""
    rows = logits.shape[0]
    code = native.lib().cb_sample_candidates(logits.data_ptr(), logits.stride(0), _ptr(mask),
                                             0 if mask is None else mask.stride(0), _ptr(temperature), _ptr(top_k),
                                             cand_val.data_ptr(), cand_id.data_ptr(), int(id_offset), rows,
                                             vocab or logits.shape[1], _stream())
    native.check(code, "cb_sample_candidates")


def sample_merge(cand_val: torch.Tensor, cand_id: torch.Tensor, sources: int, source_stride: int, rows: int,
                 out_ids: torch.Tensor, temperature: torch.Tensor | None = None, top_p: torch.Tensor | None = None,
                 top_k: torch.Tensor | None = None, seeds: torch.Tensor | None = None,
                 counters: torch.Tensor | None = None, out_logprob: torch.Tensor | None = None) -> torch.Tensor:
    """Draw every row's token from the union of ``sources`` candidate sets (same result on every rank)."""
    code = native.lib().cb_sample_merge(cand_val.data_ptr(), cand_id.data_ptr(), sources, source_stride, rows,
                                        _ptr(temperature), _ptr(top_p), _ptr(top_k), _ptr(seeds), _ptr(counters),
                                        out_ids.data_ptr(), _ptr(out_logprob), _stream())
    native.check(code, "cb_sample_merge")
    return out_ids


def verify_greedy(target_ids: torch.Tensor, draft_ids: torch.Tensor, depth: torch.Tensor, max_depth: int,
                  accepted: torch.Tensor, bonus: torch.Tensor, forced_reject_at: torch.Tensor | None = None) -> None:
    code = native.lib().cb_verify_greedy(target_ids.data_ptr(), draft_ids.data_ptr(), depth.data_ptr(), max_depth,
                                         _ptr(forced_reject_at), accepted.data_ptr(), bonus.data_ptr(),
                                         depth.numel(), _stream())
    native.check(code, "cb_verify_greedy")


def verify_sampled(q_val: torch.Tensor, q_id: torch.Tensor, p_val: torch.Tensor, p_id: torch.Tensor,
                   draft_ids: torch.Tensor, depth: torch.Tensor, max_depth: int, temperature: torch.Tensor,
                   top_p: torch.Tensor, top_k: torch.Tensor, seeds: torch.Tensor, counters: torch.Tensor,
                   accepted: torch.Tensor, bonus: torch.Tensor, emitted: torch.Tensor) -> None:
    """p / q rejection sampling of a speculative round over sparse candidate distributions (``[R, D, 20]`` draft
    candidates, ``[R, D + 1, 20]`` target candidates as written by ``sample_candidates``); ``emitted [R, D + 1]``
    receives every request's accepted drafts followed by its next token.  See ``csrc/sampling.cu``."""
    code = native.lib().cb_verify_sampled(q_val.data_ptr(), q_id.data_ptr(), p_val.data_ptr(), p_id.data_ptr(),
                                          draft_ids.data_ptr(), depth.data_ptr(), int(max_depth), temperature.data_ptr(),
                                          top_p.data_ptr(), top_k.data_ptr(), seeds.data_ptr(), counters.data_ptr(),
                                          accepted.data_ptr(), bonus.data_ptr(), emitted.data_ptr(), depth.numel(),
                                          _stream())
    native.check(code, "cb_verify_sampled")


# ------------------------------------------------------------------ mixture of experts
class MoeScratch:
    """Fixed-address routing buffers for up to ``max_tokens`` tokens (graph-capturable)."""

    def __init__(self, max_tokens: int, top_k: int, hidden: int, inter2: int, local_experts: int, mb: int, device) -> None:
        routes = max_tokens * top_k
        self.mb = mb
        self.max_items = -(-routes // mb) + local_experts
        i32 = dict(dtype=torch.int32, device=device)
        self.topk_ids = torch.empty(max_tokens, top_k, **i32)
        self.topk_w = torch.empty(max_tokens, top_k, dtype=torch.float32, device=device)
        self.counts = torch.zeros(local_experts, **i32)
        self.offsets = torch.zeros(local_experts, **i32)
        self.cursors = torch.zeros(local_experts, **i32)
        self.total = torch.zeros(1, **i32)
        self.tiles = torch.zeros(1 + 3 * self.max_items, **i32)
        self.route_pos = torch.empty(max_tokens, top_k, **i32)
        bf = dict(dtype=torch.bfloat16, device=device)
        # + mb rows of slack: a work item's TMA tile may run past the last route (those rows are never stored)
        self.xs = torch.zeros(routes + mb, hidden, **bf)
        self.gu = torch.zeros(routes + mb, inter2, **bf)
        self.act = torch.zeros(routes + mb, inter2 // 2, **bf)
        self.y = torch.zeros(routes + mb, hidden, **bf)


def moe_route(router_logits: torch.Tensor, x: torch.Tensor, top_k: int, sc: MoeScratch, normalize: bool = True,
              expert_lo: int = 0, expert_count: int | None = None) -> None:
    t, e = router_logits.shape
    cnt = e if expert_count is None else expert_count
    code = native.lib().cb_moe_route(router_logits.data_ptr(), router_logits.stride(0), x.data_ptr(), t, e, top_k,
                                     x.shape[1], int(normalize), expert_lo, cnt, sc.mb, sc.topk_ids.data_ptr(),
                                     sc.topk_w.data_ptr(), sc.counts.data_ptr(), sc.offsets.data_ptr(),
                                     sc.cursors.data_ptr(), sc.total.data_ptr(), sc.tiles.data_ptr(),
                                     sc.route_pos.data_ptr(), sc.xs.data_ptr(), _stream())
    native.check(code, "cb_moe_route")


def wq_gemm_grouped(x: torch.Tensor, w: PackedWeight, out: torch.Tensor, rows: int, sc: MoeScratch,
                    code_stride: int, meta_stride: int, ws: Workspace | None = None, swiglu: bool = False) -> torch.Tensor:
    """Per-expert ``out[rows of e] = x[rows of e] @ W_e^T`` over the work list in ``sc.tiles``; ``w`` stacks the experts.

    ``swiglu``: every expert's ``[gate; up]`` rows are interleaved and ``out`` (``N / 2`` columns) gets the activation.
    """
    ws = ws or workspace(x.device)
    assert swiglu == w.act_interleaved
    if w.fmt in (FMT_FP8, FMT_FP8_BLOCK):
        # the routed rows (plus the slack rows a work item's tile may touch) are quantized per token, then one grouped
        # launch over the stacked e4m3 experts
        a = fp8_quantize(x[:min(x.shape[0], rows + sc.mb)], ws)
        code = native.lib().cb_wq_gemm_fp8_grouped(a.q.data_ptr(), a.q.stride(0), a.scale.data_ptr(), w.codes.data_ptr(),
                                                   w.meta.data_ptr(), int(w.fmt == FMT_FP8_BLOCK), out.data_ptr(),
                                                   out.stride(0), rows, w.n, w.k,
                                                   sc.tiles.data_ptr(), sc.max_items, sc.mb, w.codes.shape[0], int(swiglu),
                                                   ws.status.data_ptr(), _stream())
        native.check(code, "cb_wq_gemm_fp8_grouped")
        return out
    entry = native.lib().cb_wq_gemm_grouped_act if swiglu else native.lib().cb_wq_gemm_grouped
    code = entry(w.fmt, x.data_ptr(), x.stride(0), w.codes.data_ptr(), _ptr(w.meta),
                                           out.data_ptr(), out.stride(0), float(w.alpha), rows, w.n, w.k, w.group_k,
                                           sc.tiles.data_ptr(), sc.max_items, sc.mb, w.codes.shape[0], code_stride, meta_stride,
                                           ws.status.data_ptr(), _stream())
    native.check(code, "cb_wq_gemm_grouped")
    return out


def moe_combine(y: torch.Tensor, sc: MoeScratch, tokens: int, out: torch.Tensor,
                residual: torch.Tensor | None = None) -> torch.Tensor:
    code = native.lib().cb_moe_combine(y.data_ptr(), sc.route_pos.data_ptr(), sc.topk_w.data_ptr(), tokens,
                                       sc.topk_ids.shape[1], y.shape[1], _ptr(residual), out.data_ptr(), _stream())
    native.check(code, "cb_moe_combine")
    return out


# ------------------------------------------------------------------ gated delta net (hybrid family)
@dataclass
class GdnSegments:
    """A step's token rows grouped by request: rows ``[row0, row0 + count)`` of state slot ``slot``, the first at
    absolute position ``pos0`` (0 = the request starts here, from zero state).  int32 device tensors of length >= num."""
    row0: torch.Tensor
    count: torch.Tensor
    slot: torch.Tensor
    pos0: torch.Tensor
    num: int

    def struct(self) -> "native.GdnSegmentsStruct":
        s = native.GdnSegmentsStruct()
        s.row0, s.count, s.slot, s.pos0 = self.row0.data_ptr(), self.count.data_ptr(), self.slot.data_ptr(), self.pos0.data_ptr()
        s.num = int(self.num)
        return s


def gdn_conv(x: torch.Tensor, w: torch.Tensor, state: torch.Tensor, seg: GdnSegments, out: torch.Tensor,
             bias: torch.Tensor | None = None, commit: bool = True) -> torch.Tensor:
    """Depthwise causal conv1d (kernel 4) + SiLU over ``x[T, C]`` per request segment; ``state[slots, 3, C]`` holds
    every request's last three inputs and is updated unless ``commit`` is False (speculative review pass).
    ``w``: fp32 ``[C, 4]`` (tap 3 multiplies the current input)."""
    c = w.shape[0]
    assert w.dtype == torch.float32 and w.shape[1] == 4 and w.is_contiguous()
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1 and out.stride(1) == 1 and x.shape[1] >= c
    assert state.dtype == torch.bfloat16 and state.shape[1:] == (3, c) and state.is_contiguous()
    st = seg.struct()
    code = native.lib().cb_gdn_conv(x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), w.data_ptr(), _ptr(bias),
                                    state.data_ptr(), ctypes.byref(st), c, int(commit), _stream())
    native.check(code, "cb_gdn_conv")
    return out


def gdn_delta(qkv: torch.Tensor, z: torch.Tensor, ba: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor,
              norm_w: torch.Tensor, state: torch.Tensor, seg: GdnSegments, out: torch.Tensor, hk: int, hv: int,
              eps_norm: float = 1e-6, eps_l2: float = 1e-6, commit: bool = True) -> torch.Tensor:
    """Gated delta rule + gated RMSNorm per (segment, value head); ``state[slots, Hv, 128, 128]`` fp32 is updated
    unless ``commit`` is False (speculative review pass: the state is read, the outputs are written, nothing else).

    ``qkv[T, 2 Hk 128 + Hv 128]`` (after ``gdn_conv``), ``z[T, Hv 128]``, ``ba[T, 2 Hv]`` = ``[b | a]``.
    """
    assert state.dtype == torch.float32 and state.shape[1:] == (hv, 128, 128) and state.is_contiguous()
    for t in (a_log, dt_bias, norm_w):
        assert t.dtype == torch.float32 and t.is_contiguous()
    d = native.GdnDeltaStruct()
    d.qkv, d.ldqkv, d.z, d.ldz, d.ba, d.ldba = qkv.data_ptr(), qkv.stride(0), z.data_ptr(), z.stride(0), ba.data_ptr(), ba.stride(0)
    d.a_log, d.dt_bias, d.norm_w, d.state = a_log.data_ptr(), dt_bias.data_ptr(), norm_w.data_ptr(), state.data_ptr()
    d.out, d.ldo, d.Hk, d.Hv, d.eps_norm, d.eps_l2 = out.data_ptr(), out.stride(0), hk, hv, eps_norm, eps_l2
    d.commit = int(commit)
    st = seg.struct()
    native.check(native.lib().cb_gdn_delta(ctypes.byref(d), ctypes.byref(st), _stream()), "cb_gdn_delta")
    return out


def sigmoid_gate(x: torch.Tensor, gate: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``out = x * sigmoid(gate)`` (bf16; the output gate of the hybrid family's full-attention layers)."""
    rows, cols = x.shape
    out = x if out is None else out
    code = native.lib().cb_sigmoid_gate(x.data_ptr(), x.stride(0), gate.data_ptr(), gate.stride(0), out.data_ptr(),
                                        out.stride(0), rows, cols, _stream())
    native.check(code, "cb_sigmoid_gate")
    return out


# ------------------------------------------------------------------ thinking-token budgets
class ReasoningBudget:
    """Device state of the thinking-token budgets: one counter per request slot (see ``csrc/sampling.cu``)."""

    def __init__(self, slots: int, end_token_id: int, forced_tokens: list[int], device) -> None:
        if not 1 <= len(forced_tokens) <= 4 or end_token_id not in forced_tokens:
            raise ValueError("the forced end sequence has 1 to 4 tokens and contains the closing token")
        self.end_token_id = int(end_token_id)
        self.forced = [int(t) for t in forced_tokens]
        self._seq = (ctypes.c_int * len(self.forced))(*self.forced)
        self.left = torch.full((slots,), -1, dtype=torch.int32, device=device)
        self.fpos = torch.zeros(slots, dtype=torch.int32, device=device)

    def apply(self, ids: torch.Tensor, row_slot: torch.Tensor, init: torch.Tensor, rows: int) -> None:
        """Run the state machine on the step's ``rows`` sampled ids in place."""
        code = native.lib().cb_reasoning_budget(ids.data_ptr(), row_slot.data_ptr(), init.data_ptr(), self.left.data_ptr(),
                                                self.fpos.data_ptr(), rows, self.end_token_id, self._seq,
                                                len(self.forced), _stream())
        native.check(code, "cb_reasoning_budget")


# ------------------------------------------------------------------ layered decoders (models/layered.py)
def _seg(seg: GdnSegments) -> "native.GdnSegmentsStruct":
    return seg.struct()


GLU = {None: 0, "silu": 1, "gelu": 2, "clamped": 3}       # Glu in csrc/wq_gemm_common.cuh


def wide_gemm(x: torch.Tensor, w: PackedWeight, out: torch.Tensor, residual: torch.Tensor | None = None,
              relu2: torch.Tensor | None = None, split: int = 0, diag_rows: int = 0, ws: Workspace | None = None,
              stream_k: bool | None = None, splits: int | None = None, glu: str | None = None, limit: float = 0.0,
              rest: torch.Tensor | None = None, gate: tuple[torch.Tensor, torch.Tensor] | None = None) -> None:
    """``x @ W^T`` with bf16-stored weights through the wide epilogue.

    ``x`` fp32: everything is fp32 (``csrc/layered.cu``); ``x`` bf16: tcgen05 with fp32 accumulation.  ``out`` gets the
    product; an fp32 ``out`` may be added to ``residual`` (the same tensor: in-place accumulation).  With ``relu2`` the
    features from ``split`` on leave there as ``max(v, 0)^2`` and ``out`` holds the first ``split``.  ``glu`` "gelu" / "silu": the
    rows of ``w`` are interleaved [gate ; up] and ``out`` gets ``gelu_tanh(gate) * up`` / ``silu(gate) * up`` (``N / 2`` columns); "clamped":
    ``g sigmoid(1.702 g) (u + 1)`` with ``g = min(gate, limit)`` and ``u`` clamped to ``limit``.  With ``rest`` only the first ``split``
    rows are interleaved, and the other features leave there as they are.  ``gate``: (logits ``[M, N]`` in ``x``'s type, bias fp32
    ``[N]``): the product times the sigmoid of their sum joins ``residual``.  ``diag_rows``: block-diagonal weights, see ``models/layered.py::BlockDiagonal``.  ``x`` may have fewer columns than ``w.k``: the rest
    read as zero."""
    m, k = x.shape[0], w.k
    assert w.fmt == FMT_BF16 and x.stride(1) == 1 and out.stride(1) == 1 and out.shape[0] == m
    assert (glu is not None) == w.act_interleaved and not (glu and (relu2 is not None or residual is not None or diag_rows))
    assert rest is None or glu and rest.dtype == x.dtype and rest.stride(1) == 1 and rest.shape == (m, w.n - split)
    assert out.shape[1] == (split if relu2 is not None else (w.n if rest is None else split) // 2 if glu else w.n), (out.shape, split, w.n)
    g = b = None
    if gate is not None:
        g, b = gate
        assert residual is not None and relu2 is None and g.dtype == x.dtype and g.stride(1) == 1 and g.shape == (m, w.n)
        assert b.dtype == torch.float32 and b.is_contiguous() and b.numel() == w.n
    ldg = 0 if g is None else g.stride(0)
    second = relu2 if rest is None else rest
    ld2 = 0 if second is None else second.stride(0)
    assert residual is None or (residual.dtype == torch.float32 and residual.stride(0) == out.stride(0))
    if relu2 is not None:
        assert relu2.dtype == x.dtype and relu2.stride(1) == 1 and relu2.shape == (m, w.n - split) and split % 4 == 0
    x_cols = min(x.shape[1], x.stride(0))
    l = native.lib()
    if x.dtype == torch.float32:
        assert out.dtype == torch.float32
        a = native.F32GemmStruct(x.data_ptr(), x.stride(0), x_cols, w.codes.data_ptr(), out.data_ptr(), out.stride(0),
                                 _ptr(residual), _ptr(second), ld2, split, diag_rows, m, w.n, k, GLU[glu], None, 0, float(limit),
                                 _ptr(g), ldg, _ptr(b))
        native.check(l.cb_f32_gemm(ctypes.byref(a), _stream()), "cb_f32_gemm")
        return
    wide32 = out.dtype == torch.float32
    assert residual is None or wide32
    assert not (glu and wide32)
    ws = ws or workspace(x.device)
    if stream_k is None:
        stream_k = splits is None and not diag_rows and use_stream_k(m, w.n, FMT_BF16, sm_count(x.device), k)
    if splits is None:
        splits = 1 if stream_k else choose_splits(m, w.n, k, fmt=FMT_BF16)
    if splits > 1 and l.cb_wq_gemm_workspace_bytes(m, w.n, splits) > ws.gemm.numel():
        splits = 1
    from .strategies import active
    a = native.WideGemmStruct(x.data_ptr(), x.stride(0), x_cols, w.codes.data_ptr(), None if wide32 else out.data_ptr(),
                              out.data_ptr() if wide32 else None, out.stride(0), _ptr(residual), _ptr(second), ld2, split,
                              diag_rows, m, w.n, k, int(stream_k), splits, active().gemm.stream_k_min_units, GLU[glu], float(limit),
                              _ptr(g), ldg, _ptr(b))
    code = l.cb_bf16_gemm_wide(ctypes.byref(a), ws.gemm.data_ptr(), ws.gemm.numel(), ws.gemm_counters.data_ptr(),
                               ws.status.data_ptr(), _stream())
    native.check(code, "cb_bf16_gemm_wide")


def row_norm(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, eps: float, rows: torch.Tensor | None = None) -> None:
    """``out[i] = x[i] / rms(x[i]) * weight`` from the fp32 residual stream (``rows``: int64 indices of the rows taken)."""
    assert x.dtype == weight.dtype == torch.float32 and x.is_contiguous() and out.stride(1) == 1
    n = x.shape[0] if rows is None else rows.numel()
    assert out.shape[0] >= n
    native.check(native.lib().cb_row_norm(x.data_ptr(), _ptr(rows), weight.data_ptr(), out.data_ptr(), out.stride(0), n,
                                          x.shape[1], float(eps), int(out.dtype == torch.float32), _stream()), "cb_row_norm")


def embed_norm(ids: torch.Tensor, table: torch.Tensor, weight: torch.Tensor, x: torch.Tensor, eps: float,
               x0: torch.Tensor | None = None) -> None:
    """``x`` (and ``x0``) = RMS norm of the embedding rows, fp32."""
    assert x.dtype == torch.float32 and x.is_contiguous() and table.dtype == torch.bfloat16
    native.check(native.lib().cb_embed_norm(ids.data_ptr(), table.data_ptr(), weight.data_ptr(), x.data_ptr(), _ptr(x0),
                                            x.shape[0], x.shape[1], table.shape[0], float(eps), _stream()), "cb_embed_norm")


def concat_rows(x: torch.Tensor, x0: torch.Tensor, out: torch.Tensor) -> None:
    """``out = [x ; x0]`` along the columns, in ``out``'s type."""
    native.check(native.lib().cb_concat_rows(x.data_ptr(), x0.data_ptr(), out.data_ptr(), out.stride(0), x.shape[0],
                                             x.shape[1], int(out.dtype == torch.float32), _stream()), "cb_concat_rows")


def embed_rows(ids: torch.Tensor, table: torch.Tensor, weight: torch.Tensor, x: torch.Tensor, h: torch.Tensor, eps: float,
               scale: float = 1.0, add: bool = False) -> None:
    """``x`` = ``scale`` times the embedding rows (fp32), added to what it holds with ``add``; ``h = x / rms(x) * weight`` in ``h``'s
    type."""
    assert x.dtype == weight.dtype == torch.float32 and x.is_contiguous() and table.dtype == torch.bfloat16 and h.stride(1) == 1
    native.check(native.lib().cb_embed_rows(ids.data_ptr(), table.data_ptr(), weight.data_ptr(), x.data_ptr(), h.data_ptr(),
                                            h.stride(0), x.shape[0], x.shape[1], table.shape[0], float(eps), float(scale), int(add),
                                            int(h.dtype == torch.float32), _stream()), "cb_embed_rows")


def add_norm_rows(y: torch.Tensor, weight: torch.Tensor, x: torch.Tensor, eps: float, next_weight: torch.Tensor | None = None,
                  h: torch.Tensor | None = None) -> None:
    """``x += y / rms(y) * weight`` on the fp32 residual; with ``h`` also ``h = x / rms(x) * next_weight``, the norm that reads
    the residual next."""
    assert x.dtype == weight.dtype == torch.float32 and x.is_contiguous() and y.stride(1) == 1 and y.shape[1] == x.shape[1]
    assert h is None or h.dtype == y.dtype and h.stride(1) == 1 and next_weight.dtype == torch.float32
    native.check(native.lib().cb_add_norm_rows(y.data_ptr(), y.stride(0), weight.data_ptr(), x.data_ptr(), _ptr(next_weight), _ptr(h),
                                               0 if h is None else h.stride(0), x.shape[0], x.shape[1], float(eps),
                                               int(y.dtype == torch.float32), _stream()), "cb_add_norm_rows")


def side_gate(x: torch.Tensor, gate: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, col: int, out: torch.Tensor) -> None:
    """``out[t, n] = gelu_tanh(x[t] . gate[n]) * table[ids[t], col + n]``: the fp32 residual gates a token's side embedding.
    ``gate`` bf16 ``[dim, columns >= W]`` with zeros behind the width; fp32 ``out``: everything is fp32."""
    dim = gate.shape[0]
    assert x.dtype == torch.float32 and x.is_contiguous() and gate.dtype == table.dtype == torch.bfloat16 and gate.is_contiguous()
    assert out.stride(1) == 1 and out.shape[1] >= dim and out.shape[0] == x.shape[0]
    native.check(native.lib().cb_side_gate(x.data_ptr(), x.shape[1], gate.data_ptr(), gate.shape[1], ids.data_ptr(), table.data_ptr(),
                                           table.shape[1], col, out.data_ptr(), out.stride(0), x.shape[0], dim, table.shape[0],
                                           int(out.dtype == torch.float32), _stream()), "cb_side_gate")


def side_input(x: torch.Tensor, gate: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, col: int, proj: PackedWeight,
               norm_w: torch.Tensor, eps: float, next_w: torch.Tensor | None, h: torch.Tensor | None, g: torch.Tensor, y: torch.Tensor,
               ws: Workspace | None = None) -> int:
    """A layer's whole side input: ``side_gate`` into ``g``, the product with ``proj`` into ``y``, ``add_norm_rows``.  One kernel
    for bf16 rows of the widths it takes, which leaves ``g`` and ``y`` alone.  Returns the launches made."""
    W, dim = x.shape[1], gate.shape[0]
    if y.dtype == torch.float32 or not native.lib().cb_side_input_fits(W, dim):
        side_gate(x, gate, ids, table, col, g)
        wide_gemm(g, proj, y, ws=ws)
        add_norm_rows(y, norm_w, x, eps, next_w, h)
        return 3
    assert x.dtype == norm_w.dtype == torch.float32 and x.is_contiguous() and gate.dtype == table.dtype == torch.bfloat16
    assert proj.fmt == FMT_BF16 and proj.n == W and (h is None) == (next_w is None) and (h is None or h.dtype == torch.bfloat16)
    a = native.SideInputStruct(x.data_ptr(), gate.data_ptr(), gate.shape[1], ids.data_ptr(), table.data_ptr(), table.shape[1], col,
                               table.shape[0], proj.codes.data_ptr(), proj.k, norm_w.data_ptr(), _ptr(next_w), _ptr(h),
                               0 if h is None else h.stride(0), x.shape[0], W, dim, float(eps))
    native.check(native.lib().cb_side_input(ctypes.byref(a), _stream()), "cb_side_input")
    return 1


class RecurrenceScratch:
    """Fixed-address buffers between the preparation and the recurrence of recurrent layers, for up to ``max_tokens`` rows of
    the largest layer they are made for (layers share them)."""

    def __init__(self, max_tokens: int, sizes, act: torch.dtype, device) -> None:
        """``sizes``: (heads, key heads, key width, value width, per channel) of every layer."""
        f32 = dict(dtype=torch.float32, device=device)
        most = lambda f: max(f(*s) for s in sizes)                                     # noqa: E731
        T = max_tokens
        self.q = torch.zeros(T * most(lambda H, G, d, e, c: G * (-(-d // 4) * 4)), **f32)
        self.k = torch.zeros_like(self.q)
        self.kq = torch.zeros(T * most(lambda H, G, d, e, c: G), **f32)
        self.v = torch.zeros(T * most(lambda H, G, d, e, c: H * (-(-e // 8) * 8)), dtype=act, device=device)
        self.coef = torch.zeros(T * most(lambda H, G, d, e, c: 2 * H), **f32)
        self.g = torch.zeros(max(1, T * most(lambda H, G, d, e, c: H * (-(-d // 4) * 4) if c else 0)), **f32)
        self.raw = torch.zeros(T * most(lambda H, G, d, e, c: H * e), **f32)


def _prepare(entry: str, x, a, dt_bias, seg: GdnSegments, sc: RecurrenceScratch, heads: int, kv_heads: int, dim: int, vdim: int,
             channel: bool, offs: tuple[int, int, int], conv=None, b=None, a_log=None, rate: float = 0.0,
             low: PackedWeight | None = None, low_rank: int = 0) -> None:
    """Preparation of a recurrence's tokens (``csrc/recurrence.cuh``).  ``offs``: columns of q, k and v in ``x``; ``conv``:
    (weights fp32 [taps, channels], bias or None, state [slots, taps - 1, channels])."""
    T = x.shape[0]
    ds, es = -(-dim // 4) * 4, -(-vdim // 8) * 8
    assert x.stride(1) == a.stride(1) == 1 and a.dtype == x.dtype
    assert all(t is None or t.dtype == torch.float32 and t.is_contiguous() for t in (a_log, dt_bias))
    assert sc.q.numel() >= T * kv_heads * ds and sc.v.numel() >= T * heads * es and sc.v.dtype == x.dtype
    assert not channel or sc.g.numel() >= T * heads * ds
    w = bias = state = None
    taps = ldw = 0
    if conv is not None:
        w, bias, state = conv
        taps, ldw = w.shape
        assert w.dtype == torch.float32 and w.is_contiguous() and state.dtype == x.dtype and state.is_contiguous()
        assert taps == 1 or tuple(state.shape[1:]) == (taps - 1, ldw)
        assert x.shape[1] == ldw and (bias is None or bias.dtype == torch.float32 and bias.numel() == ldw)
    p = native.RecPrepStruct(x.data_ptr(), x.stride(0), _ptr(w), _ptr(bias), ldw, taps, _ptr(state), *offs, _ptr(b),
                             0 if b is None else b.stride(0), a.data_ptr(), a.stride(0), _ptr(a_log), dt_bias.data_ptr(),
                             float(rate), sc.q.data_ptr(), sc.k.data_ptr(), sc.kq.data_ptr(), sc.v.data_ptr(),
                             sc.coef.data_ptr(), sc.g.data_ptr() if channel else None, None if low is None else low.codes.data_ptr(),
                             0 if low is None else low.k, low_rank, heads, kv_heads, dim, vdim, ds, es, T, int(x.dtype == torch.float32))
    st = _seg(seg)
    native.check(getattr(native.lib(), entry)(ctypes.byref(p), ctypes.byref(st), _stream()), entry)


def delta_prepare(x: torch.Tensor, b: torch.Tensor, a: torch.Tensor, conv_w: torch.Tensor, conv_state: torch.Tensor,
                  a_log: torch.Tensor, dt_bias: torch.Tensor, seg: GdnSegments, sc: RecurrenceScratch, heads: int, kv_heads: int,
                  dim: int, vdim: int) -> None:
    """Everything of a delta layer's tokens that does not depend on its state: causal depthwise convolution + SiLU of
    ``x [T, q | k | v]`` with ``conv_w`` fp32 ``[taps, channels]`` (the last row multiplies the current input) and the
    requests' last inputs ``conv_state [slots, taps - 1, channels]``, which are read and replaced; unit q / k; step sizes and
    decays from the logits ``b`` and ``a``."""
    assert b.stride(1) == 1 and b.dtype == x.dtype and dt_bias.numel() in (heads, heads * dim)
    _prepare("cb_delta_prepare", x, a, dt_bias, seg, sc, heads, kv_heads, dim, vdim, dt_bias.numel() != heads,
             (0, kv_heads * dim, 2 * kv_heads * dim), (conv_w, None, conv_state), b, a_log)


def gated_linear_prepare(x: torch.Tensor, q_off: int, k_off: int, v_off: int, a: torch.Tensor, bias: torch.Tensor, rate: float,
                         seg: GdnSegments, sc: RecurrenceScratch, heads: int, dim: int, vdim: int, low: PackedWeight | None = None,
                         low_rank: int = 0) -> None:
    """The tokens of gated linear attention: q times ``dim^-1/2``, k and v at their columns of ``x``; decays
    ``sigmoid(a + bias)^rate`` per key channel.  With ``low`` (bf16 rows) ``a`` holds the ``low.k`` inner columns of the low-rank
    logits, zero from ``low_rank`` on, and the logits ``a low^T`` are made on the way, in fp32."""
    assert bias.numel() == heads * dim and x.stride(0) % 2 == 0
    if low is None:
        assert a.shape[1] == heads * dim
    else:
        assert low.fmt == FMT_BF16 and low.n == heads * dim and a.shape[1] == low.k and a.dtype == torch.bfloat16
        assert a.data_ptr() % 16 == 0 and a.stride(0) % 8 == 0
    assert x.shape[1] >= max(q_off + heads * dim, k_off + heads * dim, v_off + heads * vdim)
    _prepare("cb_gated_linear_prepare", x, a, bias, seg, sc, heads, heads, dim, vdim, True, (q_off, k_off, v_off), rate=rate,
             low=low, low_rank=low_rank)


def ssd_prepare(x: torch.Tensor, dt: torch.Tensor, conv_w: torch.Tensor, conv_b: torch.Tensor, conv_state: torch.Tensor,
                a_log: torch.Tensor, dt_bias: torch.Tensor, seg: GdnSegments, sc: RecurrenceScratch, heads: int, groups: int,
                state: int, vdim: int) -> None:
    """The tokens of a state-space layer: convolution with bias + SiLU of ``x [T, x | B | C]`` (state as in
    ``delta_prepare``), step sizes ``softplus(dt + dt_bias)`` and decays."""
    assert dt.shape[1] == a_log.numel() == dt_bias.numel() == heads and conv_b is not None
    inner = heads * vdim
    _prepare("cb_ssd_prepare", x, dt, dt_bias, seg, sc, heads, groups, state, vdim, False,
             (inner + groups * state, inner, 0), (conv_w, conv_b, conv_state), a_log=a_log)


def _walk(entry: str, T: int, z, norm_w, skip, state, seg: GdnSegments, out, sc: RecurrenceScratch, kv_heads: int, dim: int,
          eps: float, sigmoid_gate: bool, channel: bool, decode: bool, f32: bool) -> None:
    H, e, ds = state.shape[1:]
    assert state.dtype == torch.float32 and state.is_contiguous() and ds == -(-dim // 4) * 4
    assert (sc.v.dtype == torch.float32) == f32 and sc.raw.numel() >= T * H * e
    assert z is None or z.dtype == out.dtype == sc.v.dtype and z.stride(1) == out.stride(1) == 1 and out.shape[1] == H * e
    assert all(t is None or t.dtype == torch.float32 and t.is_contiguous() for t in (norm_w, skip))
    p = native.RecWalkStruct(sc.q.data_ptr(), sc.k.data_ptr(), sc.kq.data_ptr(), sc.v.data_ptr(), sc.coef.data_ptr(),
                             sc.g.data_ptr() if channel else None, _ptr(skip), _ptr(z), 0 if z is None else z.stride(0),
                             _ptr(norm_w), state.data_ptr(), _ptr(out), 0 if out is None else out.stride(0), sc.raw.data_ptr(), H,
                             kv_heads, dim, e, ds, -(-e // 8) * 8, float(eps), int(sigmoid_gate), int(decode), T, int(f32))
    st = _seg(seg)
    native.check(getattr(native.lib(), entry)(ctypes.byref(p), ctypes.byref(st), _stream()), entry)


def delta_walk(z: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor, seg: GdnSegments, out: torch.Tensor,
               sc: RecurrenceScratch, kv_heads: int, dim: int, eps: float, sigmoid_gate: bool, channel: bool, decode: bool) -> int:
    """The recurrence over the rows prepared by ``delta_prepare`` and the gated norm of every head.  ``state`` fp32
    ``[slots, H, vdim, stride]`` is read and replaced; ``channel``: one decay per key channel; ``decode``: every segment has
    at most one row.  Returns the launches made (at most)."""
    _walk("cb_delta_walk", z.shape[0], z, norm_w, None, state, seg, out, sc, kv_heads, dim, eps, sigmoid_gate, channel, decode,
          z.dtype == torch.float32)
    return 1 if decode else 2


def gated_linear_walk(z: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor, seg: GdnSegments, out: torch.Tensor,
                      sc: RecurrenceScratch, dim: int, eps: float, decode: bool) -> int:
    """Gated linear attention over the rows of ``gated_linear_prepare``: recurrence, norm of every head, times ``silu(z)``.
    State and return value as in ``delta_walk``."""
    _walk("cb_linear_walk", z.shape[0], z, norm_w, None, state, seg, out, sc, state.shape[1], dim, eps, False, True, decode,
          z.dtype == torch.float32)
    return 1 if decode else 2


def ssd_walk(z: torch.Tensor, d: torch.Tensor, norm_w: torch.Tensor, parts: int, state: torch.Tensor, seg: GdnSegments,
             out: torch.Tensor, sc: RecurrenceScratch, groups: int, dim: int, eps: float, decode: bool) -> int:
    """State-space layer over the rows of ``ssd_prepare``: recurrence, ``d`` times the value rows, and the gated norm in
    ``parts`` equal parts across the heads.  State and return value as in ``delta_walk``."""
    T, f32 = z.shape[0], z.dtype == torch.float32
    width = norm_w.numel() // parts
    assert z.shape[1] == out.shape[1] == parts * width and z.dtype == out.dtype and d.numel() == state.shape[1]
    _walk("cb_linear_walk", T, None, None, d, state, seg, None, sc, groups, dim, eps, False, False, decode, f32)
    native.check(native.lib().cb_gated_parts_norm(sc.raw.data_ptr(), z.data_ptr(), z.stride(0), norm_w.data_ptr(), out.data_ptr(),
                                                  out.stride(0), T, parts, width, float(eps), int(f32), _stream()),
                 "cb_gated_parts_norm")
    return 2


def latent_prepare(proj: torch.Tensor, c_off: int, rank: int, c_norm: torch.Tensor, cache: torch.Tensor, slots: torch.Tensor, eps: float,
                   low: tuple[int, int, torch.Tensor, torch.Tensor] | None = None,
                   rotated: tuple[int, int, int, torch.Tensor, float, torch.Tensor, torch.Tensor, int] | None = None) -> None:
    """RMS norm of the cache latent (columns ``[c_off, c_off + rank)`` of ``proj``) into its page of ``cache`` ``[pages, 16, padded]``.
    ``low`` = (first column, rank, norm weight, destination): the same for a query latent.  ``rotated`` = (first column of the
    queries' rotated parts, of the shared key's, column of a row they go to, ``freq`` fp32 ``[2, pairs]``, factor on cosine and sine,
    positions, latent-space queries ``[T, H padded]``, heads): neighbouring channels turn with the position, queries beside their
    latent part and the key into the cached row."""
    assert cache.is_contiguous() and cache.dtype == proj.dtype and slots.dtype == torch.int32 and proj.stride(1) == 1
    q_off, q_rank, q_norm, cq = low or (0, 0, None, None)
    qr_off, r_off, col, freq, mult, positions, ql, heads = rotated or (0, 0, 0, None, 1.0, None, None, 0)
    if low:
        assert cq.dtype == proj.dtype and cq.stride(1) == 1
    if rotated:
        assert ql.dtype == proj.dtype and ql.is_contiguous() and ql.shape[1] == heads * cache.shape[2] and positions.dtype == torch.int32
        assert freq.dtype == torch.float32 and freq.is_contiguous() and freq.shape[0] == 2
    a = native.LatentPrepStruct(proj.data_ptr(), proj.stride(0), q_off, q_rank, c_off, rank, _ptr(q_norm), c_norm.data_ptr(), _ptr(cq),
                                0 if cq is None else cq.stride(0), cache.data_ptr(), cache.shape[2], slots.data_ptr(), qr_off, r_off, col,
                                0 if freq is None else freq.shape[1], _ptr(freq), float(mult), _ptr(positions), _ptr(ql), heads,
                                proj.shape[0], float(eps), int(proj.dtype == torch.float32))
    native.check(native.lib().cb_latent_prepare(ctypes.byref(a), _stream()), "cb_latent_prepare")


def latent_attention(q: torch.Tensor, gate: torch.Tensor | None, cache: torch.Tensor, page_table: torch.Tensor, seg: GdnSegments,
                     out: torch.Tensor, heads: int, window: int, scale: float, decode: bool = False, splits: int | None = None,
                     ws: Workspace | None = None) -> None:
    """Windowed softmax attention of latent-space queries ``q [T, H Rp]`` over the paged rows; a row's first columns are its value too
    (``out [T, H Rv]``).  ``gate``: logits ``[T, H]`` of a sigmoid per head, or None.  ``window`` 0: every earlier token.
    ``decode``: every segment has at most one row.  ``splits``: key splits of the bf16 form (None: as many as fill the device)."""
    T, rp, rv = q.shape[0], cache.shape[2], out.shape[1] // heads
    assert q.shape[1] == heads * rp and out.shape[1] == heads * rv and rv <= rp and q.is_contiguous() and out.is_contiguous()
    assert q.dtype == out.dtype == cache.dtype and page_table.dtype == torch.int32 and (gate is None or gate.dtype == q.dtype)
    f32 = q.dtype == torch.float32
    l = native.lib()
    partial = None
    if f32 or not l.cb_latent_attn_mma(rp, rv):
        splits = 1
    else:
        units = ctypes.c_int(0)
        l.cb_latent_attn_partial_floats(T, seg.num, heads, rv, int(decode), 1, ctypes.byref(units))
        if splits is None:
            from .strategies import active
            a = active().attention
            # a block walks tiles of 64 keys: no more splits than the longest row has tiles
            keys = page_table.shape[1] * PAGE_TOKENS if window <= 0 else min(window, page_table.shape[1] * PAGE_TOKENS)
            splits = min(a.max_splits, -(-keys // 64), max(1, a.target_ctas // (1 if decode else 2) // units.value))
        if splits > 1:
            ws = ws or workspace(q.device)
            ws.ensure_attn(l.cb_latent_attn_partial_floats(T, seg.num, heads, rv, int(decode), splits, None))
            partial = ws.attn.data_ptr()
    a = native.LatentAttnStruct(q.data_ptr(), out.data_ptr(), cache.data_ptr(), _ptr(gate), 0 if gate is None else gate.stride(0),
                                page_table.data_ptr(), page_table.shape[1], heads, rp, rv, window, float(scale), T, int(f32),
                                int(decode), splits, partial)
    st = _seg(seg)
    native.check(l.cb_latent_attn(ctypes.byref(a), ctypes.byref(st), _stream()), "cb_latent_attn")


def gqa_prepare(x: torch.Tensor, q_off: int, k_off: int, q_norm: torch.Tensor, k_norm: torch.Tensor, freq: torch.Tensor,
                mult: float, positions: torch.Tensor, slots: torch.Tensor, q: torch.Tensor, cache: torch.Tensor, heads: int,
                dim: int, eps: float) -> None:
    """Query and key heads of ``x``'s rows: RMS norm of a head, rotary positions on its first ``2 len(freq)`` channels; queries to
    ``q [T, H P]``, keys and the raw key heads (values) to their rows of ``cache [pages, G, 2, 16, P]``."""
    G, P = cache.shape[1], cache.shape[4]
    assert cache.is_contiguous() and cache.dtype == x.dtype == q.dtype and q.is_contiguous() and q.shape[1] == heads * P
    assert x.stride(1) == 1 and slots.dtype == positions.dtype == torch.int32
    assert q_norm.dtype == k_norm.dtype == freq.dtype == torch.float32
    a = native.GqaPrepStruct(x.data_ptr(), x.stride(0), q_off, k_off, q_norm.data_ptr(), k_norm.data_ptr(), freq.data_ptr(),
                             float(mult), positions.data_ptr(), slots.data_ptr(), q.data_ptr(), cache.data_ptr(), heads, G, dim, P,
                             freq.numel(), float(eps), x.shape[0], int(x.dtype == torch.float32))
    native.check(native.lib().cb_gqa_prepare(ctypes.byref(a), _stream()), "cb_gqa_prepare")


def gqa_attention(q: torch.Tensor, cache: torch.Tensor, page_table: torch.Tensor, seg: GdnSegments, out: torch.Tensor, heads: int,
                  dim: int, window: int, scale: float, sink: float | None = None, out_scale: float = 1.0, decode: bool = False,
                  splits: int | None = None, ws: Workspace | None = None, keep: int = 0, bias: torch.Tensor | None = None,
                  chunk: int = 0, pair: tuple[torch.Tensor, float, float] | None = None) -> int:
    """Windowed grouped-query attention over the paged cache of ``gqa_prepare``, ``conv_qkv`` or ``norm_qkv`` with values of
    ``dim`` channels, times ``out_scale``.  ``window`` 0: every earlier token; ``keep``: the first tokens stay visible behind the
    window; ``bias`` fp32 ``[distances, H]`` is added to the scaled scores, its last row from the last distance on; ``sink``:
    score of a softmax entry without a value.  ``chunk`` > 0 (instead of a window): a token sees its own chunk of positions, counted
    from the sequence's first.  ``pair`` = (gate logits ``[T, H dim]``, factor, eps): query and key rows hold two maps, half of their
    columns each, over the same values; the second map's output times the factor is taken from the first's, and the difference goes
    over its root mean square, times ``out_scale`` and the sigmoid of the gate.  ``decode``: every segment has at most one row.
    ``splits``: key splits of the bf16 decode form (None: as many as fill the device).  Returns the launches made."""
    G, P = cache.shape[1], cache.shape[4]
    T = q.shape[0]
    assert q.is_contiguous() and q.shape[1] == heads * P and out.stride(1) == 1 and out.shape[1] == heads * dim
    assert q.dtype == out.dtype == cache.dtype and page_table.dtype == torch.int32
    assert bias is None or bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[1] == heads
    gate, less, eps = pair or (None, 0.0, 0.0)
    assert gate is None or gate.dtype == q.dtype and gate.stride(1) == 1 and gate.shape == out.shape
    maps = 1 if pair is None else 2
    f32 = q.dtype == torch.float32
    l = native.lib()
    partial = None
    if f32 or not decode:
        splits = 1
    else:
        if splits is None:
            from .strategies import active
            units = ctypes.c_int(0)
            l.cb_gqa_attn_partial_floats(T, seg.num, heads, G, P, maps, 1, 1, ctypes.byref(units))
            a = active().attention
            # a block walks four pages at a time: no more splits than the longest row has such strides
            most = chunk or (window + keep if window > 0 else 0)
            keys = min(most or page_table.shape[1] * PAGE_TOKENS, page_table.shape[1] * PAGE_TOKENS)
            splits = min(a.max_splits, -(-keys // 64), max(1, a.target_ctas // units.value))
        if splits > 1:
            ws = ws or workspace(q.device)
            ws.ensure_attn(l.cb_gqa_attn_partial_floats(T, seg.num, heads, G, P, maps, 1, splits, None))
            partial = ws.attn.data_ptr()
    a = native.GqaAttnStruct(q.data_ptr(), out.data_ptr(), out.stride(0), cache.data_ptr(), page_table.data_ptr(),
                             page_table.shape[1], heads, G, dim, P, window, keep, chunk, float(scale), float(out_scale),
                             float("-inf") if sink is None else float(sink), _ptr(bias), 0 if bias is None else bias.shape[0] - 1,
                             _ptr(gate), 0 if gate is None else gate.stride(0), float(less), float(eps), T, int(f32), int(decode), splits,
                             partial)
    st = _seg(seg)
    native.check(l.cb_gqa_attn(ctypes.byref(a), ctypes.byref(st), _stream()), "cb_gqa_attn")
    return 2 if splits > 1 else 1


def _qkv(x: torch.Tensor, offs: tuple[int, int, int], positions: torch.Tensor, slots: torch.Tensor, q: torch.Tensor,
         cache: torch.Tensor, heads: int, dim: int, vdim: int, eps: float) -> "native.QkvPrepStruct":
    G, P = cache.shape[1], cache.shape[4]
    assert cache.is_contiguous() and cache.dtype == x.dtype == q.dtype and q.is_contiguous() and q.shape[1] == heads * P
    assert x.stride(1) == 1 and slots.dtype == positions.dtype == torch.int32 and x.shape[1] >= offs[2] + G * vdim
    return native.QkvPrepStruct(x.data_ptr(), x.stride(0), *offs, q.data_ptr(), cache.data_ptr(), slots.data_ptr(), positions.data_ptr(),
                                heads, G, dim, vdim, P, float(eps), x.shape[0], int(x.dtype == torch.float32))


def head_qkv(x: torch.Tensor, offs: tuple[int, int, int], q_norm: torch.Tensor, k_norm: torch.Tensor, freq: torch.Tensor,
             positions: torch.Tensor, slots: torch.Tensor, q: torch.Tensor, cache: torch.Tensor, heads: int, dim: int, vdim: int,
             eps: float, maps: int = 1) -> None:
    """Queries, keys and values at the columns ``offs`` of ``x``: every head (and map of it) of queries and keys over its root mean
    square, times a weight per channel, then rotary positions of channel i with channel ``i + pairs`` (``freq`` fp32 ``[2, pairs]``:
    radians per position and what rounding took from them).  Queries to ``q [T, H P]``, keys and values to
    ``cache [pages, G, 2, 16, P]``; the maps of a head share its row of ``P`` columns evenly."""
    assert q_norm.dtype == k_norm.dtype == freq.dtype == torch.float32 and q_norm.numel() == k_norm.numel() == dim
    assert freq.is_contiguous() and freq.shape[0] == 2
    a = native.HeadQkvStruct(_qkv(x, offs, positions, slots, q, cache, heads, dim, vdim, eps), q_norm.data_ptr(), k_norm.data_ptr(),
                             freq.data_ptr(), freq.shape[1], maps)
    native.check(native.lib().cb_head_qkv(ctypes.byref(a), _stream()), "cb_head_qkv")


def mingru(x: torch.Tensor, z_off: int, x_off: int, g_off: int, bias: torch.Tensor, state: torch.Tensor, seg: GdnSegments,
           out: torch.Tensor) -> None:
    """Element-wise recurrence of ``out``'s channels: ``S <- (1 - z) S + z c`` with ``z`` = sigmoid of the columns ``z_off`` of ``x`` plus
    ``bias[0]`` and the candidate ``c`` from the columns ``x_off`` plus ``bias[1]`` (``u + 1/2`` of ``u >= 0``, else its sigmoid);
    ``out`` = ``S silu(x[:, g_off:])``.  ``state`` fp32 ``[slots, channels or more]`` is read (zero at position 0) and replaced."""
    T, width = out.shape
    assert x.dtype == out.dtype and x.stride(1) == out.stride(1) == 1 and x.shape[1] >= max(z_off, x_off, g_off) + width
    assert state.dtype == bias.dtype == torch.float32 and bias.is_contiguous() and tuple(bias.shape) == (2, width)
    assert state.stride(-1) == 1 and state.dim() == 2 and state.shape[1] >= width
    a = native.MinGruStruct(x.data_ptr(), x.stride(0), z_off, x_off, g_off, bias.data_ptr(), state.data_ptr(), state.stride(0),
                            out.data_ptr(), out.stride(0), width, T, int(x.dtype == torch.float32))
    st = _seg(seg)
    native.check(native.lib().cb_mingru(ctypes.byref(a), ctypes.byref(st), _stream()), "cb_mingru")


def conv_qkv(x: torch.Tensor, offs: tuple[int, int, int], conv_w: torch.Tensor, state: torch.Tensor | None, freq: torch.Tensor,
             positions: torch.Tensor, slots: torch.Tensor, seg: GdnSegments, q: torch.Tensor, cache: torch.Tensor, heads: int, dim: int,
             vdim: int, eps: float) -> None:
    """Queries, keys and values at the columns ``offs`` of ``x``: causal depthwise convolution over the tokens of a request
    (``conv_w`` fp32 ``[taps, channels]`` over the columns from ``offs[0]`` on, the last row multiplies the current input; the
    requests' last inputs ``state [slots, taps - 1, channels]`` are read and replaced), rotary positions of channel i with channel
    ``i + pairs`` (``freq`` fp32 ``[2, pairs]``: radians per position and what rounding took from them), queries and keys of a
    head over their root mean square.  Queries to ``q [T, H P]``, keys and values to ``cache [pages, G, 2, 16, P]``."""
    taps, ldw = conv_w.shape
    assert conv_w.dtype == freq.dtype == torch.float32 and conv_w.is_contiguous() and freq.is_contiguous() and freq.shape[0] == 2
    assert taps == 1 or state.dtype == x.dtype and state.is_contiguous() and tuple(state.shape[1:]) == (taps - 1, ldw)
    a = native.ConvQkvStruct(_qkv(x, offs, positions, slots, q, cache, heads, dim, vdim, eps), conv_w.data_ptr(), ldw, taps,
                             _ptr(state), freq.data_ptr(), freq.shape[1])
    st = _seg(seg)
    native.check(native.lib().cb_conv_qkv(ctypes.byref(a), ctypes.byref(st), _stream()), "cb_conv_qkv")


def norm_qkv(x: torch.Tensor, offs: tuple[int, int, int], q_norm: torch.Tensor, k_norm: torch.Tensor, positions: torch.Tensor,
             slots: torch.Tensor, q: torch.Tensor, cache: torch.Tensor, heads: int, dim: int, vdim: int, eps: float,
             temp: tuple[float, int] = (0.0, 0)) -> None:
    """Like ``conv_qkv`` without convolution and rotation: the queries of a token together, and its keys, over their root mean
    square and times a weight per channel; queries times ``1 + coef ln(floor((position + 1) / every) + 1)`` with ``temp`` =
    (coef, every), every 0: no factor."""
    assert q_norm.dtype == k_norm.dtype == torch.float32 and q_norm.numel() == heads * dim and k_norm.numel() == cache.shape[1] * dim
    a = native.NormQkvStruct(_qkv(x, offs, positions, slots, q, cache, heads, dim, vdim, eps), q_norm.data_ptr(), k_norm.data_ptr(),
                             float(temp[0]), int(temp[1]))
    native.check(native.lib().cb_norm_qkv(ctypes.byref(a), _stream()), "cb_norm_qkv")


# ------------------------------------------------------------------ several residual streams
def stream_embed(ids: torch.Tensor, table: torch.Tensor, scale: float, x: torch.Tensor, w_in: torch.Tensor, norm_w: torch.Tensor,
                 h: torch.Tensor, eps: float) -> None:
    """All streams of ``x`` fp32 ``[T, S, W]`` = ``scale`` times the embedding rows; ``h`` = norm of their sum weighted by ``w_in``."""
    _stream_norm(x, w_in, norm_w, h, eps, x.shape[0], None, ids, table, scale)


def stream_norm(x: torch.Tensor, norm_w: torch.Tensor, h: torch.Tensor, eps: float, rows: torch.Tensor | None = None,
                w_in: torch.Tensor | None = None) -> None:
    """``h[i]`` = norm of row i's streams, summed with weights ``w_in`` (None: ones); ``rows`` int64: the rows taken."""
    _stream_norm(x, w_in, norm_w, h, eps, x.shape[0] if rows is None else rows.numel(), rows, None, None, 1.0)


def _stream_norm(x, w_in, norm_w, h, eps, n, rows, ids, table, scale) -> None:
    assert x.dtype == norm_w.dtype == torch.float32 and x.is_contiguous() and x.dim() == 3 and h.stride(1) == 1 and h.shape[0] >= n
    assert w_in is None or w_in.dtype == torch.float32 and w_in.numel() == x.shape[1]
    assert table is None or table.dtype == torch.bfloat16 and table.shape[1] == x.shape[2]
    a = native.StreamNormStruct(_ptr(ids), _ptr(table), 0 if table is None else table.shape[0], float(scale), x.data_ptr(), _ptr(rows),
                                _ptr(w_in), norm_w.data_ptr(), h.data_ptr(), h.stride(0), n, x.shape[1], x.shape[2], float(eps),
                                int(h.dtype == torch.float32))
    native.check(native.lib().cb_stream_norm(ctypes.byref(a), _stream()), "cb_stream_norm")


def stream_step(x: torch.Tensor, y: torch.Tensor | None, mix: torch.Tensor, out: torch.Tensor, h: torch.Tensor, eps: float,
                next_in: torch.Tensor | None = None, next_w: torch.Tensor | None = None, routes: "RoutedResult | None" = None) -> None:
    """A sublayer's result ``y`` joins the streams ``x`` fp32 ``[T, S, W]``: ``x_t <- sum_s mix[s, t] x_s + out[t] y``.  ``routes``:
    the result is what the token's experts left, plus ``y`` times the shared expert's gate, plus the sublayer's input ``h`` times
    the weight of the experts that return it.  With ``next_w`` ``h`` becomes the next sublayer's input, the norm of
    ``sum_s next_in[s] x_s``."""
    T, S, W = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and h.stride(1) == 1 and h.shape[0] >= T
    assert y is None or y.dtype == h.dtype and y.stride(1) == 1 and y.shape[1] >= W
    r = routes
    assert all(t is None or t.dtype == torch.float32 for t in (mix, out, next_in, next_w)) and mix.numel() == S * S and out.numel() == S
    a = native.StreamStepStruct(
        x.data_ptr(), _ptr(y), 0 if y is None else y.stride(0), None if r is None else r.rows.data_ptr(), 0 if r is None else r.rows.stride(0),
        None if r is None else r.pos.data_ptr(), None if r is None else r.weight.data_ptr(), None if r is None else _ptr(r.self_weight),
        0 if r is None else r.top, None if r is None else _ptr(r.gate), 0 if r is None or r.gate is None else r.gate.stride(0),
        mix.data_ptr(), out.data_ptr(), _ptr(next_in), _ptr(next_w), h.data_ptr(), h.stride(0), T, S, W, float(eps),
        int(h.dtype == torch.float32))
    native.check(native.lib().cb_stream_step(ctypes.byref(a), _stream()), "cb_stream_step")


# ------------------------------------------------------------------ scored experts
@dataclass
class RoutedResult:
    """What ``stream_step`` puts a routed feed-forward's result together from."""
    rows: torch.Tensor               # [routes, W] results of the experts, by place
    pos: torch.Tensor                # int32 [T, top] places, -1: none
    weight: torch.Tensor             # fp32 [T, top]
    self_weight: torch.Tensor | None # fp32 [T] weight of the token itself
    gate: torch.Tensor | None        # fp32 [T, 1] logits of the shared expert's gate (any row stride)
    top: int


class ScoredScratch:
    """Fixed-address buffers between routing and combination for up to ``max_tokens`` tokens of layers with ``experts`` experts of
    which a token uses ``top``."""

    def __init__(self, max_tokens: int, top: int, experts: int, width: int, k: int, act: torch.dtype, device) -> None:
        """``k``: columns of an expert's operand (``width`` rounded up, the rest stays zero)."""
        routes = max_tokens * top
        i32 = dict(dtype=torch.int32, device=device)
        self.ids, self.pos = torch.zeros(routes, **i32), torch.zeros(routes, **i32)
        self.weight = torch.zeros(routes, dtype=torch.float32, device=device)
        self.self_weight = torch.zeros(max_tokens, dtype=torch.float32, device=device)
        self.counts = torch.zeros(experts + 1, **i32)
        self.tiles = torch.zeros(1 + 3 * (-(-routes // 16) + experts), **i32)
        self.xs = torch.zeros(routes, k, dtype=act, device=device)
        self.ys = torch.zeros(routes, -(-width // 8) * 8, dtype=act, device=device)


def rows_per_item(tokens: int, top: int, experts: int, f32: bool) -> int:
    """Rows of a work item of the grouped products: about twice an expert's average share (one item for most experts)."""
    if f32:
        return 64                                      # the fp32 product's tile
    share = 2 * tokens * top // experts
    return 32 if share <= 32 else 64 if share <= 64 else 128 if share <= 128 else 256


def scored_route(z: torch.Tensor, correction: torch.Tensor, h: torch.Tensor, width: int, experts: int, top: int, sc: ScoredScratch) -> int:
    """Routes ``h``'s rows by the fp32 logits ``z [T, >= outputs]`` (outputs = ``correction.numel()``; those from ``experts`` on
    return the token itself) and copies them to their experts' places in ``sc.xs``.  Returns the rows of a work item."""
    T = z.shape[0]
    assert z.dtype == correction.dtype == torch.float32 and z.stride(1) == 1 and h.dtype == sc.xs.dtype and h.stride(1) == 1
    assert sc.counts.numel() == experts + 1 and T * top <= sc.ids.numel()
    mb = rows_per_item(T, top, experts, h.dtype == torch.float32)
    a = native.ScoredMoeStruct(z.data_ptr(), z.stride(0), correction.data_ptr(), h.data_ptr(), h.stride(0), sc.xs.data_ptr(), sc.xs.stride(0),
                               T, width, h.element_size(), experts, correction.numel(), top, mb, sc.ids.data_ptr(), sc.pos.data_ptr(),
                               sc.weight.data_ptr(), sc.self_weight.data_ptr(), sc.counts.data_ptr(), sc.tiles.data_ptr())
    native.check(native.lib().cb_scored_moe_route(ctypes.byref(a), _stream()), "cb_scored_moe_route")
    return mb


def grouped_gemm(x: torch.Tensor, w: PackedWeight, out: torch.Tensor, sc: ScoredScratch, rows: int, mb: int, relu2: bool = False,
                 ws: Workspace | None = None) -> None:
    """``out[rows of e] = x[rows of e] @ W_e^T`` (``relu2``: ``max(v, 0)^2`` of it) over the work list of ``scored_route`` for bf16
    experts stacked in ``w``; ``rows``: tokens times routes of a token.  fp32 ``x``: everything is fp32."""
    E = w.codes.shape[0]
    assert w.fmt == FMT_BF16 and w.codes.dim() == 3 and x.shape[1] == w.k and out.shape[1] == w.n and out.dtype == x.dtype
    assert x.stride(1) == out.stride(1) == 1
    items = -(-rows // mb) + E
    l = native.lib()
    if x.dtype == torch.float32:
        # with relu2 every feature leaves through the second output, from feature 0 on
        a = native.F32GemmStruct(x.data_ptr(), x.stride(0), x.shape[1], w.codes.data_ptr(), out.data_ptr(), out.stride(0), None,
                                 out.data_ptr() if relu2 else None, out.stride(0) if relu2 else 0, 0, 0, rows, w.n, w.k, 0,
                                 sc.tiles.data_ptr(), items)
        native.check(l.cb_f32_gemm(ctypes.byref(a), _stream()), "cb_f32_gemm")
        return
    ws = ws or workspace(x.device)
    if relu2:
        code = l.cb_wq_gemm_grouped_relu2(x.data_ptr(), x.stride(0), w.codes.data_ptr(), out.data_ptr(), out.stride(0), rows, w.n, w.k,
                                          sc.tiles.data_ptr(), items, mb, E, ws.status.data_ptr(), _stream())
    else:
        code = l.cb_wq_gemm_grouped(FMT_BF16, x.data_ptr(), x.stride(0), w.codes.data_ptr(), None, out.data_ptr(), out.stride(0), 1.0, rows,
                                    w.n, w.k, w.k, sc.tiles.data_ptr(), items, mb, E, 0, 0, ws.status.data_ptr(), _stream())
    native.check(code, "cb_wq_gemm_grouped")
