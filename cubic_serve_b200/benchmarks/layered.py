"""Layered decoders beside the closest existing model at equal size: kernels against their rooflines, prefill and decode
throughput of whole models (``bench.py --layered``).

The closest model is the hybrid family (Gated DeltaNet layers with periodic full attention) with bf16 weights; its SwiGLU
feed-forward has three matrices where a parallel layer's has two, so its width is two thirds of that: equal parameters (the
sequential layers have the same three matrices).  For the layers on several residual streams it is the family of grouped-query
decoders with routed experts: an expert there has three matrices where one here has two, so its width is two thirds.  The layers with
gated residuals have two square matrices more each: their feed-forwards are narrower by that.

Weights are random, prompts are random ids, one GPU.  Kernel times are CUDA-event times inside CUDA graphs with L2 flushed; the
roofline of a kernel is the slower of its bytes over the copy bandwidth and its operations over the pipe that runs them.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from ..models.config import ModelConfig, QuantSpec
from ..models.layered import (AttentionSpec, BiasedAttentionSpec, ConvAttentionSpec, DeltaSpec, DifferentialSpec, GatedLinearSpec,
                              LatentSpec, LayeredConfig, LayerSpec, MinGruSpec, PairSpec, RotarySpec, RoutedSpec, SsdSpec)
from ..ops import kernels as K, wq_pack
from ..utils.kernel_bench import DEV, timeit_graph

FP32_FLOPS = 148 * 128 * 2 * 1.965e9      # one fp32 multiply-add per lane and cycle


def peaks() -> dict:
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if p.is_file():
        d = json.loads(p.read_text())
        return {"hbm": d["hbm_gbs"] * 1e9, "bf16": d["bf16_tflops"] * 1e12, "source": "measured"}
    return {"hbm": 6.65e12, "bf16": 1.59e15, "source": "fallback"}


def layered_config(width: int, layers: int) -> LayeredConfig:
    """Real-model layer sizes at ``width``: heads of 128, feed-forward 3 x width, low ranks of 128, latents of 512."""
    h = width // 128
    ff = 3 * width
    delta = LayerSpec(DeltaSpec(h, h // 2, 128, 128, 4), ff)
    channel = LayerSpec(DeltaSpec(h, h, 128, 128, 4, True, 128, 128), ff)
    latent = LayerSpec(LatentSpec(h, 128, 128, 1536, 512, 128 ** -0.5, 1024), ff)
    return LayeredConfig(f"layered-{width}", 32768, width, (delta, channel, delta, latent) * (layers // 4), 1e-6)


def sequential_config(width: int, layers: int) -> LayeredConfig:
    """Real-model sequential layers at ``width``: attention heads of 128 (four per key head, window 1024) beside gated linear
    heads of 128 over half the width; every fourth layer a state-space layer of twice the width (heads of 64, state 128)."""
    h, ff = width // 128, 2 * width
    rotary = RotarySpec(64, 1e6, ("yarn", 4.0, 8192.0, 32.0, 1.0, 1.14))
    pair = LayerSpec(PairSpec(AttentionSpec(h, max(1, h // 4), 128, 128 ** -0.5, rotary, 1024), GatedLinearSpec(h // 2, 128, 128, 16.0, 64),
                              1.0, 1.0), ff)
    ssd = LayerSpec(SsdSpec(width // 32, 64, 128, 8, 4, 8), ff)
    return LayeredConfig(f"sequential-{width}", 32768, width, (ssd, pair, pair, pair) * (layers // 4), 1e-6, architecture="Loduzen",
                         side_dim=64)


EXPERTS, TOP = 64, 4


def streams_config(width: int, layers: int) -> LayeredConfig:
    """Real-model layers on two residual streams at ``width``: attention heads of 128 (four per key head), three windowed layers
    and one of every earlier token in turn, all feed-forwards routed with a shared expert."""
    h = width // 128
    ff = 3 * width // 8
    routed = RoutedSpec(EXPERTS, TOP, ff, 8, ff)
    near = LayerSpec(ConvAttentionSpec(h, max(1, h // 4), 128, 128, 4, 1.0, RotarySpec(128, 1e6), 1024, 8), routed=routed)
    far = LayerSpec(BiasedAttentionSpec(h, max(1, h // 4), 128, 128, 128 ** -0.5, 32, 512, 0.1, 4096), routed=routed)
    return LayeredConfig(f"streams-{width}", 32768, width, (near, near, near, far) * (layers // 4), 1e-6, architecture="Vimelorn",
                         streams=2, embed_scale=width ** 0.5)


YARN = ("yarn", 4.0, 8192.0, 32.0, 1.0, 1.14)


def gated_config(width: int, layers: int) -> LayeredConfig:
    """Real-model layers with gated residuals at ``width``: differential attention (two maps of 64 over values of 128, four heads per
    key head, chunks of 2048), an element-wise recurrence of 1.5 x width, latent attention over every earlier token (latents of 512
    beside a rotated part of 64)."""
    h, ff = width // 128, 5 * width // 4
    pair = LayerSpec(DifferentialSpec(h, max(1, h // 4), 64, 128, 0.125, RotarySpec(64, 1e6), 0.6, 2048), ff, limit=7.0)
    gru = LayerSpec(MinGruSpec(3 * width // 2), ff, limit=7.0)
    latent = LayerSpec(LatentSpec(h, 128, 128, 0, 512, 192 ** -0.5, 0, 64, RotarySpec(64, 1e6, YARN), False), ff, limit=7.0)
    return LayeredConfig(f"gated-{width}", 32768, width, (pair, gru, pair, latent) * (layers // 4), 1e-6, architecture="Fovunex",
                         embed_scale=1.0)


def experts_config(width: int, layers: int) -> ModelConfig:
    h = width // 128
    return ModelConfig(name=f"experts-{width}", family="gqa_moe", num_layers=layers, hidden_size=width, num_q_heads=h,
                       num_kv_heads=max(1, h // 4), head_dim=128, intermediate_size=width // 4, vocab_size=32768, rope_theta=1e6,
                       qk_norm=True, num_experts=EXPERTS, experts_per_token=TOP, moe_intermediate_size=width // 4,
                       shared_intermediate_size=width // 4, quant=QuantSpec("none", 16, 0))


def hybrid_config(width: int, layers: int) -> ModelConfig:
    h = width // 128
    return ModelConfig(name=f"hybrid-{width}", family="qwen3_5", num_layers=layers, hidden_size=width, num_q_heads=h,
                       num_kv_heads=max(1, h // 4), head_dim=128, intermediate_size=2 * width, vocab_size=32768, rope_theta=1e7,
                       rotary_dim=64, qk_norm=True, zero_centered_norm=True, gdn_interval=4, gdn_k_heads=h // 2, gdn_v_heads=h,
                       attn_output_gate=True, quant=QuantSpec("none", 16, 0))


# ------------------------------------------------------------------ kernels
def _segments(requests: int, tokens: int, pos0: int) -> K.GdnSegments:
    i32 = dict(dtype=torch.int32, device=DEV)
    return K.GdnSegments(torch.arange(requests, **i32) * tokens, torch.full((requests,), tokens, **i32),
                         torch.arange(requests, **i32), torch.full((requests,), pos0, **i32), requests)


def _line(name: str, ms: float, nbytes: float, flops: float, flop_peak: float, pk: dict) -> dict:
    roof = max(nbytes / pk["hbm"], flops / flop_peak)
    return {"kernel": name, "us": round(ms * 1e3, 1), "roofline_us": round(roof * 1e6, 1),
            "bound": "memory" if nbytes / pk["hbm"] >= flops / flop_peak else "arithmetic",
            f"fraction_of_{pk['source']}": round(roof * 1e3 / ms, 3)}


def bench_delta(requests: int, tokens: int, heads: int, key_heads: int, channel: bool, flush, pk) -> list[dict]:
    d, T, H, G = 128, requests * tokens, heads, key_heads
    C = 2 * G * d + H * d
    bf = dict(dtype=torch.bfloat16, device=DEV)
    seg = _segments(requests, tokens, 5)
    proj = torch.randn(T, C, device=DEV).to(torch.bfloat16)
    conv_w = torch.randn(4, C, device=DEV) * 0.3
    conv_state = torch.zeros(requests, 3, C, **bf)
    state = torch.randn(requests, H, d, d, device=DEV) * 0.01
    out = torch.empty(T, H * d, **bf)
    b, z = torch.randn(T, H, **bf), torch.randn(T, H * d, **bf)
    a = torch.randn(T, H * d if channel else H, **bf)
    dt = torch.zeros(H * d if channel else H, device=DEV)
    a_log, norm_w = torch.full((H,), -2.0, device=DEV), torch.ones(d, device=DEV)
    sc = K.RecurrenceScratch(T, [(H, G, d, d, channel)], torch.bfloat16, DEV)
    decode = tokens == 1
    prep = timeit_graph(lambda: K.delta_prepare(proj, b, a, conv_w, conv_state, a_log, dt, seg, sc, H, G, d, d), flush, launches=5)
    walk = timeit_graph(lambda: K.delta_walk(z, norm_w, state, seg, out, sc, G, d, 1e-6, channel, channel, decode), flush,
                        launches=5)
    kind = "channel" if channel else "head"
    shape = f"{requests} x {tokens} tokens, {H} heads"
    conv_io = T * C * 4 + 2 * requests * 3 * C * 2
    return [_line(f"delta_prepare per {kind} [{shape}]", prep, conv_io + T * (H + a.shape[1]) * 2, 0, 1, pk),
            _line(f"delta_walk + norm per {kind} [{shape}]", walk, 2 * state.numel() * 4 + T * (C + 2 * H * d) * 2,
                  4 * 2.0 * T * H * d * d, FP32_FLOPS, pk),
            _line(f"both per {kind} [{shape}]", prep + walk, 2 * state.numel() * 4 + conv_io + T * (2 * H * d + H + a.shape[1]) * 2,
                  4 * 2.0 * T * H * d * d, FP32_FLOPS, pk)]


def bench_gdn(requests: int, tokens: int, hv: int, hk: int, flush, pk) -> list[dict]:
    d, T = 128, requests * tokens
    C = (2 * hk + hv) * d
    seg = _segments(requests, tokens, 5)
    proj = torch.randn(T, C + hv * d + 2 * hv, device=DEV).to(torch.bfloat16)
    w = torch.randn(C, 4, device=DEV) * 0.3
    conv_state = torch.zeros(requests, 3, C, dtype=torch.bfloat16, device=DEV)
    state = torch.randn(requests, hv, d, d, device=DEV) * 0.01
    mix = torch.empty(T, C, dtype=torch.bfloat16, device=DEV)
    out = torch.empty(T, hv * d, dtype=torch.bfloat16, device=DEV)
    a_log, dt_bias, norm_w = torch.full((hv,), -2.0, device=DEV), torch.zeros(hv, device=DEV), torch.ones(d, device=DEV)
    conv = timeit_graph(lambda: K.gdn_conv(proj, w, conv_state, seg, mix), flush, launches=5)
    delta = timeit_graph(lambda: K.gdn_delta(mix, proj[:, C:C + hv * d], proj[:, C + hv * d:], a_log, dt_bias, norm_w, state,
                                             seg, out, hk, hv), flush, launches=5)
    shape = f"{requests} x {tokens} tokens, {hv} heads"
    conv_io = T * C * 4 + 2 * requests * 3 * C * 2
    return [_line(f"gdn_conv [{shape}]", conv, conv_io, 0, 1, pk),
            _line(f"gdn_conv + gdn_delta [{shape}]", conv + delta, 2 * state.numel() * 4 + conv_io + T * (2 * hv * d + 2 * hv) * 2,
                  4 * 2.0 * T * hv * d * d, FP32_FLOPS, pk),
            _line(f"gdn_delta [{shape}]", delta, 2 * state.numel() * 4 + T * (C + 2 * hv * d + 2 * hv) * 2,
                  4 * 2.0 * T * hv * d * d, FP32_FLOPS, pk)]


def bench_gated_linear(requests: int, tokens: int, heads: int, flush, pk) -> list[dict]:
    d, T, H = 128, requests * tokens, heads
    bf = dict(dtype=torch.bfloat16, device=DEV)
    seg = _segments(requests, tokens, 5)
    proj, bias = torch.randn(T, 4 * H * d + 64, **bf), torch.zeros(H * d, device=DEV)
    a, low = proj[:, 4 * H * d:], wq_pack.pack_bf16(torch.randn(H * d, 64, device=DEV) / 8)      # rank 64
    state, out = torch.randn(requests, H, d, d, device=DEV) * 0.01, torch.empty(T, H * d, **bf)
    norm_w = torch.ones(d, device=DEV)
    sc = K.RecurrenceScratch(T, [(H, H, d, d, True)], torch.bfloat16, DEV)
    prep = timeit_graph(lambda: K.gated_linear_prepare(proj, 0, H * d, 2 * H * d, a, bias, 1 / 16, seg, sc, H, d, d, low, 64), flush,
                        launches=5)
    walk = timeit_graph(lambda: K.gated_linear_walk(proj[:, 3 * H * d:4 * H * d], norm_w, state, seg, out, sc, d, 1e-6, tokens == 1), flush, launches=5)
    shape = f"{requests} x {tokens} tokens, {H} heads of 128"
    return [_line(f"gated_linear_prepare with decay logits [{shape}]", prep, T * (3 * H * d + 64) * 2, 0, 1, pk),
            _line(f"gated_linear_walk + norm [{shape}]", walk, 2 * state.numel() * 4 + T * (5 * H * d + 64) * 2, 3 * 2.0 * T * H * d * d, FP32_FLOPS, pk),
            _line(f"gated linear both [{shape}]", prep + walk, 2 * state.numel() * 4 + T * (5 * H * d + 64) * 2, 3 * 2.0 * T * H * d * d, FP32_FLOPS, pk)]


def bench_ssd(requests: int, tokens: int, heads: int, groups: int, flush, pk) -> list[dict]:
    P, N, T, H, G = 64, 128, requests * tokens, heads, groups
    C = H * P + 2 * G * N
    bf = dict(dtype=torch.bfloat16, device=DEV)
    seg = _segments(requests, tokens, 5)
    proj, z, dt = torch.randn(T, C, **bf), torch.randn(T, H * P, **bf), torch.randn(T, H, **bf)
    conv_w, conv_b, conv_state = torch.randn(4, C, device=DEV) * 0.3, torch.zeros(C, device=DEV), torch.zeros(requests, 3, C, **bf)
    state, out = torch.randn(requests, H, P, N, device=DEV) * 0.01, torch.empty(T, H * P, **bf)
    a_log, dt_bias, D, norm_w = torch.full((H,), -2.0, device=DEV), torch.zeros(H, device=DEV), torch.ones(H, device=DEV), torch.ones(H * P, device=DEV)
    sc = K.RecurrenceScratch(T, [(H, G, N, P, False)], torch.bfloat16, DEV)
    prep = timeit_graph(lambda: K.ssd_prepare(proj, dt, conv_w, conv_b, conv_state, a_log, dt_bias, seg, sc, H, G, N, P), flush, launches=5)
    walk = timeit_graph(lambda: K.ssd_walk(z, D, norm_w, G, state, seg, out, sc, G, N, 1e-6, tokens == 1), flush, launches=5)
    shape = f"{requests} x {tokens} tokens, {H} heads of 64, state 128"
    conv_io = T * C * 4 + 2 * requests * 3 * C * 2
    return [_line(f"ssd_prepare [{shape}]", prep, conv_io + T * H * 2, 0, 1, pk),
            _line(f"ssd_walk + norm [{shape}]", walk, 2 * state.numel() * 4 + T * (C + 2 * H * P) * 2, 3 * 2.0 * T * H * P * N, FP32_FLOPS, pk),
            _line(f"ssd both [{shape}]", prep + walk, 2 * state.numel() * 4 + conv_io + T * (2 * H * P + H) * 2, 3 * 2.0 * T * H * P * N,
                  FP32_FLOPS, pk)]


def bench_gqa(requests: int, tokens: int, ctx: int, heads: int, kv_heads: int, window: int, flush, pk) -> list[dict]:
    d, T, per = 128, requests * tokens, -(-ctx // 16)
    bf = dict(dtype=torch.bfloat16, device=DEV)
    cache = torch.randn(requests * per + 1, kv_heads, 2, 16, d, **bf)
    table = (torch.randperm(requests * per, device=DEV).to(torch.int32) + 1).view(requests, per)
    x, q, out = torch.randn(T, (heads + kv_heads) * d, **bf), torch.empty(T, heads * d, **bf), torch.empty(T, heads * d, **bf)
    qn, freq = torch.ones(d, device=DEV), torch.rand(32, device=DEV)
    seg = _segments(requests, tokens, ctx - tokens)
    pos = torch.arange(ctx - tokens, ctx, device=DEV, dtype=torch.int32).repeat(requests)
    slots = (table.long().gather(1, (pos.view(requests, tokens) // 16).long()) * 16 + pos.view(requests, tokens) % 16).to(torch.int32).view(-1)
    prep = timeit_graph(lambda: K.gqa_prepare(x, 0, heads * d, qn, qn, freq, 1.1, pos, slots, q, cache, heads, d, 1e-6), flush, launches=5)
    ms = timeit_graph(lambda: K.gqa_attention(q, cache, table, seg, out, heads, d, window, 0.09, 0.0, decode=tokens == 1), flush, launches=5)
    pairs = requests * _visible(tokens, ctx, window)
    keys = requests * (min(ctx, window + tokens - 1) if window else ctx)
    shape = f"{requests} x {tokens} at {ctx}, window {window}, {heads}/{kv_heads} heads"
    return [_line(f"gqa_prepare [{shape}]", prep, T * (2 * heads + 3 * kv_heads) * d * 2, 0, 1, pk),
            _line(f"gqa_attention [{shape}]", ms, keys * kv_heads * 2 * d * 2 + 2 * T * heads * d * 2, 4.0 * pairs * heads * d, pk["bf16"], pk)]


def bench_sequential_rows(m: int, width: int, side: int, flush, pk) -> list[dict]:
    """The gated product, the side input's steps and the fused norm, beside their plain counterparts."""
    ff = 2 * width
    bf = dict(dtype=torch.bfloat16, device=DEV)
    h, x = torch.randn(m, width, **bf), torch.randn(m, width, device=DEV)
    w = wq_pack.swiglu_interleave(wq_pack.pack_bf16(torch.randn(2 * ff, width, device=DEV) * 0.02))
    act, nw = torch.empty(m, ff, **bf), torch.ones(width, device=DEV)
    glu = timeit_graph(lambda: K.wide_gemm(h, w, act, glu="gelu"), flush, launches=5)
    silu = timeit_graph(lambda: K.wq_gemm_act(h, w, out=act), flush, launches=5)
    gate, table = torch.randn(side, width, **bf), torch.randn(4096, 8 * side, **bf)
    ids, g = torch.randint(0, 4096, (m,), device=DEV, dtype=torch.int32), torch.zeros(m, -(-side // 64) * 64, **bf)
    proj, y = wq_pack.pack_bf16(torch.zeros(width, g.shape[1], **bf)), torch.randn(m, width, **bf)
    si = timeit_graph(lambda: K.side_input(x, gate, ids, table, side, proj, nw, 1e-6, nw, h, g, y), flush, launches=5)
    add = timeit_graph(lambda: K.add_norm_rows(y, nw, x, 1e-6, nw, h), flush, launches=5)
    rn = timeit_graph(lambda: K.row_norm(x, nw, h, 1e-6), flush, launches=5)
    K.workspace(torch.device(DEV)).check_status()
    flops = 2.0 * m * 2 * ff * width
    nbytes = (2 * ff * width + m * (width + ff)) * 2
    return [_line(f"wide_gemm gate/up (gelu) [{m} x {2 * ff} x {width}]", glu, nbytes, flops, pk["bf16"], pk),
            _line("wq_gemm_act bf16 (silu), same shape", silu, nbytes, flops, pk["bf16"], pk),
            _line(f"side_input [{m} x {side} x {width}]", si, m * width * 10 + 4 * side * width + m * side * 2, 4.0 * m * side * width,
                  pk["bf16"], pk),
            _line(f"add_norm_rows [{m} x {width}]", add, m * width * 12, 0, 1, pk),
            _line(f"row_norm fp32 in [{m} x {width}]", rn, m * width * 6, 0, 1, pk)]


def _visible(tokens: int, ctx: int, window: int, keep: int = 0) -> int:
    """Keys seen by the ``tokens`` last positions of a context of ``ctx`` tokens."""
    return sum(min(p + 1, window + keep) if window else p + 1 for p in range(ctx - tokens, ctx))


def bench_qkv(requests: int, tokens: int, ctx: int, heads: int, kv_heads: int, flush, pk) -> list[dict]:
    """Preparation of both attentions and the attentions themselves, beside the rotation kernel of the int8-cached decoders."""
    d, T, per = 128, requests * tokens, -(-ctx // 16)
    bf = dict(dtype=torch.bfloat16, device=DEV)
    C = (heads + 2 * kv_heads) * d
    offs = (0, heads * d, (heads + kv_heads) * d)
    cache = torch.randn(requests * per + 1, kv_heads, 2, 16, d, **bf)
    table = (torch.randperm(requests * per, device=DEV).to(torch.int32) + 1).view(requests, per)
    x, q, out = torch.randn(T, C, **bf), torch.empty(T, heads * d, **bf), torch.empty(T, heads * d, **bf)
    seg = _segments(requests, tokens, ctx - tokens)
    pos = torch.arange(ctx - tokens, ctx, device=DEV, dtype=torch.int32).repeat(requests)
    slots = (table.long().gather(1, (pos.view(requests, tokens) // 16).long()) * 16 + pos.view(requests, tokens) % 16).to(torch.int32).view(-1)
    conv_w, state, freq = torch.randn(4, C, device=DEV) * 0.5, torch.zeros(requests, 3, C, **bf), torch.rand(2, 64, device=DEV)
    freq[1] = 0
    qn, kn, bias = torch.ones(heads * d, device=DEV), torch.ones(kv_heads * d, device=DEV), torch.randn(513, heads, device=DEV)
    decode = tokens == 1
    cv = timeit_graph(lambda: K.conv_qkv(x, offs, conv_w, state, freq, pos, slots, seg, q, cache, heads, d, d, 1e-6), flush, launches=5)
    nm = timeit_graph(lambda: K.norm_qkv(x, offs, qn, kn, pos, slots, q, cache, heads, d, d, 1e-6, (0.1, 4096)), flush, launches=5)
    near = timeit_graph(lambda: K.gqa_attention(q, cache, table, seg, out, heads, d, 1024, 0.09, decode=decode, keep=8), flush, launches=5)
    far = timeit_graph(lambda: K.gqa_attention(q, cache, table, seg, out, heads, d, 0, 0.09, decode=decode, bias=bias), flush, launches=5)
    blob = torch.zeros(requests * per + 1, kv_heads, K.kv_blob_bytes(d, 8, 8), dtype=torch.uint8, device=DEV)
    q8, w = torch.empty(T, heads, d, **bf), torch.ones(d, **bf)
    rope = timeit_graph(lambda: K.rope_kv_write(x, q8, blob, pos, slots, freq[0], heads, kv_heads, d, 8, 8, w, w), flush, launches=5)
    shape = f"{requests} x {tokens} at {ctx}, {heads}/{kv_heads} heads"
    io = T * 2 * C * 2
    attn = lambda window, keep: (requests * (min(ctx, window + keep + tokens - 1) if window else ctx) * kv_heads * 2 * d * 2      # noqa: E731
                                 + 2 * T * heads * d * 2, 4.0 * requests * _visible(tokens, ctx, window, keep) * heads * d)
    return [_line(f"conv_qkv [{shape}]", cv, io + 2 * requests * 3 * C * 2, 0, 1, pk), _line(f"norm_qkv [{shape}]", nm, io, 0, 1, pk),
            _line(f"rope_kv_write int8 with norms [{shape}]", rope, T * (C + heads * d) * 2 + T * 2 * kv_heads * (d + 16), 0, 1, pk),
            _line(f"gqa_attention window 1024, 8 kept [{shape}]", near, *attn(1024, 8), pk["bf16"], pk),
            _line(f"gqa_attention biased [{shape}]", far, *attn(0, 0), pk["bf16"], pk)]


def bench_streams(m: int, width: int, flush, pk) -> list[dict]:
    """A step between two sublayers on two streams, with a plain and a routed result, beside the norm that adds a residual and the
    combination of the other routed decoders."""
    S, top = 2, TOP
    bf = dict(dtype=torch.bfloat16, device=DEV)
    x, h, y, w = torch.randn(m, S, width, device=DEV), torch.randn(m, width, **bf), torch.randn(m, width, **bf), torch.ones(width, device=DEV)
    mix, out = torch.eye(S, device=DEV), torch.full((S,), 1e-3, device=DEV)
    rows = torch.randn(m * top, width, **bf)
    routes = K.RoutedResult(rows, torch.randperm(m * top, device=DEV).to(torch.int32), torch.rand(m * top, device=DEV),
                            torch.zeros(m, device=DEV), torch.randn(m, 1, device=DEV), top)
    plain = timeit_graph(lambda: K.stream_step(x, y, mix, out, h, 1e-6, out, w), flush, launches=5)
    full = timeit_graph(lambda: K.stream_step(x, y, mix, out, h, 1e-6, out, w, routes), flush, launches=5)
    res, wb = torch.randn(m, width, **bf), torch.ones(width, **bf)
    norm = timeit_graph(lambda: K.rmsnorm(y, wb, 1e-6, out=h, residual=res), flush, launches=5)
    sc = K.MoeScratch(m, top, width, 128, EXPERTS, 32, DEV)
    sc.route_pos.copy_(routes.pos.view(m, top))
    sc.topk_w.copy_(routes.weight.view(m, top))
    comb = timeit_graph(lambda: K.moe_combine(rows, sc, m, y, res), flush, launches=5)
    row = m * width
    return [_line(f"stream_step [{m} x {S} x {width}]", plain, row * (8 * S + 4), 0, 1, pk),
            _line(f"stream_step routed, top {top} [{m} x {S} x {width}]", full, row * (8 * S + 4 + 2 * top), 0, 1, pk),
            _line(f"rmsnorm + residual bf16 [{m} x {width}]", norm, row * 8, 0, 1, pk),
            _line(f"moe_combine + residual, top {top} [{m} x {width}]", comb, row * (4 + 2 * top), 0, 1, pk)]


def bench_experts(m: int, width: int, flush, pk) -> list[dict]:
    """Routing and the products of all experts, beside those of the gated experts of equal size."""
    from ..models.moe import MoeLayer, stack_experts
    E, top, bf = EXPERTS, TOP, dict(dtype=torch.bfloat16, device=DEV)
    ff, gf = 3 * width // 8, width // 4
    h, z, corr = torch.randn(m, width, **bf), torch.randn(m, E, device=DEV), torch.zeros(E, device=DEV)
    sc = K.ScoredScratch(m, top, E, width, width, torch.bfloat16, DEV)
    stack = lambda n, k: wq_pack.PackedWeight(wq_pack.FMT_BF16, n, k, k, torch.randn(E, n, k, **bf) * 0.02, None)      # noqa: E731
    up, down, act = stack(ff, width), stack(width, ff), torch.zeros(m * top, ff, **bf)
    route = timeit_graph(lambda: K.scored_route(z, corr, h, width, E, top, sc), flush, launches=5)
    mb = K.scored_route(z, corr, h, width, E, top, sc)
    used = len(set(sc.ids[:m * top].tolist()))
    u = timeit_graph(lambda: K.grouped_gemm(sc.xs, up, act, sc, m * top, mb, relu2=True), flush, launches=5)
    dn = timeit_graph(lambda: K.grouped_gemm(act, down, sc.ys, sc, m * top, mb), flush, launches=5)
    del up, down
    gu, cs, ms = stack_experts([wq_pack.pack_bf16(torch.randn(2 * gf, width, **bf) * 0.02) for _ in range(E)])
    dg, ds, dm = stack_experts([wq_pack.pack_bf16(torch.randn(width, gf, **bf) * 0.02) for _ in range(E)])
    layer = MoeLayer(wq_pack.pack_bf16(torch.randn(E, width, **bf)), gu, dg, (cs, ms, ds, dm), E, top, 0, E)
    layer.fuse_activation()
    old = layer.ensure_scratch(m, width, torch.device(DEV))
    zb = z.to(torch.bfloat16)
    r2 = timeit_graph(lambda: K.moe_route(zb, h, top, old), flush, launches=5)
    K.moe_route(zb, h, top, old)
    g2 = timeit_graph(lambda: K.wq_gemm_grouped(old.xs, layer.gate_up, old.act, m * top, old, cs, ms, swiglu=True), flush, launches=5)
    d2 = timeit_graph(lambda: K.wq_gemm_grouped(old.act, layer.down, old.y, m * top, old, ds, dm), flush, launches=5)
    K.workspace(torch.device(DEV)).check_status()
    R = m * top
    io = lambda n, k: (used * n * k + R * (n + k)) * 2                                   # noqa: E731
    shape = f"{m} tokens, {top} of {E}, width {width}"
    return [_line(f"scored_route [{shape}]", route, m * E * 4 + (m + R) * width * 2, 0, 1, pk),
            _line(f"moe_route [{shape}]", r2, m * E * 2 + (m + R) * width * 2, 0, 1, pk),
            _line(f"grouped up relu^2 [{shape}, {ff}]", u, io(ff, width), 2.0 * R * ff * width, pk["bf16"], pk),
            _line(f"wq_gemm_grouped gate/up bf16 [{shape}, {gf}]", g2, (used * 2 * gf * width + R * (gf + width)) * 2,
                  4.0 * R * gf * width, pk["bf16"], pk),
            _line(f"grouped down [{shape}, {ff}]", dn, io(width, ff), 2.0 * R * ff * width, pk["bf16"], pk),
            _line(f"wq_gemm_grouped down bf16 [{shape}, {gf}]", d2, io(width, gf), 2.0 * R * gf * width, pk["bf16"], pk)]


def bench_latent(requests: int, tokens: int, ctx: int, heads: int, rank: int, window: int, flush, pk) -> list[dict]:
    T, per = requests * tokens, -(-ctx // 16)
    bf = dict(dtype=torch.bfloat16, device=DEV)
    cache = torch.randn(requests * per + 1, 16, rank, **bf)
    table = (torch.randperm(requests * per, device=DEV).to(torch.int32) + 1).view(requests, per)
    q, out, gate = torch.randn(T, heads * rank, **bf) * 0.05, torch.empty(T, heads * rank, **bf), torch.randn(T, heads, **bf)
    seg = _segments(requests, tokens, ctx - tokens)
    ms = timeit_graph(lambda: K.latent_attention(q, gate, cache, table, seg, out, heads, window, 0.1, decode=tokens == 1), flush,
                      launches=5)
    K.workspace(torch.device(DEV)).check_status()
    pairs = requests * _visible(tokens, ctx, window)
    keys = requests * (min(ctx, window + tokens) if window else ctx)
    return [_line(f"latent_attn [{requests} x {tokens} at {ctx}, window {window}, {heads} heads, rank {rank}]", ms,
                  keys * rank * 2 + 2 * T * heads * rank * 2, 4.0 * pairs * heads * rank, pk["bf16"], pk)]


def _paged(requests: int, tokens: int, ctx: int):
    """Shuffled pages, positions and cache rows of the last ``tokens`` of ``ctx`` tokens of every request."""
    per = -(-ctx // 16)
    table = (torch.randperm(requests * per, device=DEV).to(torch.int32) + 1).view(requests, per)
    pos = torch.arange(ctx - tokens, ctx, device=DEV, dtype=torch.int32).repeat(requests)
    at = pos.view(requests, tokens)
    return table, pos, (table.long().gather(1, (at // 16).long()) * 16 + at % 16).to(torch.int32).view(-1)


def bench_rotated(requests: int, tokens: int, ctx: int, heads: int, flush, pk) -> list[dict]:
    """Latents of 512 beside a rotated part of 64, and the same attention over latents alone."""
    rank, rot, T = 512, 64, requests * tokens
    spec = LatentSpec(heads, 128, 128, 0, rank, 1.0, 0, rot, RotarySpec(rot, 1e6, YARN), False)
    rp, rv = spec.row_padded, spec.rank_padded
    bf = dict(dtype=torch.bfloat16, device=DEV)
    table, pos, slots = _paged(requests, tokens, ctx)
    seg = _segments(requests, tokens, ctx - tokens)
    cache = torch.randn(table.numel() + 1, 16, rp, **bf)
    proj, cn, freq = torch.randn(T, heads * rot + rank + rot, **bf), torch.ones(rank, device=DEV), spec.rotary.split_table().to(DEV)
    q, out = torch.randn(T, heads * rp, **bf) * 0.05, torch.empty(T, heads * rv, **bf)
    prep = timeit_graph(lambda: K.latent_prepare(proj, heads * rot, rank, cn, cache, slots, 1e-6,
                                                 rotated=(0, heads * rot + rank, rank, freq, 1.14, pos, q, heads)), flush, launches=5)
    decode = tokens == 1
    ms = timeit_graph(lambda: K.latent_attention(q, None, cache, table, seg, out, heads, 0, 0.1, decode=decode), flush, launches=5)
    pairs, keys = requests * _visible(tokens, ctx, 0), requests * ctx
    shape = f"{requests} x {tokens} at {ctx}, {heads} heads"
    res = [_line(f"latent_prepare rotated [{shape}]", prep, T * 2 * (2 * heads * rot + 2 * (rank + rot)), 0, 1, pk),
           _line(f"latent_attn rank 512 + 64 rotated [{shape}]", ms, keys * rp * 2 + T * heads * (rp + rv) * 2, 2.0 * pairs * heads * (rp + rv), pk["bf16"], pk)]
    del q, out, cache
    lowq, cq = torch.randn(T, 1536 + rank, **bf), torch.empty(T, 1536, **bf)
    plain = torch.randn(table.numel() + 1, 16, rank, **bf)
    qn = torch.ones(1536, device=DEV)
    lp = timeit_graph(lambda: K.latent_prepare(lowq, 1536, rank, cn, plain, slots, 1e-6, low=(0, 1536, qn, cq)), flush, launches=5)
    del plain
    return res + [_line(f"latent_prepare low-rank queries [{shape}]", lp, T * 4 * (1536 + rank), 0, 1, pk),
                  *bench_latent(requests, tokens, ctx, heads, rank, 0, flush, pk)]


def bench_pair(requests: int, tokens: int, ctx: int, heads: int, kv_heads: int, flush, pk) -> list[dict]:
    """Differential attention in chunks of 2048 and its preparation, beside attention with one map over as many keys."""
    d, e, chunk, T = 64, 128, 2048, requests * tokens
    bf = dict(dtype=torch.bfloat16, device=DEV)
    table, pos, slots = _paged(requests, tokens, ctx)
    seg = _segments(requests, tokens, ctx - tokens)
    cache = torch.randn(table.numel() + 1, kv_heads, 2, 16, 128, **bf)
    offs = (0, heads * 128, (heads + kv_heads) * 128)
    x, q, out, gate = torch.randn(T, (heads + 2 * kv_heads) * 128, **bf), torch.empty(T, heads * 128, **bf), torch.empty(T, heads * e, **bf), torch.randn(T, heads * e, **bf)
    w, freq = torch.ones(d, device=DEV), RotarySpec(d, 1e6).split_table().to(DEV)
    decode = tokens == 1
    prep = timeit_graph(lambda: K.head_qkv(x, offs, w, w, freq, pos, slots, q, cache, heads, d, e, 1e-6, 2), flush, launches=5)
    ms = timeit_graph(lambda: K.gqa_attention(q, cache, table, seg, out, heads, e, 0, 0.125, out_scale=0.4, decode=decode, chunk=chunk,
                                              pair=(gate, 0.8, 1e-6)), flush, launches=5)
    one = timeit_graph(lambda: K.gqa_attention(q, cache, table, seg, out, heads, e, 0, 0.09, decode=decode, chunk=chunk), flush, launches=5)
    pairs = requests * sum(p % chunk + 1 for p in range(ctx - tokens, ctx))
    lo = (ctx - tokens) // chunk * chunk
    kv = requests * (ctx - lo) * kv_heads * 2 * 128 * 2
    shape = f"{requests} x {tokens} at {ctx}, {heads}/{kv_heads} heads"
    return [_line(f"head_qkv two maps [{shape}]", prep, T * 2 * (heads + 2 * kv_heads) * 128 * 2, 0, 1, pk),
            _line(f"gqa_attention differential [{shape}]", ms, kv + T * heads * 3 * 128 * 2, 2.0 * pairs * heads * 2 * (d + e), pk["bf16"], pk),
            _line(f"gqa_attention one map, same keys [{shape}]", one, kv + T * heads * 2 * 128 * 2, 4.0 * pairs * heads * 128, pk["bf16"], pk),
            *bench_qkv(requests, tokens, ctx, heads, kv_heads, flush, pk)[:3]]


def bench_mingru(requests: int, tokens: int, width: int, flush, pk) -> list[dict]:
    T = requests * tokens
    bf = dict(dtype=torch.bfloat16, device=DEV)
    x, out, bias, state = torch.randn(T, 3 * width, **bf), torch.empty(T, width, **bf), torch.zeros(2, width, device=DEV), torch.zeros(requests, width, device=DEV)
    seg = _segments(requests, tokens, 5)
    ms = timeit_graph(lambda: K.mingru(x, 0, width, 2 * width, bias, state, seg, out), flush, launches=5)
    return [_line(f"mingru [{requests} x {tokens} tokens, width {width}]", ms, T * width * 8 + requests * width * 8, 0, 1, pk)]


def bench_gated_products(m: int, width: int, flush, pk) -> list[dict]:
    """Products whose epilogues gate, clamp and add, beside the plain ones of the same shapes; the entry of a loop's later pass."""
    ff = 2 * width
    bf = dict(dtype=torch.bfloat16, device=DEV)
    h, x = torch.randn(m, width, **bf), torch.randn(m, width, device=DEV)
    w = wq_pack.swiglu_interleave(wq_pack.pack_bf16(torch.randn(2 * ff, width, **bf) * 0.02))
    both = wq_pack.PackedWeight(w.fmt, w.n + width, w.k, w.k, torch.cat([w.codes, torch.randn(width, width, **bf) * 0.02]), None, act_interleaved=True)
    plain = wq_pack.pack_bf16(both.codes)
    act, rg, y = torch.empty(m, ff, **bf), torch.randn(m, width, **bf), torch.empty(m, both.n, **bf)
    down, bias, yo = wq_pack.pack_bf16(torch.randn(width, ff, **bf) * 0.02), torch.zeros(width, device=DEV), torch.empty(m, width, **bf)
    table, ids, nw = torch.randn(4096, width, **bf), torch.randint(0, 4096, (m,), device=DEV, dtype=torch.int32), torch.ones(width, device=DEV)
    out = []
    for name, fn, n, k, extra in (
            ("wide_gemm [gate, up | residual gate] (clamped)", lambda: K.wide_gemm(h, both, act, glu="clamped", limit=7.0, rest=rg, split=2 * ff), both.n, width, -m * ff * 2),
            ("wq_gemm bf16, same shape", lambda: K.wq_gemm(h, plain, out=y), both.n, width, 0),
            ("wide_gemm down (gated fp32 residual)", lambda: K.wide_gemm(act, down, x, residual=x, gate=(rg, bias)), width, ff, m * width * 8),
            ("wq_gemm bf16, same shape", lambda: K.wq_gemm(act, down, out=yo), width, ff, 0)):
        out.append(_line(f"{name} [{m} x {n} x {k}]", timeit_graph(fn, flush, launches=5), (n * k + m * (n + k)) * 2 + extra, 2.0 * m * n * k, pk["bf16"], pk))
    again = timeit_graph(lambda: K.embed_rows(ids, table, nw, x, h, 1e-6, 0.0, add=True), flush, launches=5)
    rn = timeit_graph(lambda: K.row_norm(x, nw, h, 1e-6), flush, launches=5)
    K.workspace(torch.device(DEV)).check_status()
    return out + [_line(f"embedding added + norm [{m} x {width}]", again, m * width * 12, 0, 1, pk),
                  _line(f"row_norm fp32 in [{m} x {width}]", rn, m * width * 6, 0, 1, pk)]


def bench_paged(requests: int, tokens: int, ctx: int, hq: int, hkv: int, flush, pk) -> list[dict]:
    from ..ops import eager
    d, T, per = 128, requests * tokens, -(-ctx // 16)
    blob = K.kv_blob_bytes(d, 8, 8)
    cache = torch.randint(0, 255, (requests * per + 1, hkv, blob), dtype=torch.uint8, device=DEV)
    lay = eager.blob_layout(d, 8, 8)
    one = torch.full((64,), 0.01, device=DEV).view(torch.uint8)
    cache[:, :, lay["k_scale"]:lay["v_code"]] = one
    cache[:, :, lay["v_scale"]:] = one
    table = (torch.randperm(requests * per, device=DEV).to(torch.int32) + 1).view(requests, per)
    q = torch.randn(T, hq, d, device=DEV, dtype=torch.bfloat16)
    out = torch.empty_like(q)
    qb = 16 // (hq // hkv)
    blocks = [(r, r * tokens + i, min(qb, tokens - i), ctx - tokens + i + 1) for r in range(requests) for i in range(0, tokens, qb)]
    rb = torch.tensor(blocks, dtype=torch.int32, device=DEV).t().contiguous()
    splits = max(1, min(32, 296 // (len(blocks) * hkv)))
    ms = timeit_graph(lambda: K.paged_attention(q, out, cache, table, rb[0], rb[1], rb[2], rb[3], hq, hkv, d, 8, 8, splits=splits),
                      flush, launches=5)
    K.workspace(torch.device(DEV)).check_status()
    pairs = requests * _visible(tokens, ctx, 0)
    return [_line(f"paged_attn int8 [{requests} x {tokens} at {ctx}, {hq}/{hkv} heads]", ms,
                  requests * per * hkv * blob + 2 * T * hq * d * 2, 4.0 * pairs * hq * d, pk["bf16"], pk)]


def bench_products(m: int, width: int, flush, pk) -> list[dict]:
    """The two large products of a layer with their fused epilogues, beside the same shapes through the plain GEMM."""
    h, ff = width // 128, 3 * width
    split = 4 * width + 2 * h
    x = torch.randn(m, width, device=DEV).to(torch.bfloat16)
    w_in = wq_pack.pack_bf16(torch.randn(split + ff, width, device=DEV) * 0.02)
    w_out = wq_pack.pack_bf16(torch.randn(width, width + ff, device=DEV) * 0.02)
    bf = dict(dtype=torch.bfloat16, device=DEV)
    proj, operand = torch.empty(m, split, **bf), torch.randn(m, width + ff, **bf)
    res, y_in, y_out = torch.zeros(m, width, device=DEV), torch.empty(m, split + ff, **bf), torch.empty(m, width, **bf)
    out = []
    for name, fn, n, k, extra in (
            ("wide_gemm in (relu^2, two outputs)", lambda: K.wide_gemm(x, w_in, proj, relu2=operand[:, width:], split=split), w_in.n, w_in.k, 0),
            ("wq_gemm bf16, same shape", lambda: K.wq_gemm(x, w_in, out=y_in), w_in.n, w_in.k, 0),
            ("wide_gemm out (fp32 residual)", lambda: K.wide_gemm(operand, w_out, res, residual=res), w_out.n, w_out.k, m * width * 6),
            ("wq_gemm bf16, same shape", lambda: K.wq_gemm(operand, w_out, out=y_out), w_out.n, w_out.k, 0)):
        ms = timeit_graph(fn, flush, launches=5)
        out.append(_line(f"{name} [{m} x {n} x {k}]", ms, (n * k + m * (n + k)) * 2 + extra, 2.0 * m * n * k, pk["bf16"], pk))
    K.workspace(torch.device(DEV)).check_status()
    return out


def bench_rows(m: int, width: int, flush, pk) -> list[dict]:
    x, w = torch.randn(m, width, device=DEV), torch.ones(width, device=DEV)
    h = torch.empty(m, width, dtype=torch.bfloat16, device=DEV)
    xb, wb = x.to(torch.bfloat16), w.to(torch.bfloat16)
    a = timeit_graph(lambda: K.row_norm(x, w, h, 1e-6), flush, launches=5)
    b = timeit_graph(lambda: K.rmsnorm(xb, wb, 1e-6, out=h), flush, launches=5)
    return [_line(f"row_norm fp32 in [{m} x {width}]", a, m * width * 6, 0, 1, pk),
            _line(f"rmsnorm bf16 in [{m} x {width}]", b, m * width * 4, 0, 1, pk)]


def kernels(width: int = 4096) -> list[dict]:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=DEV)
    pk = peaks()
    h = width // 128
    out = []
    for requests, tokens in ((256, 1), (8, 1024), (1, 4096)):
        out += bench_delta(requests, tokens, h, h // 2, False, flush, pk)
        out += bench_delta(requests, tokens, h, h, True, flush, pk)
        out += bench_gdn(requests, tokens, h, h // 2, flush, pk)
    for requests, tokens, ctx in ((256, 1, 1280), (1, 1, 4096), (8, 1024, 1024), (1, 4096, 4096)):
        out += bench_latent(requests, tokens, ctx, h, 512, 1024, flush, pk)
        out += bench_paged(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
    for m in (16, 256, 4096):
        out += bench_products(m, width, flush, pk)
        out += bench_rows(m, width, flush, pk)
    return out


def sequential_kernels(width: int = 4096) -> list[dict]:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=DEV)
    pk = peaks()
    h = width // 128
    out = []
    for requests, tokens in ((256, 1), (8, 1024), (1, 4096)):
        out += bench_gated_linear(requests, tokens, h // 2, flush, pk)
        out += bench_ssd(requests, tokens, width // 32, 8, flush, pk)
        out += bench_gdn(requests, tokens, h, h // 2, flush, pk)
    for requests, tokens, ctx in ((256, 1, 1280), (1, 1, 4096), (8, 1024, 1024), (1, 4096, 4096)):
        out += bench_gqa(requests, tokens, ctx, h, max(1, h // 4), 1024, flush, pk)
        out += bench_paged(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
    for m in (16, 256, 4096):
        out += bench_sequential_rows(m, width, 64, flush, pk)
    return out


def streams_kernels(width: int = 4096) -> list[dict]:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=DEV)
    pk = peaks()
    h = width // 128
    out = []
    for requests, tokens, ctx in ((256, 1, 1280), (1, 1, 4096), (8, 1024, 1024), (1, 4096, 4096)):
        out += bench_qkv(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
        out += bench_paged(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
    for m in (16, 256, 4096):
        out += bench_streams(m, width, flush, pk)
        out += bench_experts(m, width, flush, pk)
    return out


def gated_kernels(width: int = 4096) -> list[dict]:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=DEV)
    pk = peaks()
    h = width // 128
    out = []
    for requests, tokens in ((256, 1), (8, 1024), (1, 4096)):
        out += bench_mingru(requests, tokens, 3 * width // 2, flush, pk)
        out += bench_gated_linear(requests, tokens, h // 2, flush, pk)
        out += bench_gdn(requests, tokens, h, h // 2, flush, pk)
    for requests, tokens, ctx in ((256, 1, 1280), (1, 1, 4096), (8, 1024, 1024), (1, 4096, 4096)):
        out += bench_pair(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
        out += bench_rotated(requests, tokens, ctx, h, flush, pk)
        out += bench_paged(requests, tokens, ctx, h, max(1, h // 4), flush, pk)
    for m in (16, 256, 4096):
        out += bench_gated_products(m, width, flush, pk)
    return out


# ------------------------------------------------------------------ whole models
def model_throughput(cfg, concurrency: int, prompt: int, steps: int, warmup: int = 4, budget: int = 8192) -> dict:
    """Prefill and decode rates of a random model through the serving engine."""
    import gc
    import time

    import numpy as np

    from ..executor.gpu_executor import GpuExecutor
    from ..models import registry
    from ..runtime.engine import LLMEngine
    from ..runtime.scheduler import SamplingParams, SchedulerConfig
    dev = torch.device("cuda", torch.cuda.current_device())
    defn = registry.get(cfg.family)
    weights = defn.random_weights(cfg, dev, 0)
    max_len = prompt + steps + warmup + 24
    pages = concurrency * (-(-max_len // 16)) + 8
    runner = defn.build_runner(cfg, weights, num_pages=pages, max_tokens=budget, max_requests=concurrency)
    ex = GpuExecutor(runner, max_rows=concurrency, max_prefill_tokens=budget, max_model_len=max_len)
    ex.capture_decode_graphs([concurrency])
    ex.timing = True
    eng = LLMEngine(ex, num_pages=pages, scheduler_config=SchedulerConfig(
        max_running_requests=concurrency, max_batched_tokens=budget, prefill_chunk_tokens=budget, max_model_len=max_len,
        enable_prefix_cache=False))
    rng = np.random.default_rng(1)
    rates = []
    for turn in range(2):                              # the first turn warms the prefill path up
        for p in rng.integers(0, cfg.vocab_size, size=(concurrency, prompt)).tolist():
            eng.add_request(p, SamplingParams(max_tokens=steps + warmup + 8, ignore_eos=True))
        ex.device_ms = []
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        while any(r.remaining > 1 for r in eng.scheduler.running + eng.scheduler.waiting) or eng.scheduler.waiting:
            eng.step()
        torch.cuda.synchronize()
        rates.append((concurrency * prompt / (sum(ex.device_ms) / 1e3), concurrency * prompt / (time.perf_counter() - t0)))
        for _ in range(warmup):
            eng.step()
        ex.device_ms = []
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        emitted = sum(len(eng.step()) for _ in range(steps))
        torch.cuda.synchronize()
        wall = time.perf_counter() - t0
        ms = sorted(ex.device_ms)
        launches = ex.kernel_launches_last
        while eng.has_unfinished:                      # a few more tokens end every request
            eng.step()
    runner.ws.check_status()
    out = {"model": cfg.name, "layers": cfg.num_layers, "weights_gb": round(weights.nbytes() / 1e9, 2), "concurrency": concurrency,
           "prompt": prompt, "prefill_tok_s_device": round(rates[-1][0]), "prefill_tok_s_wall": round(rates[-1][1]),
           "decode_ms_per_step": round(ms[len(ms) // 2], 3), "decode_tok_s_device": round(concurrency / ms[len(ms) // 2] * 1e3),
           "decode_tok_s_wall": round(emitted / wall), "launches_per_decode_step": launches}
    del eng, ex, runner, weights
    gc.collect()
    torch.cuda.empty_cache()
    return out


KERNELS = {"parallel": kernels, "sequential": sequential_kernels, "streams": streams_kernels, "gated": gated_kernels}
MODELS = {"parallel": (layered_config, hybrid_config), "sequential": (sequential_config, hybrid_config),
          "streams": (streams_config, experts_config), "gated": (gated_config, hybrid_config)}


def run(steps: int = 32, designs: str = "all") -> None:
    """Prints one JSON line per measurement.  ``designs``: all, or one of ``KERNELS``."""
    chosen = list(KERNELS) if designs == "all" else [designs]
    for d in chosen:
        for line in KERNELS[d]():
            print(json.dumps(line), flush=True)
    models = list(dict.fromkeys(make for d in chosen for make in MODELS[d]))
    for width, layers in ((2048, 8), (4096, 8)):
        for concurrency, prompt in ((1, 4096), (16, 1024), (256, 1024)):
            for make in models:
                print(json.dumps(model_throughput(make(width, layers), concurrency, prompt, steps)), flush=True)
