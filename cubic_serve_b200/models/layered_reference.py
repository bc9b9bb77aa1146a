"""Plain model of the layered decoders (``Bumodra``, ``Loduzen``, ``Vimelorn`` and ``Fovunex`` checkpoints): the oracle of the native runner and the
model of the eager execution mode.

Everything is written from the equations, token by token where the mechanism is a recurrence, one function per
mechanism, on the raw ``config.json`` dictionary and the checkpoint's tensors by name.  It shares no code with
``models/layered.py`` (configuration, packing) or the kernels, so that the two can be compared.  Arithmetic is done in
the dtype of ``Oracle.dtype`` (fp32 by default, fp64 for comparisons that should not see the oracle's own rounding).

``Oracle.forward`` runs one request's new tokens against its explicit state; prefill in portions, token-by-token decoding
and one pass over the whole sequence give the same logits.
"""
from __future__ import annotations

import copy
import math

import torch

from ..executor.stateful_executor import StatefulEagerExecutor


# ------------------------------------------------------------------ mechanisms
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_around_zero(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + w)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def short_conv(x: torch.Tensor, w: torch.Tensor, past: torch.Tensor,
               bias: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """Causal depthwise convolution over time (with a bias per channel) and silu.  ``x`` [n, C] new inputs, ``w`` [C, taps]
    with the current input's tap last, ``past`` [taps - 1, C] inputs before ``x``.  Returns the outputs and the new ``past``."""
    taps = w.shape[1]
    ext = torch.cat([past, x])
    out = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    for j in range(taps):
        out = out + w[:, j] * ext[j:j + x.shape[0]]
    return silu(out), ext[ext.shape[0] - (taps - 1):].clone()


def delta_step(S: torch.Tensor, q, k, v, beta, decay) -> tuple[torch.Tensor, torch.Tensor]:
    """One token of the gated delta rule for all heads.  ``S`` [H, dim, vdim]; ``q``, ``k`` [H, dim]; ``v`` [H, vdim];
    ``beta`` [H]; ``decay`` [H, dim] (a head's scalar decay repeated, or one factor per key channel)."""
    S = decay.unsqueeze(-1) * S
    held = torch.einsum("hkv,hk->hv", S, k)
    u = beta.unsqueeze(-1) * (v - held)
    S = S + k.unsqueeze(-1) * u.unsqueeze(1)
    return torch.einsum("hkv,hk->hv", S, q), S


def windowed_attention(q, k, v, first: int, window: int | None, scale: float) -> torch.Tensor:
    """Softmax attention of queries at positions ``first ..`` over keys at positions ``0 ..``: position i sees j with
    ``0 <= i - j < window``.  ``q`` [n, H, d], ``k`` [m, H, d], ``v`` [m, H, e]."""
    n, m = q.shape[0], k.shape[0]
    i = torch.arange(first, first + n).unsqueeze(1)
    j = torch.arange(m).unsqueeze(0)
    seen = (i - j) >= 0
    if window is not None:
        seen &= (i - j) < window
    s = torch.einsum("nhd,mhd->hnm", q, k) * scale
    s = s.masked_fill(~seen, float("-inf"))
    return torch.einsum("hnm,mhe->nhe", torch.softmax(s, -1), v)


def squared_relu(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0) ** 2


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    """The tanh form of gelu."""
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rotary_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(radians per position of every rotated pair, factor on cosine and sine), fp64.  With ``scaling`` (YaRN) the slow pairs
    are stretched by ``factor``, the fast ones stay, a ramp over the pair index lies between."""
    n, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def pair_of(turns: float) -> float:                    # the (doubled) index that turns this often over ``original`` tokens
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x: torch.Tensor, first: int, freq: torch.Tensor, mult: float) -> torch.Tensor:
    """Rotary positions ``first ..`` on ``x`` [n, H, d]: neighbouring channels (2 i, 2 i + 1) of the first ``2 len(freq)``."""
    n, r = x.shape[0], 2 * freq.numel()
    a = torch.arange(first, first + n, dtype=torch.float64).unsqueeze(1) * freq
    c, s = (torch.cos(a) * mult).to(x.dtype).unsqueeze(1), (torch.sin(a) * mult).to(x.dtype).unsqueeze(1)
    out = x.clone()
    u, v = x[..., 0:r:2], x[..., 1:r:2]
    out[..., 0:r:2] = u * c - v * s
    out[..., 1:r:2] = v * c + u * s
    return out


def sink_attention(q, k, v, first: int, window: int | None, scale: float) -> torch.Tensor:
    """Like ``windowed_attention`` with one more score of zero in the softmax that has no value, and fewer key heads: query
    head h uses key head ``h // (H / G)``.  ``q`` [n, H, d], ``k`` [m, G, d], ``v`` [m, G, e]."""
    n, H, m = q.shape[0], q.shape[1], k.shape[0]
    rep = torch.arange(H) // (H // k.shape[1])
    i, j = torch.arange(first, first + n).unsqueeze(1), torch.arange(m).unsqueeze(0)
    seen = (i - j) >= 0
    if window is not None:
        seen &= (i - j) < window
    s = torch.einsum("nhd,mhd->hnm", q, k[:, rep]) * scale
    s = s.masked_fill(~seen, float("-inf"))
    s = torch.cat([s, torch.zeros(H, n, 1, dtype=s.dtype)], -1)
    return torch.einsum("hnm,mhe->nhe", torch.softmax(s, -1)[..., :m], v[:, rep])


def plain_short_conv(x: torch.Tensor, w: torch.Tensor, past: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """``short_conv`` without the activation."""
    taps, n = w.shape[1], x.shape[0]
    ext = torch.cat([past, x])
    out = sum(w[:, j] * ext[j:j + n] for j in range(taps))
    return out, ext[ext.shape[0] - (taps - 1):].clone()


def rotate_halves(x: torch.Tensor, first: int, dims: int, base: float) -> torch.Tensor:
    """Rotary positions ``first ..`` on ``x`` [n, H, d]: channel i of the first ``dims`` turns with channel ``i + dims / 2``."""
    n, half = x.shape[0], dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = torch.arange(first, first + n, dtype=torch.float64).view(n, 1, 1) * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def kept_window(first: int, n: int, m: int, size: int | None, keep: int) -> torch.Tensor:
    """[n, m] which of m keys the queries at positions ``first ..`` see: the last ``size`` and the first ``keep``."""
    i, j = torch.arange(first, first + n).unsqueeze(1), torch.arange(m).unsqueeze(0)
    near = (i - j) < size if size is not None else torch.ones(n, m, dtype=torch.bool)
    return (j <= i) & (near | (j < keep))


def distance_bucket(n: int, rows: int, most: int) -> int:
    """Row of a distance table with ``rows`` rows: the first half one distance each, the others in equal steps of the distance's
    logarithm up to ``most``.  Decided in integers: the largest k with ``(n / half) ** (rows - half) >= (most / half) ** k``."""
    half = rows // 2
    if n < half:
        return n
    steps = rows - half
    passed = max(k for k in range(steps + 1) if n ** steps * half ** k >= most ** k * half ** steps)
    return min(rows - 1, half + passed)


def masked_attention(q, k, v, seen, scale: float, bias=None) -> torch.Tensor:
    """Softmax attention over the keys ``seen`` [n, m]; query head h uses key head ``h // (H / G)``; ``bias`` [H, n, m] is added
    to the scaled scores."""
    rep = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    s = torch.einsum("nhd,mhd->hnm", q, k[:, rep]) * scale
    if bias is not None:
        s = s + bias
    s = s.masked_fill(~seen, float("-inf"))
    return torch.einsum("hnm,mhe->nhe", torch.softmax(s, -1), v[:, rep])


def route(z: torch.Tensor, correction: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Chosen experts [n, top] and their weights from router logits ``z`` [n, E]: softmax scores, the choice by score plus
    correction, the weights the chosen scores over their sum."""
    s = torch.softmax(z, -1)
    chosen = torch.argsort(-(s + correction), dim=-1, stable=True)[:, :top]
    picked = s.gather(1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def stream_read(xs: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """Input of a sublayer from the residual streams ``xs`` [s, n, W]."""
    return torch.einsum("s,snw->nw", w_in, xs)


def stream_write(xs: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """Streams after a sublayer with result ``y``: old streams mixed ([from, to]) and ``y`` added to each by its factor."""
    return torch.einsum("st,snw->tnw", mix, xs) + out.view(-1, 1, 1) * y


def linear_step(S: torch.Tensor, q, k, v, decay) -> tuple[torch.Tensor, torch.Tensor]:
    """One token of a linear recurrence for all heads: the state decays, takes ``k v^T`` and is read by ``q``.  ``S``
    [H, dim, vdim]; ``q``, ``k``, ``decay`` [H, dim]; ``v`` [H, vdim]."""
    S = decay.unsqueeze(-1) * S + k.unsqueeze(-1) * v.unsqueeze(1)
    return torch.einsum("hkv,hk->hv", S, q), S


def gated_parts_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """``y silu(z)``, every one of ``parts`` equal parts over its own root mean square, times ``w``."""
    y = y * silu(z)
    return rms(y.view(*y.shape[:-1], parts, -1), eps).reshape(y.shape) * w


# ------------------------------------------------------------------ layers
def delta_mixer(w, p: str, m: dict, h, st: dict, eps: float, per_channel: bool) -> torch.Tensor:
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    if not st:
        for t, c in (("q", G * d), ("k", G * d), ("v", H * e)):
            st[t] = torch.zeros(m["conv"] - 1, c, dtype=h.dtype)
        st["S"] = torch.zeros(H, d, e, dtype=h.dtype)
    mixed = {}
    for t in ("q", "k", "v"):
        mixed[t], st[t] = short_conv(h @ w[f"{p}.{t}"].T, w[f"{p}.{t}.conv"], st[t])
    rep = torch.arange(H) // (H // G)
    q = unit(mixed["q"].view(n, G, d))[:, rep] * d ** -0.5
    k = unit(mixed["k"].view(n, G, d))[:, rep]
    v = mixed["v"].view(n, H, e)
    beta = 1.0 / (1.0 + torch.exp(-(h @ w[f"{p}.b"].T)))
    rate = -torch.exp(w[f"{p}.A_log"])
    if per_channel:
        a = softplus((h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T + w[f"{p}.dt_bias"]).view(n, H, d)
        decay = torch.exp(rate.view(1, H, 1) * a)
        z = (h @ w[f"{p}.g1"].T) @ w[f"{p}.g2"].T
        gate = 1.0 / (1.0 + torch.exp(-z))
    else:
        a = softplus(h @ w[f"{p}.a"].T + w[f"{p}.dt_bias"])
        decay = torch.exp(rate * a).unsqueeze(-1).expand(n, H, d)
        gate = silu(h @ w[f"{p}.g"].T)
    o = torch.empty(n, H, e, dtype=h.dtype)
    for t in range(n):
        o[t], st["S"] = delta_step(st["S"], q[t], k[t], v[t], beta[t], decay[t])
    o = rms(o, eps) * w[f"{p}.norm"] * gate.view(n, H, e)
    return o.reshape(n, H * e) @ w[f"{p}.o"].T


def latent_mixer(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    H, d, e = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    cq = rms(h @ w[f"{p}.dq"].T, eps) * w[f"{p}.dq.norm"]
    q = (cq @ w[f"{p}.uq"].T).view(n, H, d)
    c = rms(h @ w[f"{p}.dkv"].T, eps) * w[f"{p}.dkv.norm"]
    first = st["c"].shape[0] if st else 0
    st["c"] = torch.cat([st["c"], c]) if st else c
    k = (st["c"] @ w[f"{p}.uk"].T).view(-1, H, d)
    v = (st["c"] @ w[f"{p}.uv"].T).view(-1, H, e)
    mask = m.get("mask")
    o = windowed_attention(q, k, v, first, mask["size"] if mask else None, m["scale"])
    gate = 1.0 / (1.0 + torch.exp(-(h @ w[f"{p}.g"].T)))
    o = o * gate.unsqueeze(-1)
    return o.reshape(n, H * e) @ w[f"{p}.o"].T


def attention_branch(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Grouped-query attention whose values are the keys as projected (before norm and rotation), with a sink."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    n = h.shape[0]
    q, k = (h @ w[f"{p}.q"].T).view(n, H, d), (h @ w[f"{p}.k"].T).view(n, G, d)
    first = st["k"].shape[0] if st else 0
    freq, mult = rotary_frequencies(m["rot"])
    turned = rotate_pairs(rms(k, eps) * w[f"{p}.k.norm"], first, freq, mult)
    q = rotate_pairs(rms(q, eps) * w[f"{p}.q.norm"], first, freq, mult)
    st["k"] = torch.cat([st["k"], turned]) if st else turned
    st["v"] = torch.cat([st["v"], k]) if "v" in st else k
    mask = m.get("mask")
    o = sink_attention(q, st["k"], st["v"], first, mask["size"] if mask else None, m["scale"])
    return o.reshape(n, H * d) @ w[f"{p}.o"].T


def gated_linear_branch(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    H, d, e = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    if not st:
        st["S"] = torch.zeros(H, d, e, dtype=h.dtype)
    q, k = (h @ w[f"{p}.q"].T).view(n, H, d) * d ** -0.5, (h @ w[f"{p}.k"].T).view(n, H, d)
    v = (h @ w[f"{p}.v"].T).view(n, H, e)
    z = (h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T + w[f"{p}.a2.b"]
    alpha = ((1.0 / (1.0 + torch.exp(-z))) ** (1.0 / m["tau"])).view(n, H, d)
    o = torch.empty(n, H, e, dtype=h.dtype)
    for t in range(n):
        o[t], st["S"] = linear_step(st["S"], q[t], k[t], v[t], alpha[t])
    o = (rms(o, eps) * w[f"{p}.norm"]).reshape(n, H * e) * silu(h @ w[f"{p}.g"].T)
    return o @ w[f"{p}.o"].T


def parallel_mixer(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    left = attention_branch(w, f"{p}.left", m["left"], h, st.setdefault("left", {}), eps)
    right = gated_linear_branch(w, f"{p}.right", m["right"], h, st.setdefault("right", {}), eps)
    return m["left_scale"] * left + m["right_scale"] * right


def ssd_mixer(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """State-space duality layer (Mamba-2): [z | x | B | C | dt] from one projection, x, B and C through the convolution."""
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    n, inner = h.shape[0], H * P
    z, xbc, dt = (h @ w[f"{p}.in"].T).split([inner, inner + 2 * G * N, H], -1)
    if not st:
        st["past"] = torch.zeros(m["conv"] - 1, xbc.shape[1], dtype=h.dtype)
        st["S"] = torch.zeros(H, N, P, dtype=h.dtype)
    xbc, st["past"] = short_conv(xbc, w[f"{p}.conv"], st["past"], w[f"{p}.conv.b"])
    x, B, C = xbc.split([inner, G * N, G * N], -1)
    rep = torch.arange(H) // (H // G)
    x, B, C = x.view(n, H, P), B.view(n, G, N)[:, rep], C.view(n, G, N)[:, rep]
    dt = softplus(dt + w[f"{p}.dt_bias"])
    decay = torch.exp(-torch.exp(w[f"{p}.A_log"]) * dt).unsqueeze(-1).expand(n, H, N)
    y = torch.empty(n, H, P, dtype=h.dtype)
    for t in range(n):
        y[t], st["S"] = linear_step(st["S"], C[t], B[t], dt[t].unsqueeze(-1) * x[t], decay[t])
    y = (y + w[f"{p}.D"].unsqueeze(-1) * x).reshape(n, inner)
    return gated_parts_norm(y, z, w[f"{p}.norm"], m["norm_groups"], eps) @ w[f"{p}.o"].T


def gated_feed_forward(w, p: str, h) -> torch.Tensor:
    return (gelu_tanh(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def token_side(w, p: str, x, e, eps: float) -> torch.Tensor:
    """What a layer takes from its part ``e`` of the token's side embedding, gated by the residual."""
    y = (gelu_tanh(x @ w[f"{p}.gate"].T) * e) @ w[f"{p}.proj"].T
    return rms(y, eps) * w[f"{p}.norm"]


SEQUENTIAL_MIXERS = {"parallel": parallel_mixer, "mamba2": ssd_mixer}


def conv_attention(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Attention behind short convolutions of q, k and v: rotary halves, then unit root mean squares; a window and kept first
    tokens."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    if not st:
        for t, c in (("q", H * d), ("k", G * d), ("v", G * e)):
            st[f"past_{t}"] = torch.zeros(m["conv"] - 1, c, dtype=h.dtype)
        st["k"], st["v"] = torch.zeros(0, G, d, dtype=h.dtype), torch.zeros(0, G, e, dtype=h.dtype)
    first, new = st["k"].shape[0], {}
    for t in "qkv":
        new[t], st[f"past_{t}"] = plain_short_conv(h @ w[f"{p}.{t}"].T, w[f"{p}.{t}.conv"], st[f"past_{t}"])
    rot = m["rot"]
    q, k = (rms(rotate_halves(new[t].view(n, -1, d), first, rot["dims"], rot["base"]), eps) for t in "qk")
    st["k"], st["v"] = torch.cat([st["k"], k]), torch.cat([st["v"], new["v"].view(n, G, e)])
    mask = m.get("mask") or {}
    seen = kept_window(first, n, first + n, mask.get("size"), mask.get("keep_first", 0))
    return masked_attention(q, st["k"], st["v"], seen, m["scale"]).reshape(n, H * e) @ w[f"{p}.o"].T


def biased_attention(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Attention without rotation: q and k normed over their whole projection, queries warmer with their position, a learned
    bias per bucket of distance and head."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    if not st:
        st["k"], st["v"] = torch.zeros(0, G, d, dtype=h.dtype), torch.zeros(0, G, e, dtype=h.dtype)
    first = st["k"].shape[0]
    q, k = (rms(h @ w[f"{p}.{t}"].T, eps) * w[f"{p}.{t}.norm"] for t in "qk")
    if m.get("q_temp"):
        warm = [1.0 + m["q_temp"]["coef"] * math.log((pos + 1) // m["q_temp"]["every"] + 1) for pos in range(first, first + n)]
        q = q * torch.tensor(warm, dtype=h.dtype).unsqueeze(1)
    st["k"] = torch.cat([st["k"], k.view(n, G, d)])
    st["v"] = torch.cat([st["v"], (h @ w[f"{p}.v"].T).view(n, G, e)])
    rel, total = w[f"{p}.rel"], first + n
    by_distance = rel[torch.tensor([distance_bucket(i, rel.shape[0], m["bias_max"]) for i in range(total)])]
    seen = kept_window(first, n, total, None, 0)
    gap = (torch.arange(first, total).unsqueeze(1) - torch.arange(total)).clamp(min=0)
    return masked_attention(q.view(n, H, d), st["k"], st["v"], seen, m["scale"], by_distance[gap].permute(2, 0, 1)).reshape(n, H * e) \
        @ w[f"{p}.o"].T


STREAM_MIXERS = {"attention": conv_attention, "attention_2": biased_attention}


def routed_feed_forward(w, p: str, mlp: dict, h) -> torch.Tensor:
    """Squared-relu experts with identity experts behind them, and a gated shared expert."""
    r = mlp["router"]
    chosen, weight = route(h @ w[f"{p}.router"].T, w[f"{p}.correction"], r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t].tolist(), weight[t]):
            y = h[t] if e >= r["experts"] else squared_relu(h[t] @ w[f"{p}.e{e}.up"].T) @ w[f"{p}.e{e}.down"].T
            out[t] += g * y
    if mlp.get("shared"):
        gate = 1.0 / (1.0 + torch.exp(-(h @ w[f"{p}.shared.sg"].T)))
        out = out + gate * (squared_relu(h @ w[f"{p}.shared.up"].T) @ w[f"{p}.shared.down"].T)
    return out


def silu_feed_forward(w, p: str, h) -> torch.Tensor:
    return (silu(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def same_chunk(first: int, n: int, m: int, size: int | None) -> torch.Tensor:
    """[n, m] which of m keys the queries at positions ``first ..`` see: the earlier ones of their own chunk of ``size`` positions."""
    i, j = torch.arange(first, first + n).unsqueeze(1), torch.arange(m).unsqueeze(0)
    seen = j <= i
    return seen if size is None else seen & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def rotated_latent_attention(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Latent attention whose scores have two parts: per head from the latent, and rotated from a key all heads share."""
    H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    n = h.shape[0]
    q = (h @ w[f"{p}.q"].T).view(n, H, d + r)
    down = h @ w[f"{p}.dkv"].T
    first = st["c"].shape[0] if st else 0
    freq, mult = rotary_frequencies(m["rot"])
    c = rms(down[:, :R], eps) * w[f"{p}.dkv.norm"]
    shared = rotate_pairs(down[:, R:].unsqueeze(1), first, freq, mult)[:, 0]
    turned = rotate_pairs(q[..., d:], first, freq, mult)
    st["c"] = torch.cat([st["c"], c]) if st else c
    st["r"] = torch.cat([st["r"], shared]) if "r" in st else shared
    k = (st["c"] @ w[f"{p}.uk"].T).view(-1, H, d)
    v = (st["c"] @ w[f"{p}.uv"].T).view(-1, H, e)
    k = torch.cat([k, st["r"].unsqueeze(1).expand(-1, H, r)], -1)
    o = masked_attention(torch.cat([q[..., :d], turned], -1), k, v, same_chunk(first, n, first + n, None), m["scale"])
    return o.reshape(n, H * e) @ w[f"{p}.o"].T


def differential_attention(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Two attention maps per head over the same values, the second subtracted with a learned factor; heads normed and gated."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    first = st["k"].shape[0] if st else 0
    rot = m["rot"]
    q, k = (rms((h @ w[f"{p}.{t}"].T).view(n, -1, d), eps) * w[f"{p}.{t}.norm"] for t in "qk")
    q, k = (rotate_halves(t, first, rot["dims"], rot["base"]).view(n, -1, 2, d) for t in (q, k))
    v = (h @ w[f"{p}.v"].T).view(n, G, e)
    st["k"] = torch.cat([st["k"], k]) if st else k
    st["v"] = torch.cat([st["v"], v]) if "v" in st else v
    mask = m.get("mask")
    seen = same_chunk(first, n, first + n, mask["size"] if mask else None)
    a1, a2 = (masked_attention(q[:, :, i], st["k"][:, :, i], st["v"], seen, m["scale"]) for i in range(2))
    less = torch.exp((w[f"{p}.lq1"] * w[f"{p}.lk1"]).sum()) - torch.exp((w[f"{p}.lq2"] * w[f"{p}.lk2"]).sum()) + m["diff"]
    o = rms(a1 - less * a2, eps) * (1.0 - m["diff"])
    return (o.reshape(n, H * e) * sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def mingru_mixer(w, p: str, m: dict, h, st: dict, eps: float) -> torch.Tensor:
    """Element-wise recurrence whose gate and candidate read the current token only."""
    z = sigmoid(h @ w[f"{p}.z"].T + w[f"{p}.z.b"])
    u = h @ w[f"{p}.x"].T + w[f"{p}.x.b"]
    candidate = torch.where(u >= 0, u + 0.5, sigmoid(u))
    S = st["S"] if st else torch.zeros(m["width"], dtype=h.dtype)
    out = torch.empty_like(u)
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * candidate[t]
        out[t] = S
    st["S"] = S
    return (out * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


GATED_MIXERS = {"latent_attention": rotated_latent_attention, "attention": differential_attention, "mingru": mingru_mixer}


def clamped_feed_forward(w, p: str, h, limit: float) -> torch.Tensor:
    g, u = torch.clamp(h @ w[f"{p}.gate"].T, max=limit), torch.clamp(h @ w[f"{p}.up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[f"{p}.down"].T


def layer_schedule(cfg: dict) -> list[tuple[int, bool]]:
    """The layer runs in order: (layer index, whether the pass's entry projection comes right before it)."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, r = loop["start"], loop["stop"], loop["times"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(r) for i in range(a, b)]
            + [(i, False) for i in range(b, n)])


class Oracle:
    def __init__(self, cfg: dict, weights: dict[str, torch.Tensor], dtype=torch.float32) -> None:
        self.cfg, self.dtype = cfg, dtype
        self.w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
        self.schedule = layer_schedule(cfg)

    def new_state(self) -> "OracleState":
        return OracleState([{} for _ in self.schedule])

    @torch.no_grad()
    def forward(self, tokens, state=None, positions3=None, embeds=None, last_only: bool = False, trace: list | None = None):
        """Append ``tokens`` to ``state``; returns (logits, state).  ``trace`` receives the residual after every run."""
        w, cfg = self.w, self.cfg
        eps = float(cfg["norm"]["eps"])
        state = state if state is not None else self.new_state()
        ids = torch.as_tensor(list(tokens), dtype=torch.long)
        if cfg["architecture"] == "Loduzen":
            return self._sequential(ids, state, eps, last_only, trace)
        if cfg["architecture"] == "Vimelorn":
            return self._streams(ids, state, eps, last_only, trace)
        if cfg["architecture"] == "Fovunex":
            return self._gated(ids, state, eps, last_only, trace)
        x0 = rms_around_zero(w["embed"][ids], w["embed.norm"], eps)
        x = x0
        for (i, enters), st in zip(self.schedule, state.runs):
            if enters:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T
            layer, p = cfg["layers"][i], f"l{i}"
            h = rms_around_zero(x, w[f"{p}.norm1"], eps)
            kind, m = layer["type"], layer["mixer"]
            if kind == "latent_attention":
                y = latent_mixer(w, f"{p}.mix", m, h, st, eps)
            elif kind in ("delta", "channel_delta"):
                y = delta_mixer(w, f"{p}.mix", m, h, st, eps, kind == "channel_delta")
            else:
                raise ValueError(f"unknown mixer {kind!r}")
            if layer.get("mlp"):
                y = y + squared_relu(h @ w[f"{p}.mlp.up"].T) @ w[f"{p}.mlp.down"].T
            x = x + y
            if trace is not None:
                trace.append(x.clone())
        state.length += len(ids)
        if last_only:
            x = x[-1:]
        return rms_around_zero(x, w["final.norm"], eps) @ w["head"].T, state


    def _sequential(self, ids, state, eps: float, last_only: bool, trace):
        """Pre-norm layers, mixer then feed-forward then the token's side input; plain norm weights, tied output head."""
        w, cfg = self.w, self.cfg
        side = cfg.get("token_side")
        x = w["embed"][ids]
        for i, (layer, st) in enumerate(zip(cfg["layers"], state.runs)):
            p = f"l{i}"
            h = rms(x, eps) * w[f"{p}.norm1"]
            x = x + SEQUENTIAL_MIXERS[layer["type"]](w, f"{p}.mix", layer["mixer"], h, st, eps)
            if layer.get("mlp"):
                x = x + gated_feed_forward(w, f"{p}.mlp", rms(x, eps) * w[f"{p}.norm2"])
            if side:
                e = w["side.embed"][ids, i * side["dim"]:(i + 1) * side["dim"]]
                x = x + token_side(w, f"{p}.side", x, e, eps)
            if trace is not None:
                trace.append(x.clone())
        state.length += len(ids)
        if last_only:
            x = x[-1:]
        return (rms(x, eps) * w["final.norm"]) @ w["embed"].T, state


    def _streams(self, ids, state, eps: float, last_only: bool, trace):
        """Pre-norm sublayers that read and write several residual streams; a scaled embedding, untied head."""
        w, cfg = self.w, self.cfg
        xs = (w["embed"][ids] * cfg["embedding"]["scale"]).repeat(cfg["streams"], 1, 1)
        for i, (layer, st) in enumerate(zip(cfg["layers"], state.runs)):
            p, mlp = f"l{i}", layer.get("mlp")
            subs = [(1, lambda h: STREAM_MIXERS[layer["type"]](w, f"{p}.mix", layer["mixer"], h, st, eps))]
            if mlp:
                subs.append((2, lambda h: silu_feed_forward(w, f"{p}.mlp", h) if mlp["kind"] == "dense"
                             else routed_feed_forward(w, f"{p}.mlp", mlp, h)))
            for q, sub in subs:
                u = stream_read(xs, w[f"{p}.hc{q}.in"])
                y = sub(rms(u, eps) * w[f"{p}.norm{q}"])
                xs = stream_write(xs, w[f"{p}.hc{q}.mix"], w[f"{p}.hc{q}.out"], y)
            if trace is not None:
                trace.append(xs.sum(0))
        state.length += len(ids)
        x = xs.sum(0)
        if last_only:
            x = x[-1:]
        return (rms(x, eps) * w["final.norm"]) @ w["head"].T, state


    def _gated(self, ids, state, eps: float, last_only: bool, trace):
        """Pre-norm layers whose results pass a gate per channel that reads the same normed input; norms with one number; the
        embedding output is added again before every later pass of the loop."""
        w, cfg = self.w, self.cfg
        x0 = w["embed"][ids] * cfg["embedding"]["scale"]
        x, passes = x0, 0
        for (i, enters), st in zip(self.schedule, state.runs):
            if enters:
                passes += 1
                x = x + x0 if passes > 1 else x
            layer, p = cfg["layers"][i], f"l{i}"
            h = rms(x, eps) * w[f"{p}.norm1"]
            y = GATED_MIXERS[layer["type"]](w, f"{p}.mix", layer["mixer"], h, st, eps)
            x = x + y * sigmoid(h @ w[f"{p}.rg1"].T + w[f"{p}.rg1.b"])
            if layer.get("mlp"):
                h = rms(x, eps) * w[f"{p}.norm2"]
                y = clamped_feed_forward(w, f"{p}.mlp", h, layer["mlp"]["limit"])
                x = x + y * sigmoid(h @ w[f"{p}.rg2"].T + w[f"{p}.rg2.b"])
            if trace is not None:
                trace.append(x.clone())
        state.length += len(ids)
        if last_only:
            x = x[-1:]
        return (rms(x, eps) * w["final.norm"]) @ w["head"].T, state


class OracleState:
    def __init__(self, runs: list[dict]) -> None:
        self.runs, self.length = runs, 0

    def copy(self) -> "OracleState":
        return copy.deepcopy(self)


class LayeredEagerExecutor(StatefulEagerExecutor):
    """``execute(segments)`` of the eager execution mode: one explicit state per request slot (no pages, no prefix sharing)."""

    accepts_features = False

    def __init__(self, cfg, weights: dict[str, torch.Tensor], raw_config: dict | None = None) -> None:
        self.cfg = cfg
        super().__init__(Oracle(raw_config if raw_config is not None else cfg.to_config(), weights))

    def _new_state(self) -> OracleState:
        return self.model.new_state()

    def _copy(self, state: OracleState) -> OracleState:
        return state.copy()
