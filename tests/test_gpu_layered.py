"""Layered decoders on the GPU: every mechanism alone against the oracle's equations, then whole models through the executor,
the scheduler and the engine."""
import sys
from pathlib import Path

import numpy as np
import pytest
import torch
from torch.overrides import TorchFunctionMode

sys.path.insert(0, str(Path(__file__).parent))
from layered_cases import (ALL, channel, clamped, config, delta, differential, far, gated, latent, mamba2, mingru, near,  # noqa: E402
                           parallel, prompt, rotated, routed, sequential, streams, tensors, write)

from cubic_serve_b200.models import layered_reference as R  # noqa: E402

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]


def segs(spans):
    """``[(count, slot, pos0)]`` -> device segments, rows packed in order."""
    from cubic_serve_b200.ops import kernels as K
    i32 = dict(dtype=torch.int32, device=DEV)
    row0 = np.cumsum([0] + [c for c, _, _ in spans])[:-1].tolist()
    col = [row0] + [[s[j] for s in spans] for j in range(3)]
    return K.GdnSegments(*(torch.tensor(c, **i32) for c in col), len(spans))


def close(got, want, dtype, exact=2e-5, rough=2e-2):
    """Largest error relative to the largest wanted magnitude."""
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-9)
    assert err <= (exact if dtype == torch.float32 else rough), float(err)


# ------------------------------------------------------------------ products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m, n, k, stream_k", [(1, 40, 64, None), (17, 200, 128, None), (5, 131, 640, None), (300, 260, 192, None),
                                               (64, 512, 2048, None), (33, 300, 256, True), (520, 384, 128, True), (520, 512, 192, True)])
def test_wide_gemm(dtype, m, n, k, stream_k):
    from cubic_serve_b200.ops import kernels as K, wq_pack
    g = torch.Generator().manual_seed(m)
    x = (torch.randn(m, k, generator=g)).to(dtype)
    w = wq_pack.pack_bf16(torch.randn(n, k, generator=g) / k ** 0.5)
    want = x.double() @ w.codes.double().t()
    xd, wd = x.to(DEV), w.to(DEV)
    y = torch.full((m, n), 7.0, dtype=dtype, device=DEV)
    K.wide_gemm(xd, wd, y, stream_k=stream_k)
    close(y, want, dtype, rough=6e-3)
    # fp32 output accumulated into a residual
    res = torch.randn(m, n, generator=g)
    r = res.to(DEV)
    K.wide_gemm(xd, wd, r, residual=r, stream_k=stream_k)
    close(r, want + res, torch.float32, exact=1e-5)
    # two outputs, the second behind the squared relu, at an offset of a wider buffer
    split = (n // 2) // 8 * 8
    wide = torch.full((m, 16 + n - split + 8), 5.0, dtype=dtype, device=DEV)
    a = torch.full((m, split), 7.0, dtype=dtype, device=DEV)
    K.wide_gemm(xd, wd, a, relu2=wide[:, 16:16 + n - split], split=split, stream_k=stream_k)
    close(a, want[:, :split], dtype, rough=6e-3)
    close(wide[:, 16:16 + n - split], want[:, split:].clamp_min(0) ** 2, dtype, rough=1.5e-2)
    assert (wide[:, :16] == 5).all() and (wide[:, 16 + n - split:] == 5).all()
    K.workspace(torch.device(DEV)).check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("splits", [2, 5])
def test_wide_gemm_split_over_k(dtype, splits):
    from cubic_serve_b200.ops import kernels as K, wq_pack
    if dtype == torch.float32:
        pytest.skip("the fp32 product has no splits")
    x, w = torch.randn(40, 1024).to(dtype), wq_pack.pack_bf16(torch.randn(136, 1024) / 32)
    want = x.double() @ w.codes.double().t()
    y = torch.zeros(40, 136, device=DEV)
    K.wide_gemm(x.to(DEV), w.to(DEV), y, residual=y, splits=splits)
    close(y, want, torch.float32, exact=1e-5)
    out, act = torch.zeros(40, 64, dtype=dtype, device=DEV), torch.zeros(40, 72, dtype=dtype, device=DEV)
    K.wide_gemm(x.to(DEV), w.to(DEV), out, relu2=act, split=64, splits=splits)
    close(out, want[:, :64], dtype, rough=6e-3)
    close(act, want[:, 64:].clamp_min(0) ** 2, dtype, rough=1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, n, k, m", [(5, 64, 16, 3), (3, 128, 24, 40), (6, 24, 64, 9), (4, 32, 128, 300), (7, 20, 64, 2), (1, 16, 64, 5)])
def test_block_diagonal_product(dtype, H, n, k, m):
    from cubic_serve_b200.models.layered import BlockDiagonal
    from cubic_serve_b200.ops import kernels as K
    w = (torch.randn(H, n, k) / k ** 0.5).to(torch.bfloat16)
    b = BlockDiagonal.pack(w)
    x = torch.randn(m, H, k).to(dtype)
    kg = b.w.k
    cols = torch.zeros(m, -(-H // b.heads) * kg, dtype=dtype)
    for h in range(H):
        c = (h // b.heads) * kg + (h % b.heads) * k
        cols[:, c:c + k] = x[:, h]
    y = torch.zeros(m, H * n, dtype=dtype, device=DEV)
    K.wide_gemm(cols.to(DEV), b.w.to(DEV), y, diag_rows=b.rows)
    close(y, torch.einsum("thk,hnk->thn", x.double(), w.double()).reshape(m, H * n), dtype, rough=6e-3)


# ------------------------------------------------------------------ rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 68, 67, 2048, 8704])
def test_row_kernels(dtype, W):
    from cubic_serve_b200.ops import kernels as K
    x, w = torch.randn(7, W) * 3, torch.randn(W) * 0.2
    ld = -(-W // 64) * 64
    out = torch.full((7, ld), 9.0, dtype=dtype, device=DEV)
    K.row_norm(x.to(DEV), (1 + w).to(DEV), out, 1e-3)
    close(out[:, :W], R.rms_around_zero(x.double(), w.double(), 1e-3), dtype, exact=1e-6, rough=6e-3)
    assert (out[:, W:] == 9).all()
    rows = torch.tensor([4, 0, 6], device=DEV)
    K.row_norm(x.to(DEV), (1 + w).to(DEV), out, 1e-3, rows=rows)
    close(out[:3, :W], R.rms_around_zero(x.double()[[4, 0, 6]], w.double(), 1e-3), dtype, exact=1e-6, rough=6e-3)
    table, ids = torch.randn(11, W).to(torch.bfloat16), torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    e, e0 = torch.zeros(4, W, device=DEV), torch.zeros(4, W, device=DEV)
    K.embed_norm(ids.to(DEV), table.to(DEV), (1 + w).to(DEV), e, 1e-3, e0)
    close(e, R.rms_around_zero(table.double()[ids.long()], w.double(), 1e-3), torch.float32, exact=1e-6)
    assert torch.equal(e, e0)
    both = torch.zeros(4, -(-2 * W // 64) * 64, dtype=dtype, device=DEV)
    K.concat_rows(e, e0 * 2, both)
    close(both[:, :2 * W], torch.cat([e, e0 * 2], 1).double().cpu(), dtype, exact=0, rough=4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sampler_reads_both_logit_types(dtype):
    from cubic_serve_b200.ops import kernels as K
    lg = torch.randn(5, 1003).to(dtype)
    lg[2, 7] = lg[2, 900] = 50.0
    ids = torch.zeros(5, dtype=torch.int32, device=DEV)
    K.sample(lg.to(DEV), ids)
    want = lg.float().argmax(-1)
    want[2] = 7
    assert ids.cpu().tolist() == want.tolist()


# ------------------------------------------------------------------ delta rule
def delta_case(H, G, d, e, taps, per_channel, T, seed=0):
    g = torch.Generator().manual_seed(seed)
    C = 2 * G * d + H * e
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)                    # noqa: E731
    return {"x": bf(T, C), "conv": torch.randn(C, taps, generator=g) / taps ** 0.5, "b": bf(T, H),
            "a": bf(T, H * d if per_channel else H), "z": bf(T, H * e), "a_log": torch.randn(H, generator=g) * 0.5 - 1.5,
            "dt": torch.randn(H * d if per_channel else H, generator=g) * 0.5, "norm": 1 + 0.2 * torch.randn(e, generator=g)}


def delta_oracle(c, H, G, d, e, taps, per_channel, eps, past=None, S=None):
    """The mechanism from the projections on, in fp64: (outputs, convolution history, state)."""
    f = {k: v.double() for k, v in c.items()}
    T = f["x"].shape[0]
    past = torch.zeros(taps - 1, f["x"].shape[1], dtype=torch.float64) if past is None else past
    S = torch.zeros(H, d, e, dtype=torch.float64) if S is None else S
    y, past = R.short_conv(f["x"], f["conv"], past)
    rep = torch.arange(H) // (H // G)
    q = R.unit(y[:, :G * d].view(T, G, d))[:, rep] * d ** -0.5
    k = R.unit(y[:, G * d:2 * G * d].view(T, G, d))[:, rep]
    v = y[:, 2 * G * d:].view(T, H, e)
    rate, sp = -torch.exp(f["a_log"]), R.softplus(f["a"] + f["dt"])
    decay = torch.exp(rate.view(1, H, 1) * sp.view(T, H, d)) if per_channel else torch.exp(rate * sp).unsqueeze(-1).expand(T, H, d)
    o = torch.empty(T, H, e, dtype=torch.float64)
    for t in range(T):
        o[t], S = R.delta_step(S, q[t], k[t], v[t], 1 / (1 + torch.exp(-f["b"][t])), decay[t])
    gate = 1 / (1 + torch.exp(-f["z"])) if per_channel else R.silu(f["z"])
    return R.rms(o, eps) * f["norm"] * gate.view(T, H, e), past, S


def run_delta(c, shape, dtype, spans, conv_state, state, eps=1e-5, decode=None):
    from cubic_serve_b200.ops import kernels as K
    H, G, d, e, taps, per_channel = shape
    T, C = c["x"].shape
    pad = -(-C // 8) * 8
    x = torch.zeros(T, pad, dtype=dtype)
    x[:, :C] = c["x"]
    w = torch.zeros(taps, pad)
    w[:, :C] = c["conv"].t()
    dev = {k: v.to(DEV, dtype).contiguous() for k, v in c.items() if k in "baz"}
    f32 = {k: c[k].float().to(DEV).contiguous() for k in ("a_log", "dt", "norm")}
    sc = K.RecurrenceScratch(T, [(H, G, d, e, per_channel)], dtype, DEV)
    seg = spans if not isinstance(spans, list) else segs(spans)
    out = torch.full((T, H * e + 8), 3.0, dtype=dtype, device=DEV)[:, :H * e]
    K.delta_prepare(x.to(DEV), dev["b"], dev["a"], w.to(DEV), conv_state, f32["a_log"], f32["dt"], seg, sc, H, G, d, e)
    K.delta_walk(dev["z"], f32["norm"], state, seg, out, sc, G, d, eps, per_channel, per_channel,
                 T == seg.num if decode is None else decode)
    return out.clone().reshape(T, H, e)


def delta_states(shape, dtype, slots):
    H, G, d, e, taps, _ = shape
    pad = -(-(2 * G * d + H * e) // 8) * 8
    return (torch.full((slots, max(1, taps - 1), pad), 5.0, dtype=dtype, device=DEV),          # stale contents: a fresh request
            torch.full((slots, H, e, -(-d // 4) * 4), 5.0, device=DEV))                        # must not read them


SHAPES = [(4, 2, 64, 64, 4), (2, 2, 128, 128, 4), (3, 1, 20, 13, 3), (2, 1, 7, 9, 5), (1, 1, 16, 16, 1), (2, 2, 160, 144, 2),
          (6, 3, 32, 200, 3), (2, 1, 256, 24, 4), (2, 2, 96, 64, 7)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("shape", SHAPES)
def test_delta_layer_in_portions(dtype, per_channel, shape):
    """Portions of several sizes (down to two tokens, one at the end) on a slot with stale contents, against token by token."""
    shape = (*shape, per_channel)
    T = 75
    c = delta_case(*shape, T)
    want, past, S = delta_oracle(c, *shape, 1e-5)
    conv_state, state = delta_states(shape, dtype, 3)
    got, i = [], 0
    for n in (2, 37, 16, 17, 2, 1):
        part = {k: (v[i:i + n] if k in ("x", "b", "a", "z") else v) for k, v in c.items()}
        got.append(run_delta(part, shape, dtype, [(n, 1, i)], conv_state, state))
        i += n
    close(torch.cat(got), want, dtype, exact=5e-5)
    close(state[1, :, :, :shape[2]].transpose(1, 2), S, torch.float32, exact=2e-5 if dtype == torch.float32 else 2e-2)
    if shape[4] > 1:
        close(conv_state[1, :, :c["x"].shape[1]], past, torch.float32, exact=0)
    assert (state[0] == 5).all() and (state[2] == 5).all() and (conv_state[0] == 5).all()      # other slots are untouched


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64, 4), (3, 1, 20, 13, 3), (2, 2, 128, 128, 2)])
def test_delta_layer_batches(dtype, per_channel, shape):
    """Unequal requests in one step equal each alone; decode steps with a padding segment; a slot used again."""
    shape = (*shape, per_channel)
    lens, slots = (33, 1, 2, 50, 16), (4, 0, 3, 1, 2)
    cs = [delta_case(*shape, n + 1, seed=n) for n in lens]
    oracle = [delta_oracle({k: (v[:n] if k in ("x", "b", "a", "z") else v) for k, v in c.items()} | {"conv": cs[0]["conv"], "a_log": cs[0]["a_log"],
              "dt": cs[0]["dt"], "norm": cs[0]["norm"]}, *shape, 1e-5) for c, n in zip(cs, lens)]
    conv_state, state = delta_states(shape, dtype, 5)
    shared = {k: cs[0][k] for k in ("conv", "a_log", "dt", "norm")}
    batch = {k: torch.cat([c[k][:n] for c, n in zip(cs, lens)]) for k in ("x", "b", "a", "z")} | shared
    out = run_delta(batch, shape, dtype, [(n, s, 0) for n, s in zip(lens, slots)], conv_state, state)
    for o, (want, _, _) in zip(out.split(lens), oracle):
        close(o, want, dtype, exact=5e-5)
    # one decoded token each, with a padding segment between them
    order = [0, 1, None, 2, 3, 4]
    rows = {k: torch.cat([cs[i][k][lens[i]:] if i is not None else torch.zeros_like(cs[0][k][:1]) for i in order])
            for k in ("x", "b", "a", "z")} | shared
    spans = [(1, slots[i], lens[i]) if i is not None else (0, 0, 0) for i in order]
    bucket = segs(spans)
    bucket.row0 = torch.arange(len(order), dtype=torch.int32, device=DEV)        # row j belongs to segment j
    out = run_delta(rows, shape, dtype, bucket, conv_state, state, decode=True)
    for j, i in enumerate(order):
        if i is None:
            continue
        part = {k: (cs[i][k][lens[i]:] if k in ("x", "b", "a", "z") else shared[k]) for k in cs[i]}
        want, past, S = delta_oracle(part, *shape, 1e-5, oracle[i][1], oracle[i][2])
        close(out[j:j + 1], want, dtype, exact=5e-5)
        close(state[slots[i], :, :, :shape[2]].transpose(1, 2), S, torch.float32, exact=2e-5 if dtype == torch.float32 else 2e-2)


# ------------------------------------------------------------------ latent attention
def latent_widths(R_):
    return next(p for p in (64, 128, 256, 512, 1024) if R_ <= p)


class LatentCase:
    """Latents of several requests on shuffled pages of one cache, and queries in latent space."""

    def __init__(self, lens, H, rank, dtype, seed=0, spare=3):
        g = torch.Generator().manual_seed(seed)
        self.H, self.rank, self.rp, self.dtype, self.lens = H, rank, latent_widths(rank), dtype, lens
        self.c = [torch.randn(n, rank, generator=g).to(dtype) for n in lens]
        self.q = [torch.randn(n, H, rank, generator=g).to(dtype) for n in lens]
        self.gate = [torch.randn(n, H, generator=g).to(dtype) for n in lens]
        per = [-(-n // 16) for n in lens]
        ids = (torch.randperm(sum(per) + spare, generator=g) + 1).tolist()
        self.table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        # pages nobody owns and the unwritten rest of last pages hold garbage that must not be used
        self.cache = torch.full((sum(per) + spare + 1, 16, self.rp), 1e4, dtype=dtype)
        for r, n in enumerate(per):
            pages = [ids.pop() for _ in range(n)]
            self.table[r, :n] = torch.tensor(pages)
            flat = torch.full((n * 16, self.rp), 1e4, dtype=dtype)
            flat[:lens[r], :rank] = self.c[r]
            flat[:lens[r], rank:] = 0
            self.cache[pages] = flat.view(n, 16, self.rp)

    def run(self, spans, window, scale, splits=None, decode=None):
        """``spans``: (request, first, count) in batch order; returns the outputs of every span ``[count, H, rank]``."""
        from cubic_serve_b200.ops import kernels as K
        T = sum(n for _, _, n in spans)
        q = torch.zeros(T, self.H, self.rp, dtype=self.dtype)
        gate = torch.zeros(T, self.H + 3, dtype=self.dtype)
        i = 0
        for r, first, n in spans:
            q[i:i + n, :, :self.rank] = self.q[r][first:first + n]
            gate[i:i + n, 2:2 + self.H] = self.gate[r][first:first + n]
            i += n
        out = torch.full((T, self.H * self.rp), 3.0, dtype=self.dtype, device=DEV)
        seg = segs([(n, r, first) for r, first, n in spans])
        K.latent_attention(q.view(T, -1).to(DEV), gate.to(DEV)[:, 2:2 + self.H], self.cache.to(DEV), self.table.to(DEV), seg, out,
                           self.H, window, scale, decode=T == len(spans) if decode is None else decode, splits=splits)
        out = out.view(T, self.H, self.rp)
        assert (out[:, :, self.rank:] == 0).all()
        return out[:, :, :self.rank].split([n for _, _, n in spans])

    def want(self, r, first, n, window, scale):
        c = self.c[r].double()
        k = c[:first + n].unsqueeze(1).expand(-1, self.H, -1)
        o = R.windowed_attention(self.q[r][first:first + n].double(), k, k, first, window or None, scale)
        return o / (1 + torch.exp(-self.gate[r][first:first + n].double())).unsqueeze(-1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, rank, window", [(6, 64, 37), (5, 48, 0), (32, 512, 130), (70, 128, 16), (16, 200, 100), (1, 100, 1), (3, 600, 50),
                                             (40, 256, 17)])
def test_latent_attention_prefill_portions_and_decode(dtype, H, rank, window):
    lens = (150, 3, 61, 16)
    case = LatentCase(lens, H, rank, dtype, seed=H)
    scale = 1.5 / rank ** 0.5
    whole = case.run([(r, 0, n) for r, n in enumerate(lens)], window, scale)
    for r, n in enumerate(lens):
        close(whole[r], case.want(r, 0, n, window, scale), dtype, rough=1e-2)
    # portions beside single tokens, in another order
    spans = [(2, 40, 21), (0, 149, 1), (1, 1, 2), (3, 15, 1)]
    for (r, first, n), o in zip(spans, case.run(spans, window, scale)):
        close(o, case.want(r, first, n, window, scale), dtype, rough=1e-2)
    # decode, with and without key splits (a split may see no key at all)
    spans = [(r, n - 1, 1) for r, n in enumerate(lens)]
    for splits in (None, 1, 2, 7):
        for (r, first, n), o in zip(spans, case.run(spans, window, scale, splits=splits)):
            close(o, case.want(r, first, n, window, scale), dtype, rough=1e-2)
    for splits in (3, 9):
        for r, o in enumerate(case.run([(r, 0, n) for r, n in enumerate(lens)], window, scale, splits=splits)):
            close(o, case.want(r, 0, lens[r], window, scale), dtype, rough=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 31, 33, 63, 64, 65, 129])
def test_window_edge_shows_one_key(dtype, window):
    """One key carries a score that outweighs all others and a value nothing else has: it is seen by exactly the queries whose
    window holds it, in a prompt and decoded, wherever the edge falls on a page or a key tile."""
    n, H, rank = 200, 4, 64
    for j in (0, 15, 16, 47, 64):
        case = LatentCase((n,), H, rank, dtype, seed=window)
        case.c[0] *= 0.1
        case.q[0] *= 0.1
        case.q[0][:, :, 0] = 6.0
        case.c[0][:, 0] = 0.0
        case.c[0][:, 1] = 0.0
        case.c[0][j, 0], case.c[0][j, 1] = 6.0, 40.0
        case.gate[0].zero_()
        per = -(-n // 16)
        flat = torch.zeros(per * 16, case.rp, dtype=dtype)
        flat[:n, :rank] = case.c[0]
        case.cache[case.table[0].long()] = flat.view(per, 16, case.rp)
        out = case.run([(0, 0, n)], window, 1.0)[0][:, :, 1].float().cpu()
        seen = torch.tensor([0 <= i - j < window for i in range(n)])
        assert ((out > 10).all(1) == seen).all() and ((out.abs() < 1).all(1) == ~seen).all(), (window, j)
        for i in (j + window - 1, j + window):                # just inside and just outside, decoded
            if j <= i < n:
                for splits in (None, 4):
                    one = case.run([(0, i, 1)], window, 1.0, splits=splits)[0][0, :, 1].float().cpu()
                    assert ((one > 10).all() if seen[i] else (one.abs() < 1).all()), (window, j, i)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_prepare_norms_and_pages(dtype):
    from cubic_serve_b200.ops import kernels as K
    T, qr, rank, off, rp = 5, 40, 72, 48, 128
    proj = torch.randn(T, 128).to(dtype)
    qn, cn = 1 + 0.1 * torch.randn(qr), 1 + 0.1 * torch.randn(rank)
    cq = torch.zeros(T, 64, dtype=dtype, device=DEV)
    cache = torch.zeros(4, 16, rp, dtype=dtype, device=DEV)
    slots = torch.tensor([17, 63, -1, 0, 32], dtype=torch.int32)
    K.latent_prepare(proj.to(DEV), off, rank, cn.to(DEV), cache, slots.to(DEV), 1e-4, low=(0, qr, qn.to(DEV), cq))
    p = proj.double()
    close(cq[:, :qr], R.rms(p[:, :qr], 1e-4) * qn.double(), dtype, exact=1e-6, rough=6e-3)
    assert (cq[:, qr:] == 0).all()
    want = torch.zeros(64, rp, dtype=torch.float64)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            want[s, :rank] = (R.rms(p[t, off:off + rank], 1e-4) * cn.double())
    close(cache.view(64, rp), want, dtype, exact=1e-6, rough=6e-3)


# ------------------------------------------------------------------ whole models through scheduler and executor
# rms of the logit difference over the rms of the logits: at 19 of 20 positions, and anywhere.  In bf16 a position whose
# softmax or decay amplifies rounding stands out; fp32 is the sharp comparison.
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}
WORST = {"float32": 2e-5, "bfloat16": 8e-2}


def engine_for(tmp_path, name, dtype, max_tokens=512, requests=4, seed=1, raw=None):
    from cubic_serve_b200.utils.trace_run import build_engine
    raw = raw or ALL[name]
    w = tensors(raw, seed)
    return build_engine(str(write(tmp_path / "model", raw, w)), dtype, max_tokens, max_requests=requests), raw, w


def session_for(*a, **k):
    from cubic_serve_b200.runtime.imposed import ImposedSession
    eng, raw, w = engine_for(*a, **k)
    return ImposedSession(eng), raw, R.Oracle(raw, w, torch.float64)


class RoundedProducts(TorchFunctionMode):
    """Operands and results of every matrix product rounded to bf16: the least a bf16 model rounds.  ``scale``: what is rounded
    is this many times larger, so that other values round up and down."""

    def __init__(self, scale):
        super().__init__()
        self.scale = scale

    def __torch_function__(self, func, types, args=(), kwargs=None):
        if func in (torch.Tensor.__matmul__, torch.Tensor.matmul, torch.matmul):
            r = lambda t: (t * self.scale).to(torch.bfloat16).to(t.dtype) / self.scale      # noqa: E731
            return r(func(r(args[0]), r(args[1])))
        return func(*args, **(kwargs or {}))


def error(got, want):
    d = torch.as_tensor(np.asarray(got)).double() - want
    d -= d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


def rounding(oracle, ids, want, dtype):
    """What rounding alone does at every position: a norm over values that cancel amplifies it at some of them."""
    if dtype == "float32":
        return None
    errs = []
    for scale in (1.0, 1.19, 1.41, 1.68):
        with RoundedProducts(scale):
            errs.append(error(oracle.forward(ids)[0], want))
    return torch.stack(errs).amax(0)


def off(got, want, dtype, noise=None):
    err = error(got, want)
    own = torch.zeros_like(err) if noise is None else 3 * noise
    assert (err <= own.clamp_min(WORST[dtype])).all(), (float(err.max()), int(err.argmax()))
    assert (err > own.clamp_min(LIMIT[dtype])).sum() <= max(1, len(err) // 20), sorted(err.tolist())[-12:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALL))
def test_prefill_portions_and_decode_agree(tmp_path, name, dtype):
    """A prompt in one step, in portions down to two tokens, and token by token through the decode graphs."""
    if dtype == "bfloat16" and getattr(ALL[name], "close_calls", False):
        pytest.skip("a position whose choice of experts hangs on rounding is off by an expert: compared in fp32")
    s, raw, oracle = session_for(tmp_path, name, dtype)
    ids = prompt(raw, 113, 4)
    want, _ = oracle.forward(ids)
    noise = rounding(oracle, ids, want, dtype)
    for cuts in ([113], [2] * 6 + [101], [16, 17, 80], [50, 1, 1, 60, 1], [1] * 113, [3, 107, 2, 1]):
        got, i = [], 0
        for c in cuts:
            got.append(s.step([("a", ids[i:i + c], list(range(c)))])[0])
            i += c
        s.end(["a"])
        off(np.concatenate(got), want, dtype, noise)
    s.engine.executor.runner.ws.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name, runs", [("all", 6), ("seq", 4), ("str", 5), ("gat", 7), ("gat_odd", 12)])
def test_residual_after_every_run(tmp_path, name, runs, dtype):
    s, raw, oracle = session_for(tmp_path, name, dtype)
    ids = prompt(raw, 40, 9)
    ref = []
    oracle.forward(ids, trace=ref)
    runner = s.engine.executor.runner
    runner.trace = []
    s.step([("a", ids, [])])
    assert len(runner.trace) == len(ref) == runs
    for got, want in zip(runner.trace, ref):
        close(got, want, torch.float32, exact=1e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["all", "odd", "seq", "seq_odd", "str", "str_odd", "str_select", "gat", "gat_odd"])
def test_unequal_requests_share_steps_pages_and_slots(tmp_path, name, dtype):
    """Up to four live requests, portions beside single tokens, requests that pause, end and make room for others in a pool
    that is too small for all of them."""
    if dtype == "bfloat16" and getattr(ALL[name], "close_calls", False):
        pytest.skip("compared in fp32")
    s, raw, oracle = session_for(tmp_path, name, dtype, max_tokens=288)
    lens = {"a": 100, "b": 37, "c": 1, "d": 60, "e": 90, "f": 33, "g": 16, "h": 130}
    ids = {r: prompt(raw, n, i) for i, (r, n) in enumerate(lens.items())}
    want = {r: oracle.forward(t)[0] for r, t in ids.items()}
    noise = {r: rounding(oracle, t, want[r], dtype) for r, t in ids.items()}
    at = dict.fromkeys(lens, 0)
    rng = np.random.default_rng(3)
    live, todo = [], list(lens)
    pages_seen, steps = set(), 0
    while live or todo:
        while todo and len(live) < 4 and sum(-(-lens[r] // 64) * 64 for r in live + todo[:1]) <= 288:
            live.append(todo.pop(0))
        entries = []
        for r in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                                       # left out of this step
            n = int(rng.choice([1, 1, 2, 3, 16, 29, 64]))
            n = min(n, lens[r] - at[r])
            entries.append((r, ids[r][at[r]:at[r] + n], list(range(n))))
        if not entries:
            continue
        for (r, t, _), got in zip(entries, s.step(entries)):
            here = slice(at[r], at[r] + len(t))
            off(got, want[r][here], dtype, None if noise[r] is None else noise[r][here])
            at[r] += len(t)
        pages_seen |= {p for r in live if r in s.engine.requests for p in s.engine.requests[r].pages}
        done = [r for r in live if at[r] == lens[r]]
        s.end(done)
        live = [r for r in live if r not in done]
        steps += 1
    assert s.engine.pool.num_used == 0 and len(pages_seen) <= 18 and steps > 20
    s.engine.executor.runner.ws.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("raw", [
    config(90, 64, [latent(4, 16, 16, 32, 48, 70, 0.5, 64), delta(2, 1, 16, 32, 4, 64), latent(3, 16, 16, 32, 40, 17, 0.5, 0)], (0, 2, 2)),
    sequential(90, 64, [parallel((4, 2, 16, 70, 0.5, 16, 300.0, (3.0, 60, 8.0, 1.0)), (2, 16, 24, 8.0), (1.0, 0.8), 64),
                        mamba2(2, 24, 16, 1, 4, 2, 48), parallel((3, 1, 24, 17, 0.4, 8, 80.0, None), (1, 20, 16, 4.0), (0.8, 1.1), 0)], 8),
    streams(90, 64, [near(4, 2, 16, 24, 4, 0.6, 16, 300.0, 70, 9, routed(4, 2, 32, 1, 32)), far(3, 1, 16, 16, 0.5, 60, (0.5, 32), 64, 12),
                     near(3, 3, 24, 16, 2, 0.5, 8, 80.0, 17, 33, 0)], 2, 3.0),
    gated(90, 64, [differential(4, 2, 16, 24, 0.5, 16, 300.0, 0.4, 70, clamped(64)), mingru(48, clamped(48, 1.0)),
                   rotated(3, 16, 8, 16, 40, 0.4, 300.0, (3.0, 60, 8.0, 1.0), None), differential(3, 3, 24, 16, 0.5, 8, 80.0, 0.2, 17, None)], (1, 3, 2), 0.8),
], ids=["Bumodra", "Loduzen", "Vimelorn", "Fovunex"])
def test_long_decoding_passes_the_window(tmp_path, raw, dtype):
    """Decoded tokens move every window past the prompt; first tokens of the sequence included."""
    s, raw, oracle = session_for(tmp_path, "", dtype, raw=raw)
    ids = prompt(raw, 230, 2)
    want, _ = oracle.forward(ids)
    got = [s.step([("a", ids[:5], list(range(5)))])[0]]
    for i in range(5, 230):
        got.append(s.step([("a", ids[i:i + 1], [0])])[0])
    off(np.concatenate(got), want, dtype)


def test_far_tokens_reach_through_kept_places_and_the_biased_layer(tmp_path):
    """Changing the first token moves the logits far behind every window as the oracle says: it is kept.  A token that is neither
    kept nor in a window moves them through the layer that sees every earlier token only, one in the middle of nowhere not at all
    without such a layer."""
    from cubic_serve_b200.runtime.imposed import ImposedSession
    from cubic_serve_b200.utils.trace_run import build_engine
    windowed = near(4, 2, 16, 16, 3, 0.5, 8, 100.0, 20, 2, 48)
    for layers, moves in (([windowed], (True, False)), ([windowed, far(2, 1, 16, 16, 0.4, 40, None, 0, 6)], (True, True))):
        raw = streams(80, 64, layers, 2, 4.0)
        w = tensors(raw, 3)
        s = ImposedSession(build_engine(str(write(tmp_path / str(len(layers)), raw, w)), "float32", 512))
        oracle = R.Oracle(raw, w, torch.float64)
        ids = prompt(raw, 300, 7)
        base = oracle.forward(ids)[0][-1]
        for at, expected in zip((0, 120), moves):
            other = ids.copy()
            other[at] = (ids[at] + 11) % 80
            want = oracle.forward(other)[0][-1]
            moved = float((base - want).pow(2).mean().sqrt() / base.pow(2).mean().sqrt())
            assert moved > 20 * LIMIT["float32"] if expected else moved == 0.0, (at, moved)
            for t, row in ((ids, base), (other, want)):
                s.step([("a", t[:150], [])])
                s.step([("a", t[150:299], [])])
                off(s.step([("a", t[299:], [0])])[0], row[None], "float32")
                s.end(["a"])


@pytest.mark.parametrize("raw", [
    config(80, 64, [channel(2, 1, 32, 32, 3, 64), delta(2, 2, 32, 32, 4, 64)]),
    sequential(80, 64, [mamba2(2, 32, 24, 2, 3, 1, 64), parallel((2, 1, 16, 9, 0.3, 8, 100.0, None), (2, 24, 24, 16.0), (0.8, 1.5), 64)], 8),
    gated(80, 64, [mingru(96, clamped(64)), differential(2, 1, 16, 24, 0.3, 8, 100.0, 0.3, 9, clamped(64))], (0, 1, 2)),
], ids=["Bumodra", "Loduzen", "Fovunex"])
def test_far_token_reaches_through_the_state(tmp_path, raw):
    """With slow decays and no attention that far back, changing an early token moves the logits as the oracle says."""
    w = tensors(raw, 3)
    for n in w:
        if n.endswith(".A_log"):
            w[n] = torch.full_like(w[n], -7.0)
        elif n.endswith(".a2.b"):
            w[n] = torch.full_like(w[n], 5.0)
        elif n.endswith(".z.b"):
            w[n] = torch.full_like(w[n], -6.0)
    from cubic_serve_b200.runtime.imposed import ImposedSession
    from cubic_serve_b200.utils.trace_run import build_engine
    s = ImposedSession(build_engine(str(write(tmp_path, raw, w)), "float32", 512))
    oracle = R.Oracle(raw, w, torch.float64)
    ids = prompt(raw, 300, 7)
    other = ids.copy()
    other[3] = (ids[3] + 11) % 80
    la, lb = oracle.forward(ids)[0][-1], oracle.forward(other)[0][-1]
    moved = (la - lb).pow(2).mean().sqrt() / la.pow(2).mean().sqrt()
    assert moved > 20 * LIMIT["float32"]                        # the far token matters, and the comparison can see it
    for t, want in ((ids, la), (other, lb)):
        s.step([("a", t[:150], [])])
        s.step([("a", t[150:299], [])])
        off(s.step([("a", t[299:], [0])])[0], want[None], "float32")
        s.end(["a"])


# ------------------------------------------------------------------ generation through the engine
def greedy(oracle, ids, n):
    lg, st = oracle.forward(ids, last_only=True)
    out = []
    for _ in range(n):
        out.append(int(lg[0].argmax()))
        lg, st = oracle.forward([out[-1]], st, last_only=True)
    return out


def serving_backend(model, *flags):
    from cubic_serve_b200.cli import build_parser, parse_speculative_config
    from cubic_serve_b200.runtime.serving import build_backend
    args = build_parser().parse_args(["serve", str(model), "--max-running-requests", "6", "--gpu-memory-gib", "8", "--gpu-reserve-gib",
                                      "0.5", "--token-budget", "64", "--prefill-chunk-tokens", "48", "--max-model-len", "256", *flags])
    backend, _ = build_backend(args, [0], 1, parse_speculative_config(None), 8, 8)
    backend.close()
    return backend.engine


@pytest.mark.parametrize("prefix", [False, True])
@pytest.mark.parametrize("raw", [
    config(300, 64, [delta(2, 1, 16, 16, 3, 64), latent(2, 16, 16, 24, 32, 20, 0.25, 0), channel(2, 2, 16, 16, 2, 48)], (0, 2, 2)),
    sequential(300, 64, [mamba2(2, 16, 8, 1, 3, 2, 48), parallel((4, 2, 16, 20, 0.3, 8, 90.0, (2.0, 50, 4.0, 1.0)), (2, 12, 16, 8.0), (0.9, 0.8), 64)], 8),
    streams(300, 64, [near(4, 2, 16, 24, 3, 0.5, 8, 90.0, 20, 3, routed(4, 2, 32, 1, 24)), far(2, 1, 16, 16, 0.3, 20, (0.4, 8), 48)], 2, 3.0),
    gated(300, 64, [rotated(2, 16, 8, 16, 32, 0.3, 90.0, (2.0, 50, 4.0, 1.0), clamped(64)), mingru(48, None),
                    differential(4, 2, 16, 24, 0.3, 8, 90.0, 0.4, 20, clamped(48))], (1, 3, 2), 0.5),
], ids=["Bumodra", "Loduzen", "Vimelorn", "Fovunex"])
def test_greedy_generation_through_the_serving_stack(tmp_path, raw, prefix):
    """``cubic serve`` with --dtype float32: scheduler, prefix cache with state snapshots, overlapped decode graphs, sampler."""
    from cubic_serve_b200.runtime.scheduler import SamplingParams
    w = tensors(raw, 5)
    eng = serving_backend(write(tmp_path, raw, w), "--dtype", "float32", "--prefix-cache" if prefix else "--no-prefix-cache")
    oracle = R.Oracle(raw, w, torch.float64)
    shared = prompt(raw, 70, 0)
    prompts = [shared, prompt(raw, 1, 1), shared + prompt(raw, 9, 2), prompt(raw, 130, 3), shared[:64] + prompt(raw, 3, 4)]
    want = [greedy(oracle, p, 12) for p in prompts]
    for turn in range(2):                                       # the second turn resumes from cached prefixes
        got = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
        assert got == want, turn
    assert (eng.prefix.hit_rate > 0) == prefix
    eng.executor.runner.ws.check_status()


@pytest.mark.parametrize("name", ["all", "seq", "str", "gat"])
def test_bf16_serving_samples_and_preempts(tmp_path, name):
    """bf16 through the same stack: greedy tokens are the oracle's wherever its margin is clear, seeded sampling repeats, and a
    pool that is too small for all requests recomputes the preempted ones to the same tokens."""
    from cubic_serve_b200.executor.gpu_executor import GpuExecutor
    from cubic_serve_b200.models import registry
    from cubic_serve_b200.models.checkpoint import admit_checkpoint
    from cubic_serve_b200.runtime.engine import LLMEngine
    from cubic_serve_b200.runtime.scheduler import SamplingParams, SchedulerConfig
    raw = ALL[name]
    w = tensors(raw, 6)
    ck = admit_checkpoint(write(tmp_path, raw, w))
    defn = registry.get("layered")
    outs = []
    for pages in (64, 9):
        runner = defn.build_runner(ck.cfg, defn.load_weights(ck, torch.device(DEV)), num_pages=pages, max_tokens=64, max_requests=3)
        ex = GpuExecutor(runner, max_rows=3, max_prefill_tokens=64, max_model_len=96)
        assert ex.capture_decode_graphs() == [1, 2] and ex.execution_plan is not None
        eng = LLMEngine(ex, num_pages=pages, scheduler_config=SchedulerConfig(max_running_requests=3, max_batched_tokens=64,
                                                                              max_model_len=96, enable_prefix_cache=False))
        outs.append(eng.generate([prompt(raw, n, n) for n in (40, 33, 20)], SamplingParams(max_tokens=24, ignore_eos=True)))
        sampled = [eng.generate([prompt(raw, 12, 8)], SamplingParams(max_tokens=10, temperature=0.8, top_k=5, seed=3, ignore_eos=True))
                   for _ in range(2)]
        assert sampled[0] == sampled[1]
    oracle = R.Oracle(raw, w, torch.float64)
    for n, out, again in zip((40, 33, 20), *outs):
        lg, _ = oracle.forward(prompt(raw, n, n) + out)
        for i, tok in enumerate(out):                           # the oracle on the generated sequence
            row = lg[n - 1 + i]
            top = row.topk(2).values
            assert tok == int(row.argmax()) or float(row.max() - row[tok]) < 0.15 * float(row.std()), (i, float(top[0] - top[1]))
        same = next((i for i, (x, y) in enumerate(zip(out, again)) if x != y), len(out))
        assert same > 8                                         # recomputed context: equal to rounding


@pytest.mark.parametrize("name", ["small", "seq_small", "str_small", "gat_small"])
def test_trace_run_program(tmp_path, name):
    """The program itself: lines in, files out, two requests in one step, exit code 0."""
    import json
    import subprocess
    raw = ALL[name]
    w = tensors(raw, 2)
    write(tmp_path / "m", raw, w)
    a, b = prompt(raw, 30, 1), prompt(raw, 21, 2)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": a[:29], "want": [0, 28]}, {"id": "y", "tokens": b[:20], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b[20:], "want": [0]}, {"id": "x", "tokens": a[29:], "want": [0]}],
              "end": ["x", "y"]}]
    root = Path(__file__).resolve().parents[1]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "64"], input="".join(json.dumps(l) + "\n" for l in lines), text=True, capture_output=True)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
        oracle = R.Oracle(raw, w, torch.float64)
        la, lb = oracle.forward(a)[0], oracle.forward(b)[0]
        off(np.fromfile(out / "0.f32", "<f4").reshape(2, -1), la[[0, 28]], dtype)
        off(np.fromfile(out / "1.f32", "<f4").reshape(2, -1), torch.stack([lb[20], la[29]]), dtype)


def test_imposed_steps_of_a_quantized_decoder(tmp_path):
    """The same session drives the other native decoders: portions and decode graphs give the logits of one pass."""
    from cubic_serve_b200.models.checkpoint import write_random_checkpoint
    from cubic_serve_b200.models.config import ModelConfig, QuantSpec
    from cubic_serve_b200.runtime.imposed import ImposedSession
    from cubic_serve_b200.utils.trace_run import build_engine
    cfg = ModelConfig(name="dense", num_layers=2, hidden_size=256, num_q_heads=4, num_kv_heads=2, head_dim=128, intermediate_size=512,
                      vocab_size=512, quant=QuantSpec("cubic", 4, 128))
    s = ImposedSession(build_engine(str(write_random_checkpoint(tmp_path, cfg, seed=1, std=0.05)), "bfloat16", 256))
    ids = np.random.default_rng(0).integers(0, 512, 90).tolist()
    whole = s.step([("a", ids, list(range(90)))])[0]
    s.end(["a"])
    got, i = [], 0
    for c in (40, 1, 2, 46, 1):
        got.append(s.step([("b", ids[i:i + c], list(range(c)))])[0])
        i += c
    d = torch.as_tensor(np.concatenate(got) - whole).double()
    assert (d.pow(2).mean(-1).sqrt() < 3e-2 * torch.as_tensor(whole).double().pow(2).mean(-1).sqrt()).all()
    with pytest.raises(SystemExit) as e:
        build_engine(str(tmp_path), "float32", 256)
    assert e.value.code == 3
