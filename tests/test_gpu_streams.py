"""Mechanisms of the layered decoders on several residual streams on the GPU, each alone against the oracle's equations: convolved and
normed queries, keys and values, attention with kept tokens, distance biases and values of another width, streams, scored experts."""
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
from test_gpu_layered import DEV, DTYPES, close, segs  # noqa: E402
from test_gpu_sequential import GqaCase  # noqa: E402

from cubic_serve_b200.models import layered_reference as R  # noqa: E402

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m, n, split, k, how", [(1, 40, 8, 64, {}), (17, 200, 72, 128, {}), (300, 260, 16, 192, {}), (33, 300, 128, 256, {"stream_k": True}),
                                                 (520, 384, 96, 128, {"stream_k": True}), (40, 136, 24, 1024, {"splits": 2}), (9, 72, 8, 1024, {"splits": 5})])
def test_fp32_output_beside_squared_relu(dtype, m, n, split, k, how):
    """The router's logits leave in fp32 beside the activated features of the same product."""
    from cubic_serve_b200.ops import kernels as K, wq_pack
    if dtype == torch.float32 and how:
        pytest.skip("the fp32 product has one form")
    g = torch.Generator().manual_seed(m + n)
    x = torch.randn(m, k, generator=g).to(dtype)
    w = wq_pack.pack_bf16(torch.randn(n, k, generator=g) / k ** 0.5)
    want = x.double() @ w.codes.double().t()
    z = torch.full((m, split), 7.0, device=DEV)
    wide = torch.full((m, 16 + n - split + 8), 5.0, dtype=dtype, device=DEV)
    K.wide_gemm(x.to(DEV), w.to(DEV), z, relu2=wide[:, 16:16 + n - split], split=split, **how)
    close(z, want[:, :split], torch.float32, exact=1e-5)
    close(wide[:, 16:16 + n - split], want[:, split:].clamp_min(0) ** 2, dtype, rough=1.5e-2)
    assert (wide[:, :16] == 5).all() and (wide[:, 16 + n - split:] == 5).all()
    K.workspace(torch.device(DEV)).check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m, ff, k, how", [(1, 16, 64, {}), (17, 80, 128, {}), (300, 144, 192, {}), (33, 160, 256, {"stream_k": True}), (40, 96, 1024, {"splits": 2})])
def test_gated_silu_product(dtype, m, ff, k, how):
    from cubic_serve_b200.ops import kernels as K, wq_pack
    if dtype == torch.float32 and how:
        pytest.skip("the fp32 product has one form")
    g = torch.Generator().manual_seed(m + ff)
    x = (torch.randn(m, k, generator=g) * 1.5).to(dtype)
    w = wq_pack.pack_bf16(torch.cat([torch.randn(ff, k, generator=g) / k ** 0.5 for _ in range(2)]))
    want = R.silu(x.double() @ w.codes[:ff].double().t()) * (x.double() @ w.codes[ff:].double().t())
    out = torch.full((m, ff + 16), 7.0, dtype=dtype, device=DEV)
    K.wide_gemm(x.to(DEV), wq_pack.swiglu_interleave(w).to(DEV), out[:, 8:8 + ff], glu="silu", **how)
    close(out[:, 8:8 + ff], want, dtype, exact=1e-5, rough=1e-2)
    assert (out[:, :8] == 7).all() and (out[:, 8 + ff:] == 7).all()


# ------------------------------------------------------------------ queries, keys and values
class Qkv:
    """Projected rows of several requests and where their keys and values go."""

    def __init__(self, H, G, d, e, dtype, seed=0, taps=1):
        g = torch.Generator().manual_seed(seed)
        self.g, self.H, self.G, self.d, self.e, self.dtype, self.taps = g, H, G, d, e, dtype, taps
        self.P = -(-max(d, e) // 64) * 64
        r8 = lambda n: -(-n // 8) * 8                                                  # noqa: E731
        k = r8(H * d)
        self.rel = (0, k, k + r8(G * d))                                              # offsets from the first query on
        self.width = r8(self.rel[2] + G * e)
        self.offs = tuple(8 + o for o in self.rel)

    def columns(self, q, k, v):
        """``[n, ...]`` rows of q, k and v where the kernel reads them; the columns between hold garbage."""
        x = torch.full((q.shape[0], 8 + self.width + 8), 50.0).to(self.dtype)
        for o, t in zip(self.offs, (q, k, v)):
            x[:, o:o + t.shape[1]] = t
        return x.to(DEV)

    def rows(self, n):
        return tuple(torch.randn(n, c, generator=self.g).to(self.dtype) for c in (self.H * self.d, self.G * self.d, self.G * self.e))

    def outputs(self, T, pages):
        return (torch.full((T, self.H * self.P), 9.0, dtype=self.dtype, device=DEV),
                torch.full((pages, self.G, 2, 16, self.P), 3.0, dtype=self.dtype, device=DEV))

    def check(self, q, cache, slots, wq, wk, wv, untouched=True):
        """Queries in order, keys and values at their slots, zeros behind their widths; other rows are untouched."""
        T = wq.shape[0]
        q = q[:T].view(T, self.H, self.P)
        close(q[:, :, :self.d], wq, self.dtype, exact=5e-6, rough=8e-3)
        assert (q[:, :, self.d:] == 0).all()
        rows = cache.permute(2, 0, 3, 1, 4).reshape(2, -1, self.G, self.P)
        at = torch.tensor([s for s in slots if s >= 0])
        live = torch.tensor([i for i, s in enumerate(slots) if s >= 0])
        for r, w, want in ((rows[0], self.d, wk), (rows[1], self.e, wv)):
            close(r[at][:, :, :w], want[live], self.dtype, exact=5e-6, rough=8e-3)
            assert (r[at][:, :, w:] == 0).all()
        if untouched:
            rest = torch.ones(rows.shape[1], dtype=torch.bool)
            rest[at] = False
            assert (rows[:, rest] == 3).all()


QKV_SHAPES = [(6, 2, 24, 40, 6, 3), (4, 4, 64, 64, 32, 4), (3, 1, 13, 9, 3, 6), (5, 5, 18, 21, 0, 2), (40, 1, 128, 128, 64, 1), (2, 1, 200, 136, 20, 4),
              (2, 2, 130, 256, 65, 3), (8, 2, 48, 16, 10, 16), (1, 1, 7, 5, 2, 5), (2, 1, 136, 24, 68, 2)]


def conv_want(c, w, past, q, k, v, pos, pairs, base, eps):
    out, new = [], []
    for t, x, o in zip("qkv", (q, k, v), c.rel):
        wt = w[:, o:o + x.shape[1]].t().double()
        y, p = R.plain_short_conv(x.double(), wt, past[t])
        out.append(y)
        new.append(p)
    n = q.shape[0]
    turned = []
    for y in out[:2]:
        y = y.view(n, -1, c.d)
        y = torch.stack([R.rotate_halves(y[t:t + 1], int(pos[t]), 2 * pairs, base)[0] for t in range(n)])
        turned.append(R.rms(y, eps))
    return turned[0], turned[1], out[2].view(n, c.G, c.e), dict(zip("qkv", new))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, e, pairs, taps", QKV_SHAPES)
def test_conv_qkv_in_portions_and_batches(dtype, H, G, d, e, pairs, taps):
    """Portions down to one token on a slot with stale contents, unequal requests in one step, padding rows and segments, far
    positions; other slots' history stays."""
    from cubic_serve_b200.ops import kernels as K
    c = Qkv(H, G, d, e, dtype, seed=H + d, taps=taps)
    base, eps, slots_n = 300.0, 1e-4, 5
    w = torch.zeros(taps, c.width)
    for o, n in zip(c.rel, (H * d, G * d, G * e)):
        w[:, o:o + n] = torch.randn(taps, n, generator=c.g) / taps ** 0.5
    exact = torch.tensor([base ** (-i / max(pairs, 1)) for i in range(pairs)], dtype=torch.float64)
    freq = torch.stack([exact.float(), (exact - exact.float().double()).float()]).to(DEV).contiguous()
    state = torch.full((slots_n, max(1, taps - 1), c.width), 7.0, dtype=dtype, device=DEV)
    fresh = lambda: {t: torch.zeros(taps - 1, n, dtype=torch.float64) for t, n in zip("qkv", (H * d, G * d, G * e))}   # noqa: E731
    past = {1: fresh(), 3: fresh(), 0: fresh()}
    at = {1: 0, 3: 0, 0: 0}
    far = {1: 0, 3: 990000, 0: 77}                       # added to the rotary positions only: a request may be far along
    page = {1: 0, 3: 6, 0: 12}
    # (slot, tokens) of every step; slot None: a padding segment
    for step in ([(1, 2)], [(1, 37)], [(3, 16), (1, 17), (0, 1)], [(1, 2), (3, 33)], [(1, 1), (None, 0), (3, 1), (0, 1)], [(3, 2), (0, 18)], [(1, 1)]):
        decode = all(n <= 1 for _, n in step)
        rows, want, slots, pos, spans = [], [], [], [], []
        for slot, n in step:
            if slot is None:
                spans.append((0, 0, 0))
                if decode:                              # row j belongs to segment j
                    rows.append(c.rows(1))
                    want.append(None)
                    slots.append(-1)
                    pos.append(0)
                continue
            x = c.rows(n)
            first = at[slot]
            p = torch.arange(first, first + n) + far[slot]
            *y, past[slot] = conv_want(c, w, past[slot], *x, p, pairs, base, eps)
            rows.append(x)
            want.append(y)
            slots += [page[slot] * 16 + first + i for i in range(n)]
            pos += p.tolist()
            spans.append((n, slot, first))
            at[slot] += n
        T = len(slots)
        seg = segs(spans)
        if decode:
            seg.row0 = torch.arange(T, dtype=torch.int32, device=DEV)
        q, cache = c.outputs(T, 18)
        K.conv_qkv(c.columns(*(torch.cat(t) for t in zip(*rows))), c.offs, w.to(DEV), state if taps > 1 else None, freq,
                   torch.tensor(pos, dtype=torch.int32, device=DEV), torch.tensor(slots, dtype=torch.int32, device=DEV), seg, q, cache, H, d, e, eps)
        live = [i for i, y in enumerate(want) if y is not None]
        keep = torch.tensor([i for i, s in enumerate(slots) if s >= 0])
        c.check(q.view(T, -1)[keep.to(DEV)], cache, [s for s in slots if s >= 0], *(torch.cat([want[i][j] for i in live]) for j in range(3)))
        if taps > 1:
            for slot in (1, 3, 0):
                for t, o in zip("qkv", c.rel):
                    n = past[slot][t].shape[1]
                    if at[slot]:
                        close(state[slot, :, o:o + n], past[slot][t], torch.float32, exact=0)
            assert (state[2] == 7).all() and (state[4] == 7).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, e", [s[:4] for s in QKV_SHAPES])
@pytest.mark.parametrize("temp", [(0.0, 0), (0.6, 7), (0.25, 1)])
def test_norm_qkv(dtype, H, G, d, e, temp):
    """Norms over whole projections (tiny rows: eps decides), the query factor around its steps."""
    from cubic_serve_b200.ops import kernels as K
    c = Qkv(H, G, d, e, dtype, seed=H)
    x = c.rows(8)
    for t in x:
        t[3] *= 1e-3
    qn, kn = 1 + 0.3 * torch.randn(H * d, generator=c.g), 1 + 0.3 * torch.randn(G * d, generator=c.g)
    pos = [0, 5, 6, 7, 12, 13, 1000000, 20]
    slots = [17, 63, -1, 0, 32, 31, 5, 40]
    q, cache = c.outputs(8, 4)
    K.norm_qkv(c.columns(*x), c.offs, qn.to(DEV), kn.to(DEV), torch.tensor(pos, dtype=torch.int32, device=DEV),
               torch.tensor(slots, dtype=torch.int32, device=DEV), q, cache, H, d, e, 1e-4, temp)
    f = torch.tensor([1 + temp[0] * torch.log(torch.tensor((p + 1) // temp[1] + 1.0, dtype=torch.float64)) if temp[1] else 1.0 for p in pos],
                     dtype=torch.float64).unsqueeze(1)
    wq, wk = R.rms(x[0].double(), 1e-4) * qn.double() * f, R.rms(x[1].double(), 1e-4) * kn.double()
    c.check(q, cache, slots, wq.view(8, H, d), wk.view(8, G, d), x[2].double().view(8, G, e))
    if temp == (0.6, 7) and dtype == torch.float32:     # positions 5 and 6 lie on two sides of a step
        assert abs(float(f[2] / f[1]) - (1 + 0.6 * 0.6931471805599453)) < 1e-9


# ------------------------------------------------------------------ attention
class KeptCase(GqaCase):
    """Values of a width of their own, kept first tokens, a bias by distance and head."""

    def __init__(self, lens, H, G, d, e, dtype, seed=0, bias=None, gain=1.0):
        g = torch.Generator().manual_seed(seed + 7)
        self.e = e
        super().__init__(lens, H, G, max(d, e), dtype, seed, gain=gain)
        self.k = [t[..., :d] for t in self.k]
        self.q = [t[..., :d] for t in self.q]
        self.v = [t[..., :e] for t in self.v]
        self.d = d
        self.bias = None if bias is None else (1.5 * torch.randn(bias + 1, H, generator=g))
        self.fill()

    def fill(self):
        self.cache = torch.full((self.pages, self.G, 2, 16, self.P), 1e4, dtype=self.dtype)
        for r, n in enumerate(self.lens):
            for p in range(-(-n // 16)):
                page, m = self.cache[self.table[r, p]], min(16, n - 16 * p)
                for which, t in ((0, self.k[r]), (1, self.v[r])):
                    page[:, which, :m] = 0
                    page[:, which, :m, :t.shape[2]] = t[16 * p:16 * p + m].transpose(0, 1)

    def run(self, spans, window, scale, keep=0, splits=None, decode=None):
        from cubic_serve_b200.ops import kernels as K
        T = sum(n for _, _, n in spans)
        q = torch.zeros(T, self.H, self.P, dtype=self.dtype)
        q[:, :, :self.d] = torch.cat([self.q[r][first:first + n] for r, first, n in spans])
        wide = torch.full((T, -(-self.H * self.e // 8) * 8 + 16), 3.0, dtype=self.dtype, device=DEV)
        out = wide[:, 8:8 + self.H * self.e]
        K.gqa_attention(q.view(T, -1).to(DEV), self.cache.to(DEV), self.table.to(DEV), segs([(n, r, first) for r, first, n in spans]), out, self.H,
                        self.e, window, scale, decode=T == len(spans) if decode is None else decode, splits=splits, keep=keep,
                        bias=None if self.bias is None else self.bias.to(DEV))
        assert (wide[:, :8] == 3).all() and (wide[:, 8 + self.H * self.e:] == 3).all()
        return out.reshape(T, self.H, self.e).split([n for _, _, n in spans])

    def want(self, r, first, n, window, scale, keep=0):
        k, v, q = self.k[r][:first + n].double(), self.v[r][:first + n].double(), self.q[r][first:first + n].double()
        bias = None
        if self.bias is not None:
            gap = (torch.arange(first, first + n).unsqueeze(1) - torch.arange(first + n)).clamp(0, self.bias.shape[0] - 1)
            bias = self.bias.double()[gap].permute(2, 0, 1)
        return R.masked_attention(q, k, v, R.kept_window(first, n, first + n, window or None, keep), scale, bias)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, e, window, keep, bias", [
    (6, 2, 64, 40, 37, 5, None), (3, 1, 13, 21, 30, 16, None), (32, 8, 128, 128, 90, 33, None), (40, 1, 72, 136, 16, 64, None), (4, 4, 200, 64, 50, 70, None),
    (1, 1, 24, 24, 1, 1, None), (70, 1, 128, 24, 20, 100, None), (6, 2, 64, 40, 0, 0, 30), (3, 1, 13, 9, 0, 0, 1), (32, 8, 128, 128, 0, 0, 64),
    (20, 1, 72, 200, 0, 0, 300), (40, 1, 48, 48, 0, 0, 90), (2, 1, 256, 16, 0, 0, 20), (150, 1, 40, 33, 0, 0, 50), (16, 1, 64, 64, 0, 0, 700), (5, 5, 80, 80, 33, 18, 40)])
def test_kept_and_biased_attention_prefill_portions_and_decode(dtype, H, G, d, e, window, keep, bias):
    lens = (230, 3, 61, 16)
    case = KeptCase(lens, H, G, d, e, dtype, seed=H, bias=bias)
    scale = 1.5 / d ** 0.5
    for r, o in enumerate(case.run([(r, 0, n) for r, n in enumerate(lens)], window, scale, keep)):
        close(o, case.want(r, 0, lens[r], window, scale, keep), dtype, rough=1.2e-2)
    spans = [(2, 40, 21), (0, 229, 1), (1, 1, 2), (3, 15, 1), (0, 150, 70)]
    for (r, first, n), o in zip(spans, case.run(spans, window, scale, keep)):
        close(o, case.want(r, first, n, window, scale, keep), dtype, rough=1.2e-2)
    spans = [(r, n - 1, 1) for r, n in enumerate(lens)]
    for splits in (None, 1, 2, 7):
        for (r, first, n), o in zip(spans, case.run(spans, window, scale, keep, splits=splits)):
            close(o, case.want(r, first, n, window, scale, keep), dtype, rough=1.2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window, keep", [(1, 1), (16, 5), (17, 16), (33, 17), (64, 3), (65, 64), (20, 65), (100, 31)])
def test_kept_edge_shows_one_key(dtype, window, keep):
    """One key carries a score that outweighs all others and a value nothing else has: it is seen by the queries whose window holds
    it, and by all later ones if it is among the first tokens."""
    n, H, G, d = 220, 6, 2, 40
    for j in sorted({0, keep - 1, keep, keep + 1, 16, 63, 64}):
        case = KeptCase((n,), H, G, d, d, dtype, seed=window, gain=0.1)
        case.q[0] *= 0.1
        case.q[0][:, :, 0] = 6.0
        case.k[0][:, :, 0], case.v[0][:, :, 1] = 0.0, 0.0
        case.k[0][j, :, 0], case.v[0][j, :, 1] = 6.0, 40.0
        case.fill()
        seen = torch.tensor([i >= j and (i - j < window or j < keep) for i in range(n)])
        for spans in ([(0, 0, n)], [(0, 0, 100), ], [(0, 101, 119)]):
            first = spans[0][1]
            out = case.run(spans, window, 1.0, keep)[0][:, :, 1].float().cpu()
            want = seen[first:first + out.shape[0]]
            assert ((out > 10).all(1) == want).all() and ((out.abs() < 1).all(1) == ~want).all(), (window, keep, j, spans)
        for i in (j + window - 1, j + window, n - 1):
            if j <= i < n:
                for splits in (None, 4):
                    one = case.run([(0, i, 1)], window, 1.0, keep, splits=splits)[0][0, :, 1].float().cpu()
                    assert ((one > 10).all() if seen[i] else (one.abs() < 1).all()), (window, keep, j, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("far", [3, 40, 64, 900])
def test_bias_of_one_distance_shows_one_key(dtype, far):
    """A bias that stands out at one distance (and head) picks exactly the key that far back; the last row serves all farther keys."""
    n, H = 170, 4
    case = KeptCase((n,), H, 2, 32, 32, dtype, seed=far, gain=0.05, bias=far)
    for dist in (0, 1, far // 2, far):
        if dist > n:
            continue
        case.bias = torch.zeros(far + 1, H)
        case.bias[dist, 1] = 9.0
        for spans in ([(0, 0, n)], [(0, 60, 110)], [(0, 169, 1)], [(0, 64, 1)]):
            got = case.run(spans, 0, 0.2)[0]
            close(got, case.want(*spans[0], 0, 0.2), dtype, rough=1.2e-2)


# ------------------------------------------------------------------ residual streams
STREAM_SHAPES = [(2, 64), (1, 192), (3, 67), (2, 2048), (4, 68), (8, 96), (5, 130), (2, 8704), (3, 8192)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S, W", STREAM_SHAPES)
def test_stream_embedding_step_and_norm(dtype, S, W):
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(S * W)
    rnd = lambda *s: torch.randn(*s, generator=g)                                       # noqa: E731
    table, ids = rnd(11, W).to(torch.bfloat16), torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32)
    w_in, mix, out, nw = rnd(S), rnd(S, S), rnd(S), 1 + 0.2 * rnd(W)
    ld = -(-W // 64) * 64
    x, h = torch.zeros(5, S, W, device=DEV), torch.full((5, ld), 9.0, dtype=dtype, device=DEV)
    K.stream_embed(ids.to(DEV), table.to(DEV), 7.25, x, w_in.to(DEV), nw.to(DEV), h, 1e-3)
    e = (table.double()[ids.long()] * 7.25).repeat(S, 1, 1)
    assert torch.equal(x.double().cpu().transpose(0, 1), e) and (h[:, W:] == 9).all()
    close(h[:, :W], R.rms(R.stream_read(e, w_in.double()), 1e-3) * nw.double(), dtype, exact=3e-6, rough=6e-3)
    # streams that differ, a result beside them, the next sublayer's input
    xs = rnd(S, 5, W)
    x = xs.transpose(0, 1).contiguous().to(DEV)
    y = rnd(5, -(-W // 8) * 8).to(dtype)
    want = R.stream_write(xs.double(), mix.double(), out.double(), y[:, :W].double())
    K.stream_step(x, y.to(DEV)[:, :W], mix.to(DEV), out.to(DEV), h, 1e-3, w_in.to(DEV), nw.to(DEV))
    close(x.transpose(0, 1), want, torch.float32, exact=2e-6)
    close(h[:, :W], R.rms(R.stream_read(want, w_in.double()), 1e-3) * nw.double(), dtype, exact=2e-5, rough=6e-3)
    assert (h[:, W:] == 9).all()
    before = h.clone()                                                                  # nothing reads the last sublayer's streams
    K.stream_step(x, y.to(DEV)[:, :W], mix.to(DEV), out.to(DEV), h, 1e-3)
    want = R.stream_write(want, mix.double(), out.double(), y[:, :W].double())
    close(x.transpose(0, 1), want, torch.float32, exact=4e-6)
    assert torch.equal(h, before)
    rows = torch.tensor([4, 0, 2], device=DEV)
    K.stream_norm(x, nw.to(DEV), h, 1e-3, rows=rows)
    close(h[:3, :W], (R.rms(want.sum(0), 1e-3) * nw.double())[[4, 0, 2]], dtype, exact=1e-4, rough=6e-3)
    assert torch.equal(h[3:], before[3:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S, W, top", [(2, 64, 3), (3, 67, 1), (1, 2048, 6), (4, 68, 32), (2, 8704, 2)])
@pytest.mark.parametrize("shared", [True, False])
def test_stream_step_puts_routed_results_together(dtype, S, W, top, shared):
    """Results by place (some routes have none), the token itself, the gated shared expert, through the same step."""
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(S + W)
    rnd = lambda *s: torch.randn(*s, generator=g)                                       # noqa: E731
    T = 6
    xs, w_in, mix, out, nw = rnd(S, T, W), rnd(S), rnd(S, S), rnd(S), 1 + 0.2 * rnd(W)
    ld = -(-W // 64) * 64
    h0, rows, y = rnd(T, ld).to(dtype), rnd(T * top, -(-W // 8) * 8).to(dtype), rnd(T, -(-W // 8) * 8).to(dtype)
    pos = torch.randperm(T * top, generator=g).to(torch.int32).view(T, top)
    pos[1] = -1
    pos[2, 0] = -1
    weight, own, gate = torch.rand(T, top, generator=g), torch.rand(T, generator=g), rnd(T, 3)
    own[4] = 0.0
    res = own.double().unsqueeze(1) * h0[:, :W].double()
    for t in range(T):
        for k in range(top):
            if pos[t, k] >= 0:
                res[t] += weight[t, k].double() * rows[pos[t, k], :W].double()
    if shared:
        res = res + y[:, :W].double() / (1 + torch.exp(-gate[:, 1:2].double()))
    want = R.stream_write(xs.double(), mix.double(), out.double(), res)
    x, h, gd = xs.transpose(0, 1).contiguous().to(DEV), h0.to(DEV), gate.to(DEV)
    routes = K.RoutedResult(rows.to(DEV)[:, :W], pos.to(DEV).view(-1), weight.to(DEV).view(-1), own.to(DEV), gd[:, 1:2] if shared else None, top)
    K.stream_step(x, y.to(DEV)[:, :W] if shared else None, mix.to(DEV), out.to(DEV), h, 1e-3, w_in.to(DEV), nw.to(DEV), routes)
    close(x.transpose(0, 1), want, torch.float32, exact=3e-6)
    close(h[:, :W], R.rms(R.stream_read(want, w_in.double()), 1e-3) * nw.double(), dtype, exact=2e-5, rough=6e-3)


# ------------------------------------------------------------------ scored experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, experts, identity, top, W", [(1, 5, 3, 3, 64), (7, 1, 0, 1, 96), (50, 40, 9, 6, 67), (300, 8, 0, 2, 128), (33, 250, 6, 32, 64),
                                                          (700, 3, 1, 4, 72), (16, 2, 30, 2, 64)])
def test_scored_routing_and_grouped_products(dtype, T, experts, identity, top, W):
    """Choices and weights are the oracle's, places are a permutation by expert, the counters are zero again; products of all
    experts over the places, also with experts that have no token or all of them."""
    from cubic_serve_b200.ops import kernels as K, wq_pack
    g = torch.Generator().manual_seed(T + experts)
    n, kp, ff = experts + identity, -(-W // 64) * 64, 56
    h = torch.zeros(T, kp, dtype=dtype)
    h[:, :W] = torch.randn(T, W, generator=g).to(dtype)
    z = torch.randn(T, n + 3, generator=g) * 3
    corr = 0.2 * torch.randn(n, generator=g)
    up, down = torch.zeros(experts, ff, kp, dtype=torch.bfloat16), torch.zeros(experts, W, 64, dtype=torch.bfloat16)
    up[:, :, :W] = torch.randn(experts, ff, W, generator=g) / W ** 0.5
    down[:, :, :ff] = torch.randn(experts, W, ff, generator=g) / ff ** 0.5
    packed = lambda t: wq_pack.PackedWeight(wq_pack.FMT_BF16, t.shape[1], t.shape[2], t.shape[2], t.to(DEV), None)        # noqa: E731
    sc = K.ScoredScratch(T + 5, top, experts, W, kp, dtype, DEV)
    act = torch.zeros((T + 5) * top, 64, dtype=dtype, device=DEV)
    for turn in range(3):
        if turn == 1:
            corr = torch.zeros(n)
            corr[0] = 2.0                                                               # everybody chooses the first
        if turn == 2:
            z[:] = 0.5                                                                  # ties go to the first ones
            corr[:] = 0.0
        mb = K.scored_route(z.to(DEV)[:, :n], corr.to(DEV), h.to(DEV), W, experts, top, sc)
        chosen, weight = R.route(z[:, :n].double(), corr.double(), top)
        ids, pos = sc.ids[:T * top].cpu().view(T, top), sc.pos[:T * top].cpu().view(T, top)
        assert torch.equal(ids, torch.where(chosen < experts, chosen, -1).int())
        close(sc.weight[:T * top].view(T, top), weight, torch.float32, exact=2e-6)
        own = torch.where(chosen >= experts, weight, torch.zeros_like(weight)).sum(1)
        assert (sc.self_weight[:T].double().cpu() - own).abs().max() < 2e-6 and (sc.counts == 0).all()
        live = ids >= 0
        order = ids[live][torch.argsort(pos[live])]
        assert sorted(pos[live].tolist()) == list(range(int(live.sum()))) and (pos[~live] == -1).all() and (order.diff() >= 0).all()
        tiles = sc.tiles.cpu().tolist()
        items = [tiles[1 + 3 * i:4 + 3 * i] for i in range(tiles[0])]
        assert all(0 < r <= mb for _, _, r in items) and sum(r for _, _, r in items) == len(order)
        assert all((order[a:a + r] == e).all() for e, a, r in items)
        assert torch.equal(sc.xs.cpu()[pos[live].long(), :W], h[live.nonzero()[:, 0], :W])
        K.grouped_gemm(sc.xs, packed(up), act[:, :ff], sc, T * top, mb, relu2=True)
        K.grouped_gemm(act, packed(down), sc.ys[:, :W], sc, T * top, mb)
        if len(order):
            t_of = live.nonzero()[torch.argsort(pos[live]), 0]
            a = torch.einsum("rk,rnk->rn", h.double()[t_of], up.double()[order.long()]).clamp_min(0) ** 2
            close(act[:len(order), :ff], a, dtype, exact=1e-5, rough=1.5e-2)
            y = torch.einsum("rk,rnk->rn", act[:len(order), :ff].double().cpu(), down.double()[order.long()][:, :, :ff])
            close(sc.ys[:len(order), :W], y, dtype, exact=1e-5, rough=6e-3)
    K.workspace(torch.device(DEV)).check_status()
