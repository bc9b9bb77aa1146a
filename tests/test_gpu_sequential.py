"""Mechanisms of the sequential layered decoders on the GPU, each alone against the oracle's equations: gated products, token side
inputs, sink attention over paged keys and values, gated linear attention, state-space recurrences."""
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
from test_gpu_layered import DEV, DTYPES, close, segs  # noqa: E402

from cubic_serve_b200.models import layered_reference as R  # noqa: E402

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ products and rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m, ff, k, how", [(1, 16, 64, {}), (17, 80, 128, {}), (5, 48, 640, {}), (300, 144, 192, {}), (33, 160, 256, {"stream_k": True}),
                                           (520, 192, 128, {"stream_k": True}), (40, 96, 1024, {"splits": 2}), (9, 64, 1024, {"splits": 5})])
def test_gated_gelu_product(dtype, m, ff, k, how):
    from cubic_serve_b200.ops import kernels as K, wq_pack
    if dtype == torch.float32 and how:
        pytest.skip("the fp32 product has one form")
    g = torch.Generator().manual_seed(m + ff)
    x = (torch.randn(m, k, generator=g) * 1.5).to(dtype)
    gate, up = (torch.randn(ff, k, generator=g) / k ** 0.5 for _ in range(2))
    w = wq_pack.pack_bf16(torch.cat([gate, up]))
    want = R.gelu_tanh(x.double() @ w.codes[:ff].double().t()) * (x.double() @ w.codes[ff:].double().t())
    out = torch.full((m, ff + 16), 7.0, dtype=dtype, device=DEV)
    K.wide_gemm(x.to(DEV), wq_pack.swiglu_interleave(w).to(DEV), out[:, 8:8 + ff], glu="gelu", **how)
    close(out[:, 8:8 + ff], want, dtype, exact=1e-5, rough=1e-2)
    assert (out[:, :8] == 7).all() and (out[:, 8 + ff:] == 7).all()
    K.workspace(torch.device(DEV)).check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_gelu_extremes(dtype):
    """Gates far from zero in both directions stay finite and take their limits."""
    from cubic_serve_b200.ops import kernels as K, wq_pack
    x = torch.zeros(4, 64, dtype=dtype)
    x[0, 0], x[1, 0], x[2, 0], x[3, 0] = 1e4, -1e4, 3.0, -3.0
    w = torch.zeros(32, 64)
    w[:16, 0], w[16:, 0] = 1.0, 0.5
    out = torch.zeros(4, 16, dtype=dtype, device=DEV)
    K.wide_gemm(x.to(DEV), wq_pack.swiglu_interleave(wq_pack.pack_bf16(w)).to(DEV), out, glu="gelu")
    v = x[:, 0].double()
    got, want = out.double().cpu(), (R.gelu_tanh(v) * 0.5 * v).unsqueeze(1).expand(4, 16)
    assert torch.isfinite(got).all() and ((got - want).abs() <= (1e-5 if dtype == torch.float32 else 1e-2) * (want.abs() + 0.1)).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 68, 67, 2048, 8704])
def test_embedding_and_normed_addition(dtype, W):
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(W)
    table, w = torch.randn(11, W, generator=g).to(torch.bfloat16), 1 + 0.2 * torch.randn(W, generator=g)
    ids = torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32)
    ld = -(-W // 64) * 64
    x, h = torch.zeros(5, W, device=DEV), torch.full((5, ld), 9.0, dtype=dtype, device=DEV)
    K.embed_rows(ids.to(DEV), table.to(DEV), w.to(DEV), x, h, 1e-3)
    e = table.double()[ids.long()]
    assert torch.equal(x.double().cpu(), e) and (h[:, W:] == 9).all()
    close(h[:, :W], R.rms(e, 1e-3) * w.double(), dtype, exact=1e-6, rough=6e-3)
    # tiny rows: eps decides the norm
    y = torch.randn(5, -(-W // 8) * 8, generator=g).to(dtype)
    y[2] *= 1e-3
    nw = torch.randn(W, generator=g)
    want = e + R.rms(y.double()[:, :W], 1e-3) * nw.double()
    K.add_norm_rows(y.to(DEV)[:, :W], nw.to(DEV), x, 1e-3, w.to(DEV), h)
    close(x, want, torch.float32, exact=1e-6)
    close(h[:, :W], R.rms(want, 1e-3) * w.double(), dtype, exact=1e-6, rough=6e-3)
    before = h.clone()
    K.add_norm_rows(y.to(DEV)[:, :W], nw.to(DEV), x, 1e-3)
    close(x, want + R.rms(y.double()[:, :W], 1e-3) * nw.double(), torch.float32, exact=1e-6)
    assert torch.equal(h, before)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, W, dim", [(1, 64, 16), (5, 68, 5), (17, 67, 8), (300, 256, 40), (1, 2048, 64), (33, 4096, 24), (130, 1024, 130),
                                       (3000, 96, 12), (16, 8192, 72)])
def test_side_gate(dtype, T, W, dim):
    """Widths that are no multiple of a fragment, more outputs than a block has, clusters that share the columns."""
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T + W)
    x, w = torch.randn(T, W, generator=g), (torch.randn(dim, W, generator=g) / W ** 0.5).to(torch.bfloat16)
    table, ids = torch.randn(19, 3 * dim + 2, generator=g).to(torch.bfloat16), torch.randint(0, 19, (T,), generator=g).to(torch.int32)
    padded = torch.zeros(dim, -(-W // 64) * 64, dtype=torch.bfloat16)
    padded[:, :W] = w
    ld = -(-dim // 64) * 64
    out = torch.full((T, ld), 9.0, dtype=dtype, device=DEV)
    K.side_gate(x.to(DEV), padded.to(DEV), ids.to(DEV), table.to(DEV), dim + 1, out)
    want = R.gelu_tanh(x.double() @ w.double().t()) * table.double()[ids.long(), dim + 1:2 * dim + 1]
    close(out[:, :dim], want, dtype, exact=1e-5, rough=1e-2)
    assert (out[:, dim:] == 9).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, W, dim", [(1, 64, 16), (5, 72, 5), (17, 68, 8), (300, 520, 40), (1, 2048, 64), (33, 4096, 24), (40, 1024, 130),
                                       (600, 96, 12), (16, 8192, 33), (19, 6144, 64), (4, 8704, 16)])
def test_side_input(dtype, T, W, dim):
    """The whole step, in one kernel (clusters of one to eight blocks) where the sizes allow it: residual, next norm, and neither
    of them touched where there is no next norm."""
    from cubic_serve_b200.ops import kernels as K, wq_pack
    g = torch.Generator().manual_seed(T + W)
    x, w = torch.randn(T, W, generator=g), (torch.randn(dim, W, generator=g) / W ** 0.5).to(torch.bfloat16)
    table, ids = torch.randn(19, 3 * dim + 2, generator=g).to(torch.bfloat16), torch.randint(0, 19, (T,), generator=g).to(torch.int32)
    gate = torch.zeros(dim, -(-W // 64) * 64, dtype=torch.bfloat16)
    gate[:, :W] = w
    kp = -(-dim // 64) * 64
    proj = torch.zeros(W, kp, dtype=torch.bfloat16)
    proj[:, :dim] = (torch.randn(W, dim, generator=g) / dim ** 0.5).to(torch.bfloat16)
    nw, nx = torch.randn(W, generator=g), 1 + 0.2 * torch.randn(W, generator=g)
    e = table.double()[ids.long(), dim + 1:2 * dim + 1]
    y = (R.gelu_tanh(x.double() @ w.double().t()) * e) @ proj[:, :dim].double().t()
    want = x.double() + R.rms(y, 1e-3) * nw.double()
    packed = wq_pack.pack_bf16(proj).to(DEV)
    for follow in (True, False):
        xd = x.to(DEV)
        h = torch.full((T, -(-W // 64) * 64), 9.0, dtype=dtype, device=DEV)
        gs, ys = torch.zeros(T, kp, dtype=dtype, device=DEV), torch.zeros(T, -(-W // 8) * 8, dtype=dtype, device=DEV)
        n = K.side_input(xd, gate.to(DEV), ids.to(DEV), table.to(DEV), dim + 1, packed, nw.to(DEV), 1e-3, nx.to(DEV) if follow else None,
                         h if follow else None, gs, ys[:, :W])
        assert n == (1 if dtype == torch.bfloat16 and dim <= 64 and W % 8 == 0 and W <= 8192 else 3)
        close(xd, want, torch.float32, exact=2e-5 if dtype == torch.float32 else 1e-2)
        if follow:
            close(h[:, :W], R.rms(want, 1e-3) * nx.double(), dtype, exact=2e-5, rough=1.5e-2)
            assert (h[:, W:] == 9).all()
        else:
            assert (h == 9).all()


# ------------------------------------------------------------------ sink attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, pairs", [(6, 2, 24, 6), (3, 1, 13, 3), (4, 4, 64, 32), (2, 1, 200, 20), (5, 5, 18, 0), (40, 1, 128, 64)])
def test_gqa_prepare(dtype, H, G, d, pairs):
    """Head norms, rotation of neighbouring pairs (positions up to a million), values before both, pages; padding rows write
    nothing."""
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(H)
    T, P, q_off = 6, -(-d // 64) * 64, 8
    k_off = q_off + -(-H * d // 8) * 8
    x = torch.randn(T, k_off + -(-G * d // 8) * 8, generator=g).to(dtype)
    qn, kn = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    freq = (100.0 ** (-torch.arange(pairs) / max(pairs, 1))).float()
    pos = torch.tensor([0, 1, 15, 1000, 999999, 77], dtype=torch.int32)
    slots = torch.tensor([17, 63, -1, 0, 32, 31], dtype=torch.int32)
    q = torch.full((T, H * P), 9.0, dtype=dtype, device=DEV)
    cache = torch.zeros(4, G, 2, 16, P, dtype=dtype, device=DEV)
    K.gqa_prepare(x.to(DEV), q_off, k_off, qn.to(DEV), kn.to(DEV), freq.to(DEV), 1.25, pos.to(DEV), slots.to(DEV), q, cache, H, d, 1e-4)
    xd = x.double()
    qh, kh = xd[:, q_off:q_off + H * d].view(T, H, d), xd[:, k_off:k_off + G * d].view(T, G, d)

    def turned(v, w):
        n = R.rms(v, 1e-4) * w.double()
        return torch.stack([R.rotate_pairs(n[t:t + 1], int(pos[t]), freq.double(), 1.25)[0] for t in range(T)])

    got = q.view(T, H, P)
    close(got[:, :, :d], turned(qh, qn), dtype, exact=4e-6, rough=8e-3)
    assert (got[:, :, d:] == 0).all()
    keys, vals = torch.zeros(64, G, P, dtype=torch.float64), torch.zeros(64, G, P, dtype=torch.float64)
    kt = turned(kh, kn)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            keys[s, :, :d], vals[s, :, :d] = kt[t], kh[t]
    rows = cache.permute(2, 0, 3, 1, 4).reshape(2, 64, G, P)
    close(rows[0], keys, dtype, exact=4e-6, rough=8e-3)
    assert torch.equal(rows[1].double().cpu(), vals)


class GqaCase:
    """Keys and values of several requests on shuffled pages of one cache, and queries."""

    def __init__(self, lens, H, G, d, dtype, seed=0, spare=3, gain=1.0):
        g = torch.Generator().manual_seed(seed)
        self.H, self.G, self.d, self.P, self.dtype, self.lens = H, G, d, -(-d // 64) * 64, dtype, lens
        self.k = [(gain * torch.randn(n, G, d, generator=g)).to(dtype) for n in lens]
        self.v = [torch.randn(n, G, d, generator=g).to(dtype) for n in lens]
        self.q = [torch.randn(n, H, d, generator=g).to(dtype) for n in lens]
        per = [-(-n // 16) for n in lens]
        ids = (torch.randperm(sum(per) + spare, generator=g) + 1).tolist()
        self.table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        for r, n in enumerate(per):
            self.table[r, :n] = torch.tensor([ids.pop() for _ in range(n)])
        self.pages = sum(per) + spare + 1
        self.fill()

    def fill(self):
        # pages nobody owns and the unwritten rest of last pages hold garbage that must not be used
        self.cache = torch.full((self.pages, self.G, 2, 16, self.P), 1e4, dtype=self.dtype)
        for r, n in enumerate(self.lens):
            for p in range(-(-n // 16)):
                page, m = self.cache[self.table[r, p]], min(16, n - 16 * p)
                for which, t in ((0, self.k[r]), (1, self.v[r])):
                    page[:, which, :m] = 0
                    page[:, which, :m, :self.d] = t[16 * p:16 * p + m].transpose(0, 1)

    def run(self, spans, window, scale, sink=0.0, out_scale=1.0, splits=None, decode=None):
        from cubic_serve_b200.ops import kernels as K
        T = sum(n for _, _, n in spans)
        q = torch.zeros(T, self.H, self.P, dtype=self.dtype)
        q[:, :, :self.d] = torch.cat([self.q[r][first:first + n] for r, first, n in spans])
        ld = -(-self.H * self.d // 8) * 8 + 16
        wide = torch.full((T, ld), 3.0, dtype=self.dtype, device=DEV)
        out = wide[:, 8:8 + self.H * self.d]
        seg = segs([(n, r, first) for r, first, n in spans])
        K.gqa_attention(q.view(T, -1).to(DEV), self.cache.to(DEV), self.table.to(DEV), seg, out, self.H, self.d, window, scale, sink,
                        out_scale, decode=T == len(spans) if decode is None else decode, splits=splits)
        assert (wide[:, :8] == 3).all() and (wide[:, 8 + self.H * self.d:] == 3).all()
        return out.reshape(T, self.H, self.d).split([n for _, _, n in spans])

    def want(self, r, first, n, window, scale, sink=0.0, out_scale=1.0):
        k, v, q = self.k[r][:first + n].double(), self.v[r][:first + n].double(), self.q[r][first:first + n].double()
        if sink is None:
            rep = torch.arange(self.H) // (self.H // self.G)
            return out_scale * R.windowed_attention(q, k[:, rep], v[:, rep], first, window or None, scale)
        return out_scale * R.sink_attention(q, k, v, first, window or None, scale)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, window", [(6, 2, 64, 37), (3, 1, 13, 0), (32, 8, 128, 130), (40, 1, 72, 16), (4, 4, 200, 100), (1, 1, 24, 1),
                                             (70, 1, 128, 50), (150, 1, 40, 33), (10, 5, 256, 17), (9, 3, 160, 0)])
def test_gqa_attention_prefill_portions_and_decode(dtype, H, G, d, window):
    lens = (150, 3, 61, 16)
    case = GqaCase(lens, H, G, d, dtype, seed=H)
    scale = 1.5 / d ** 0.5
    whole = case.run([(r, 0, n) for r, n in enumerate(lens)], window, scale)
    for r, n in enumerate(lens):
        close(whole[r], case.want(r, 0, n, window, scale), dtype, rough=1e-2)
    # portions beside single tokens, in another order, scaled
    spans = [(2, 40, 21), (0, 149, 1), (1, 1, 2), (3, 15, 1)]
    for (r, first, n), o in zip(spans, case.run(spans, window, scale, out_scale=0.6)):
        close(o, case.want(r, first, n, window, scale, out_scale=0.6), dtype, rough=1e-2)
    # decode, with and without key splits (a split may see no key at all)
    spans = [(r, n - 1, 1) for r, n in enumerate(lens)]
    for splits in (None, 1, 2, 7):
        for (r, first, n), o in zip(spans, case.run(spans, window, scale, splits=splits, out_scale=1.7)):
            close(o, case.want(r, first, n, window, scale, out_scale=1.7), dtype, rough=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shift", [-30.0, -3.0, 0.0, 30.0])
def test_sink_takes_its_share(dtype, shift):
    """Scores far below the sink leave almost nothing, scores far above it almost everything; without a sink the weights sum to
    one."""
    case = GqaCase((90, 40), 4, 2, 32, dtype, seed=5, gain=0.2)
    for r in range(2):                                     # a channel that all scores share
        case.q[r][:, :, 0], case.k[r][:, :, 0] = 1.0, shift
    case.fill()
    for sink in (0.0, None):
        outs = [(0, 0, o) for o in [case.run([(0, 0, 90), (1, 0, 40)], 25, 1.0, sink=sink)[0]]]
        outs += [(0, 89, o) for splits in (1, 4) for o in [case.run([(0, 89, 1), (1, 39, 1)], 25, 1.0, sink=sink, splits=splits)[0]]]
        for r, first, o in outs:
            want = case.want(r, first, o.shape[0], 25, 1.0, sink=sink)
            assert torch.isfinite(o.float()).all()
            err = (o.double().cpu() - want).abs().max() / want.abs().max()
            assert err <= (2e-5 if dtype == torch.float32 else 1.5e-2), (sink, first, float(err))
    plain = case.want(0, 0, 90, 25, 1.0, sink=None)
    kept = case.want(0, 0, 90, 25, 1.0)
    if shift == -30.0:
        assert kept.abs().max() < 1e-9 * plain.abs().max()
    if shift == 0.0:
        assert (kept[0] - plain[0]).abs().max() > 0.3 * plain[0].abs().max()          # a single visible key shares with the sink


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 31, 33, 63, 64, 65, 129])
def test_window_edge_shows_one_key(dtype, window):
    """One key carries a score that outweighs all others and a value nothing else has: it is seen by exactly the queries whose
    window holds it, in a prompt and decoded, wherever the edge falls on a page or a key tile."""
    n, H, G, d = 200, 6, 2, 40
    for j in (0, 15, 16, 47, 64):
        case = GqaCase((n,), H, G, d, dtype, seed=window, gain=0.1)
        case.q[0] *= 0.1
        case.q[0][:, :, 0] = 6.0
        case.k[0][:, :, 0], case.v[0][:, :, 1] = 0.0, 0.0
        case.k[0][j, :, 0], case.v[0][j, :, 1] = 6.0, 40.0
        case.fill()
        out = case.run([(0, 0, n)], window, 1.0)[0][:, :, 1].float().cpu()
        seen = torch.tensor([0 <= i - j < window for i in range(n)])
        assert ((out > 10).all(1) == seen).all() and ((out.abs() < 1).all(1) == ~seen).all(), (window, j)
        for i in (j + window - 1, j + window):                # just inside and just outside, decoded
            if j <= i < n:
                for splits in (None, 4):
                    one = case.run([(0, i, 1)], window, 1.0, splits=splits)[0][0, :, 1].float().cpu()
                    assert ((one > 10).all() if seen[i] else (one.abs() < 1).all()), (window, j, i)


# ------------------------------------------------------------------ recurrences
ROWWISE = ("x", "a", "dt", "z")


class GatedLinear:
    """Gated linear attention from the projections on."""
    eps = 1e-5

    def __init__(self, H, d, e, tau=8.0):
        self.H, self.d, self.e, self.tau = H, d, e, tau
        self.offs = (8, 16 + -(-H * d // 8) * 8, 24 + 2 * -(-H * d // 8) * 8)
        self.cols = self.offs[2] + -(-H * e // 8) * 8

    def case(self, T, seed=0):
        g = torch.Generator().manual_seed(seed)
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)                # noqa: E731
        return {"x": bf(T, self.cols), "a": bf(T, self.H * self.d), "z": bf(T, self.H * self.e),
                "bias": torch.randn(self.H * self.d, generator=g), "norm": 1 + 0.2 * torch.randn(self.e, generator=g)}

    def oracle(self, c, state=None):
        H, d, e = self.H, self.d, self.e
        f = {k: v.double() for k, v in c.items()}
        T = f["x"].shape[0]
        q, k, v = (f["x"][:, o:o + H * w].view(T, H, w) for o, w in zip(self.offs, (d, d, e)))
        alpha = (1 / (1 + torch.exp(-(f["a"] + f["bias"])))) ** (1 / self.tau)
        S = torch.zeros(H, d, e, dtype=torch.float64) if state is None else state
        o = torch.empty(T, H, e, dtype=torch.float64)
        for t in range(T):
            o[t], S = R.linear_step(S, q[t] * d ** -0.5, k[t], v[t], alpha.view(T, H, d)[t])
        return R.rms(o, self.eps) * f["norm"] * R.silu(f["z"]).view(T, H, e), S

    def states(self, dtype, slots):                            # stale contents: a fresh request must not read them
        return (torch.full((slots, self.H, self.e, -(-self.d // 4) * 4), 5.0, device=DEV),)

    def run(self, c, dtype, seg, states, decode):
        from cubic_serve_b200.ops import kernels as K
        T = c["x"].shape[0]
        dev = {k: c[k].to(DEV, dtype if k in ROWWISE else torch.float32).contiguous() for k in c}
        sc = K.RecurrenceScratch(T, [(self.H, self.H, self.d, self.e, True)], dtype, DEV)
        out = torch.full((T, self.H * self.e + 8), 3.0, dtype=dtype, device=DEV)[:, :self.H * self.e]
        K.gated_linear_prepare(dev["x"], *self.offs, dev["a"], dev["bias"], 1 / self.tau, seg, sc, self.H, self.d, self.e)
        K.gated_linear_walk(dev["z"], dev["norm"], states[0], seg, out, sc, self.d, self.eps, decode)
        return out.clone().reshape(T, self.H, self.e)

    def check_state(self, states, slot, want, dtype):
        close(states[0][slot, :, :, :self.d].transpose(1, 2), want, torch.float32, exact=2e-5 if dtype == torch.float32 else 1e-2)


class Ssd:
    """A state-space layer from the projections on."""
    eps = 1e-5

    def __init__(self, H, P, N, G, taps, parts):
        self.H, self.P, self.N, self.G, self.taps, self.parts = H, P, N, G, taps, parts
        self.C = H * P + 2 * G * N

    def case(self, T, seed=0):
        g = torch.Generator().manual_seed(seed)
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)                # noqa: E731
        n = lambda *s: torch.randn(*s, generator=g)                                    # noqa: E731
        return {"x": bf(T, self.C), "dt": bf(T, self.H), "z": bf(T, self.H * self.P), "conv": n(self.C, self.taps) / self.taps ** 0.5,
                "conv_b": 0.3 * n(self.C), "a_log": 0.5 * n(self.H) - 1.0, "dt_bias": 0.5 * n(self.H), "D": n(self.H),
                "norm": 1 + 0.2 * n(self.H * self.P)}

    def oracle(self, c, state=None):
        H, P, N, G = self.H, self.P, self.N, self.G
        f = {k: v.double() for k, v in c.items()}
        T = f["x"].shape[0]
        past, S = state if state is not None else (torch.zeros(self.taps - 1, self.C, dtype=torch.float64),
                                                   torch.zeros(H, N, P, dtype=torch.float64))
        y, past = R.short_conv(f["x"], f["conv"], past, f["conv_b"])
        rep = torch.arange(H) // (H // G)
        x, B, C = y.split([H * P, G * N, G * N], 1)
        x, B, C = x.view(T, H, P), B.view(T, G, N)[:, rep], C.view(T, G, N)[:, rep]
        dt = R.softplus(f["dt"] + f["dt_bias"])
        decay = torch.exp(-torch.exp(f["a_log"]) * dt).unsqueeze(-1).expand(T, H, N)
        o = torch.empty(T, H, P, dtype=torch.float64)
        for t in range(T):
            o[t], S = R.linear_step(S, C[t], B[t], dt[t].unsqueeze(-1) * x[t], decay[t])
        o = (o + f["D"].unsqueeze(-1) * x).reshape(T, H * P)
        return R.gated_parts_norm(o, f["z"], f["norm"], self.parts, self.eps).view(T, H, P), (past, S)

    def states(self, dtype, slots):
        return (torch.full((slots, self.H, self.P, -(-self.N // 4) * 4), 5.0, device=DEV),
                torch.full((slots, max(1, self.taps - 1), -(-self.C // 8) * 8), 5.0, dtype=dtype, device=DEV))

    def run(self, c, dtype, seg, states, decode):
        from cubic_serve_b200.ops import kernels as K
        T, pad = c["x"].shape[0], -(-self.C // 8) * 8
        x, w, b = torch.zeros(T, pad, dtype=dtype), torch.zeros(self.taps, pad), torch.zeros(pad)
        x[:, :self.C], w[:, :self.C], b[:self.C] = c["x"], c["conv"].t(), c["conv_b"]
        dev = {k: c[k].to(DEV, dtype if k in ROWWISE else torch.float32).contiguous() for k in c}
        sc = K.RecurrenceScratch(T, [(self.H, self.G, self.N, self.P, False)], dtype, DEV)
        out = torch.full((T, self.H * self.P + 8), 3.0, dtype=dtype, device=DEV)[:, :self.H * self.P]
        K.ssd_prepare(x.to(DEV), dev["dt"], w.to(DEV), b.to(DEV), states[1], dev["a_log"], dev["dt_bias"], seg, sc, self.H, self.G,
                      self.N, self.P)
        K.ssd_walk(dev["z"], dev["D"], dev["norm"], self.parts, states[0], seg, out, sc, self.G, self.N, self.eps, decode)
        return out.clone().reshape(T, self.H, self.P)

    def check_state(self, states, slot, want, dtype):
        past, S = want
        close(states[0][slot, :, :, :self.N].transpose(1, 2), S, torch.float32, exact=2e-5 if dtype == torch.float32 else 2e-2)
        if self.taps > 1:
            close(states[1][slot, :, :self.C], past, torch.float32, exact=0)


LAYERS = [GatedLinear(2, 64, 64), GatedLinear(3, 20, 28), GatedLinear(2, 128, 128, 16.0), GatedLinear(2, 7, 9, 3.0), GatedLinear(1, 16, 16, 1.0),
          GatedLinear(1, 160, 72), GatedLinear(2, 96, 200), GatedLinear(6, 256, 24),
          Ssd(4, 64, 64, 2, 4, 2), Ssd(2, 128, 128, 2, 4, 1), Ssd(6, 5, 7, 3, 6, 5), Ssd(1, 16, 16, 1, 1, 1), Ssd(4, 130, 136, 1, 2, 4),
          Ssd(8, 24, 20, 1, 3, 3), Ssd(3, 40, 256, 1, 4, 1), Ssd(16, 100, 32, 4, 4, 1)]
NAMES = ["-".join([type(l).__name__] + [str(v) for v in vars(l).values() if isinstance(v, (int, float))]) for l in LAYERS]


def rows_of(c, lo, hi):
    return {k: (v[lo:hi] if k in ROWWISE else v) for k, v in c.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", LAYERS, ids=NAMES)
def test_recurrence_in_portions(dtype, layer):
    """Portions of several sizes (down to two tokens, one at the end) on a slot with stale contents, against token by token."""
    T = 75
    c = layer.case(T)
    want, state = layer.oracle(c)
    states = layer.states(dtype, 3)
    got, i = [], 0
    for n in (2, 37, 16, 17, 2, 1):
        got.append(layer.run(rows_of(c, i, i + n), dtype, segs([(n, 1, i)]), states, n == 1))
        i += n
    close(torch.cat(got), want, dtype, exact=5e-5)
    layer.check_state(states, 1, state, dtype)
    for s in states:
        assert (s[0] == 5).all() and (s[2] == 5).all()         # other slots are untouched
    # token by token from the start on the same slot
    one = [layer.run(rows_of(c, t, t + 1), dtype, segs([(1, 1, t)]), states, True) for t in range(20)]
    close(torch.cat(one), want[:20], dtype, exact=5e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [l for l in LAYERS if l.H in (3, 4, 6)], ids=[n for l, n in zip(LAYERS, NAMES) if l.H in (3, 4, 6)])
def test_recurrence_batches(dtype, layer):
    """Unequal requests in one step equal each alone; decode steps with a padding segment; a slot used again."""
    lens, slots = (33, 1, 2, 50, 16), (4, 0, 3, 1, 2)
    cs = [layer.case(n + 1, seed=n) for n in lens]
    shared = {k: v for k, v in cs[0].items() if k not in ROWWISE}
    cs = [{**c, **shared} for c in cs]
    oracle = [layer.oracle(rows_of(c, 0, n)) for c, n in zip(cs, lens)]
    states = layer.states(dtype, 5)
    keys = [k for k in ROWWISE if k in cs[0]]
    batch = {k: torch.cat([c[k][:n] for c, n in zip(cs, lens)]) for k in keys} | shared
    out = layer.run(batch, dtype, segs([(n, s, 0) for n, s in zip(lens, slots)]), states, False)
    for o, (want, _) in zip(out.split(lens), oracle):
        close(o, want, dtype, exact=5e-5)
    order = [0, 1, None, 2, 3, 4]
    rows = {k: torch.cat([cs[i][k][lens[i]:] if i is not None else torch.zeros_like(cs[0][k][:1]) for i in order]) for k in keys} | shared
    bucket = segs([(1, slots[i], lens[i]) if i is not None else (0, 0, 0) for i in order])
    bucket.row0 = torch.arange(len(order), dtype=torch.int32, device=DEV)              # row j belongs to segment j
    out = layer.run(rows, dtype, bucket, states, True)
    for j, i in enumerate(order):
        if i is None:
            continue
        want, state = layer.oracle(rows_of(cs[i], lens[i], lens[i] + 1), oracle[i][1])
        close(out[j:j + 1], want, dtype, exact=5e-5)
        layer.check_state(states, slots[i], state, dtype)


@pytest.mark.parametrize("layer, rank", [(GatedLinear(3, 20, 28), 12), (GatedLinear(2, 128, 64, 16.0), 64), (GatedLinear(2, 7, 9, 3.0), 33),
                                         (GatedLinear(1, 160, 16), 100)], ids=["20", "128", "7", "160"])
def test_low_rank_decays(layer, rank):
    """Decay logits made by the preparation from their inner columns equal the product done before it, in prompts and decoding."""
    from cubic_serve_b200.ops import kernels as K, wq_pack
    H, d, T, kp = layer.H, layer.d, 37, -(-rank // 64) * 64
    c = layer.case(T, 3)
    g = torch.Generator().manual_seed(rank)
    inner, w = torch.randn(T, rank, generator=g).to(torch.bfloat16), (2 * torch.randn(H * d, rank, generator=g) / rank ** 0.5).to(torch.bfloat16)
    z = inner.double() @ w.double().t() + c["bias"].double()
    want = (1 / (1 + torch.exp(-z))) ** (1 / layer.tau)
    a, low = torch.zeros(T, kp + 8, dtype=torch.bfloat16), torch.zeros(H * d, kp, dtype=torch.bfloat16)
    a[:, :rank], low[:, :rank] = inner, w
    ds = -(-d // 4) * 4
    for spans in ([(T, 0, 0)], [(5, 0, 0), (1, 1, 3), (31, 2, 0)], [(1, t, 4) for t in range(T)]):
        sc = K.RecurrenceScratch(T, [(H, H, d, layer.e, True)], torch.bfloat16, DEV)
        K.gated_linear_prepare(c["x"].to(DEV), *layer.offs, a.to(DEV)[:, :kp], c["bias"].to(DEV), 1 / layer.tau, segs(spans), sc, H, d,
                               layer.e, wq_pack.pack_bf16(low).to(DEV), rank)
        got = sc.g[:T * H * ds].view(T, H, ds)
        assert (got[:, :, :d].double().cpu() - want.view(T, H, d)).abs().max() < 5e-6 and (got[:, :, d:] == 0).all()


def test_decay_of_every_channel_counts():
    """One key channel forgets, one keeps: a value written far back comes back through the right one only."""
    layer = GatedLinear(1, 8, 4, 1.0)
    c = layer.case(60)
    q, k, v = layer.offs
    c["x"].zero_()
    c["x"][0, k:k + 2], c["x"][0, v] = 1.0, 3.0                # written by the first token into channels 0 and 1
    c["a"].zero_()
    c["bias"].zero_()
    c["bias"][0], c["bias"][1] = 12.0, -3.0                    # channel 0 keeps, channel 1 forgets
    c["z"].fill_(4.0)
    for read, seen in ((0, True), (1, False)):
        c["x"][59].zero_()
        c["x"][59, q + read] = 2.0
        want, _ = layer.oracle(c)
        states = layer.states(torch.float32, 2)
        layer.run(rows_of(c, 0, 40), torch.float32, segs([(40, 1, 0)]), states, False)
        got = layer.run(rows_of(c, 40, 60), torch.float32, segs([(20, 1, 40)]), states, False)[-1]
        assert torch.allclose(got.double().cpu(), want[-1], atol=1e-5)
        assert (float(got[0, 0].abs()) > 1) == seen
