"""Mechanisms of the layered decoders with gated residuals on the GPU, each alone against the oracle's equations: products with gates and
clamped activations, latent attention with a rotated key part, differential attention in chunks, element-wise recurrences."""
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
from test_gpu_layered import DEV, DTYPES, LatentCase, close, segs  # noqa: E402
from test_gpu_sequential import GqaCase  # noqa: E402

from cubic_serve_b200.models import layered_reference as R  # noqa: E402

pytestmark = pytest.mark.gpu
FORMS = [(1, 64, {}), (17, 128, {}), (300, 192, {}), (33, 256, {"stream_k": True}), (520, 128, {"stream_k": True}), (40, 1024, {"splits": 2}),
         (9, 1024, {"splits": 5})]


def padded(m, n, dtype, left=8, right=8, fill=7.0):
    """A buffer and the columns of it that a kernel may write."""
    wide = torch.full((m, left + -(-n // 8) * 8 + right), fill, dtype=dtype, device=DEV)
    return wide, wide[:, left:left + n]


def untouched(wide, n, left=8, fill=7.0):
    return (wide[:, :left] == fill).all() and (wide[:, left + n:] == fill).all()


def split_freq(exact):
    return torch.stack([exact.float(), (exact - exact.float().double()).float()]).to(DEV).contiguous()


# ------------------------------------------------------------------ products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff, limit", [(64, 1.0), (44, 0.3), (160, 7.0)])
@pytest.mark.parametrize("m, k, how", FORMS)
def test_clamped_activation_beside_plain_rows(dtype, m, k, how, ff, limit):
    """One product: the first rows leave through the clamped activation, the others as they are."""
    from cubic_serve_b200.models.layered import _pack_glu
    from cubic_serve_b200.ops import kernels as K
    if dtype == torch.float32 and how:
        pytest.skip("the fp32 product has one form")
    g = torch.Generator().manual_seed(m + ff)
    gate, up, rest = (torch.randn(n, k, generator=g).mul(2 / k ** 0.5).to(torch.bfloat16) for n in (ff, ff, 72))
    x = torch.randn(m, k, generator=g).to(dtype)
    w, rows = _pack_glu(gate, up, rest)
    assert rows % 128 == 0 and w.n == rows + 72
    # W_down is the identity on the activation
    want = R.clamped_feed_forward({"p.gate": gate.double(), "p.up": up.double(), "p.down": torch.eye(ff, dtype=torch.float64)}, "p",
                                  x.double(), limit)
    act, other = padded(m, rows // 2, dtype), padded(m, 72, dtype)
    K.wide_gemm(x.to(DEV), w.to(DEV), act[1], glu="clamped", limit=limit, rest=other[1], split=rows, **how)
    close(act[1][:, :ff], want, dtype, exact=1e-5, rough=1.5e-2)
    assert (act[1][:, ff:] == 0).all() and untouched(act[0], rows // 2) and untouched(other[0], 72)
    close(other[1], x.double() @ rest.double().t(), dtype, exact=1e-5, rough=6e-3)
    K.workspace(torch.device(DEV)).check_status()


def test_clamps_act_on_their_own_sides():
    """A gate far below the limit passes, one above is held; the other factor is held on both sides and moved by one."""
    from cubic_serve_b200.models.layered import _pack_glu
    from cubic_serve_b200.ops import kernels as K
    x = torch.eye(64)
    gate, up = torch.zeros(16, 64), torch.zeros(16, 64)
    for c, (gv, uv) in enumerate([(9.0, 9.0), (9.0, -9.0), (-3.0, 9.0), (-3.0, -9.0), (0.5, 0.25), (1.0, -1.0), (-60.0, 0.0)]):
        gate[:, c], up[:, c] = gv, uv
    w, rows = _pack_glu(gate.to(torch.bfloat16), up.to(torch.bfloat16))
    want = R.clamped_feed_forward({"p.gate": gate.double(), "p.up": up.double(), "p.down": torch.eye(16, dtype=torch.float64)}, "p",
                                  x.double(), 1.25)
    for dtype in DTYPES:
        out = torch.zeros(64, 16, dtype=dtype, device=DEV)
        K.wide_gemm(x.to(DEV, dtype), w.to(DEV), out, glu="clamped", limit=1.25)
        close(out, want, dtype, exact=1e-6, rough=5e-3)
        assert (out[7:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [40, 131, 260])
@pytest.mark.parametrize("m, k, how", FORMS)
def test_gated_addition_to_the_residual(dtype, m, k, how, n):
    from cubic_serve_b200.ops import kernels as K, wq_pack
    if dtype == torch.float32 and how:
        pytest.skip("the fp32 product has one form")
    g = torch.Generator().manual_seed(m + n)
    x, w = torch.randn(m, k, generator=g).to(dtype), wq_pack.pack_bf16(torch.randn(n, k, generator=g) / k ** 0.5)
    z, b, res = (2 * torch.randn(m, n, generator=g)).to(dtype), torch.randn(n, generator=g), torch.randn(m, n, generator=g)
    z[0, 0], z[0, 1] = -200.0, 200.0                      # shut, and open
    wide, logits = padded(m, n, dtype)
    logits.copy_(z)
    y = res.to(DEV)
    K.wide_gemm(x.to(DEV), w.to(DEV), y, residual=y, gate=(logits, b.to(DEV)), **how)
    close(y, res + R.sigmoid(z.double() + b.double()) * (x.double() @ w.codes.double().t()), torch.float32, exact=1e-5)
    K.workspace(torch.device(DEV)).check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 68, 67, 2048, 8704])
def test_scaled_embedding_and_its_second_addition(dtype, W):
    from cubic_serve_b200.ops import kernels as K
    table, ids = torch.randn(11, W).to(torch.bfloat16), torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    w = 1 + 0.2 * torch.randn(W)
    x, h = torch.full((4, W), 5.0, device=DEV), torch.full((4, -(-W // 64) * 64), 9.0, dtype=dtype, device=DEV)
    e = 0.3 * table.double()[ids.long()]
    K.embed_rows(ids.to(DEV), table.to(DEV), w.to(DEV), x, h, 1e-3, 0.3)
    close(x, e, torch.float32, exact=1e-6)
    close(h[:, :W], R.rms(e, 1e-3) * w.double(), dtype, exact=1e-6, rough=6e-3)
    x.mul_(-2.5)
    K.embed_rows(ids.to(DEV), table.to(DEV), w.to(DEV), x, h, 1e-3, 0.3, add=True)
    close(x, -1.5 * e, torch.float32, exact=1e-6)
    close(h[:, :W], R.rms(-1.5 * e, 1e-3) * w.double(), dtype, exact=1e-6, rough=6e-3)
    assert (h[:, W:] == 9).all()


# ------------------------------------------------------------------ latent attention with a rotated part
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, rank, rot, yarn, T", [(6, 72, 12, (3.0, 40, 4.0, 0.5), 5), (1, 17, 2, None, 3), (40, 512, 64, (8.0, 4096, 32.0, 1.0), 7), (3, 100, 256, None, 2),
                                                   (32, 512, 64, None, 520)])
def test_rotated_rows(dtype, H, rank, rot, yarn, T):
    """Latents normed, key and query parts turned, near and far along a sequence; padding rows leave the cache alone."""
    from cubic_serve_b200.models.layered import LatentSpec, _read_rotary
    from cubic_serve_b200.ops import kernels as K
    conf = {"dims": rot, "base": 700.0}
    if yarn:
        conf["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    spec = LatentSpec(H, 8, 8, 0, rank, 1.0, 0, rot, _read_rotary(conf), False)
    spec.validate()
    g = torch.Generator().manual_seed(H + T)
    r8 = lambda n: -(-n // 8) * 8                                                      # noqa: E731
    c_off = 16 + r8(H * rot)
    r_off = c_off + r8(rank)
    proj = torch.randn(T, r_off + r8(rot) + 8, generator=g).to(dtype)
    cn = 1 + 0.2 * torch.randn(rank, generator=g)
    pos = torch.randint(0, 9, (T,), generator=g, dtype=torch.int32)
    pos[0], pos[1] = 0, 990000
    slots = torch.randperm(16 * (T // 8 + 2), generator=g)[:T].to(torch.int32)
    slots[T // 2] = -1
    ql = torch.zeros(T, H * spec.row_padded, dtype=dtype, device=DEV)
    cache = torch.zeros(T // 8 + 2, 16, spec.row_padded, dtype=dtype, device=DEV)
    K.latent_prepare(proj.to(DEV), c_off, rank, cn.to(DEV), cache, slots.to(DEV), 1e-4,
                     rotated=(16, r_off, spec.rot_col, spec.rotary.split_table().to(DEV), spec.rotary.factor, pos.to(DEV), ql, H))
    freq, mult = R.rotary_frequencies(conf)
    p = proj.double()
    want_q, rows = torch.zeros(T, H, spec.row_padded, dtype=torch.float64), torch.zeros(cache.shape[0] * 16, spec.row_padded, dtype=torch.float64)
    for t in range(T):
        at = slice(spec.rot_col, spec.rot_col + rot)
        want_q[t, :, at] = R.rotate_pairs(p[t, 16:16 + H * rot].view(1, H, rot), int(pos[t]), freq, mult)[0]
        if slots[t] >= 0:
            rows[slots[t], :rank] = R.rms(p[t, c_off:c_off + rank], 1e-4) * cn.double()
            rows[slots[t], at] = R.rotate_pairs(p[t, r_off:r_off + rot].view(1, 1, rot), int(pos[t]), freq, mult)[0, 0]
    close(ql.view(T, H, -1), want_q, dtype, exact=3e-6, rough=6e-3)
    close(cache.view(-1, spec.row_padded), rows, dtype, exact=3e-6, rough=6e-3)


class RotatedCase(LatentCase):
    """Latents with a rotated part behind them; no gate."""

    def __init__(self, lens, H, rank, rot, dtype, seed=0):
        from cubic_serve_b200.models.layered import LatentSpec, RotarySpec
        super().__init__(lens, H, rank, dtype, seed)
        spec = LatentSpec(H, 8, 8, 0, rank, 1.0, 0, rot, RotarySpec(rot, 10.0), False)
        self.rp, self.rv, self.col, self.rot = spec.row_padded, spec.rank_padded, spec.rot_col, rot
        g = torch.Generator().manual_seed(seed + 1)
        self.kr = [torch.randn(n, rot, generator=g).to(dtype) for n in lens]
        self.qr = [torch.randn(n, H, rot, generator=g).to(dtype) for n in lens]
        self.fill()

    def row(self, latent, turned):
        out = torch.zeros(*latent.shape[:-1], self.rp, dtype=self.dtype)
        out[..., :self.rank], out[..., self.col:self.col + self.rot] = latent, turned
        return out

    def fill(self):
        self.cache = torch.full((self.cache.shape[0], 16, self.rp), 1e4, dtype=self.dtype)
        for r, n in enumerate(self.lens):
            per = -(-n // 16)
            flat = torch.full((per * 16, self.rp), 1e4, dtype=self.dtype)
            flat[:n] = self.row(self.c[r], self.kr[r])
            self.cache[self.table[r, :per].long()] = flat.view(per, 16, self.rp)

    def run(self, spans, scale, splits=None, decode=None):
        from cubic_serve_b200.ops import kernels as K
        q = torch.cat([self.row(self.q[r][a:a + n], self.qr[r][a:a + n]) for r, a, n in spans])
        T = q.shape[0]
        out = torch.full((T, self.H * self.rv), 3.0, dtype=self.dtype, device=DEV)
        K.latent_attention(q.view(T, -1).to(DEV), None, self.cache.to(DEV), self.table.to(DEV), segs([(n, r, a) for r, a, n in spans]), out,
                           self.H, 0, scale, decode=T == len(spans) if decode is None else decode, splits=splits)
        return out.view(T, self.H, self.rv)[:, :, :self.rank].split([n for _, _, n in spans])

    def want(self, r, first, n, scale):
        k = torch.cat([self.c[r], self.kr[r]], -1)[:first + n].double().unsqueeze(1)
        q = torch.cat([self.q[r], self.qr[r]], -1)[first:first + n].double()
        return R.masked_attention(q, k, self.c[r][:first + n].double().unsqueeze(1), R.same_chunk(first, n, first + n, None), scale)


ROTATED = [(6, 72, 12), (5, 120, 32), (32, 512, 64), (70, 128, 64), (16, 250, 40), (1, 44, 16), (3, 500, 100), (40, 256, 64), (7, 19, 6), (128, 512, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, rank, rot", ROTATED)
def test_rotated_latent_attention_prefill_portions_and_decode(dtype, H, rank, rot):
    lens = (150, 3, 61, 16)
    case = RotatedCase(lens, H, rank, rot, dtype, seed=H)
    scale = 1.5 / (rank + rot) ** 0.5
    spans = [(r, 0, n) for r, n in enumerate(lens)]
    for r, o in enumerate(case.run(spans, scale)):
        close(o, case.want(r, 0, lens[r], scale), dtype, rough=1e-2)
    spans = [(2, 40, 21), (0, 149, 1), (1, 1, 2), (3, 15, 1)]
    for (r, first, n), o in zip(spans, case.run(spans, scale)):
        close(o, case.want(r, first, n, scale), dtype, rough=1e-2)
    spans = [(r, n - 1, 1) for r, n in enumerate(lens)]
    for splits in (None, 1, 2, 7):
        for (r, first, n), o in zip(spans, case.run(spans, scale, splits=splits)):
            close(o, case.want(r, first, n, scale), dtype, rough=1e-2)
    for r, o in enumerate(case.run([(r, 0, n) for r, n in enumerate(lens)], scale, splits=3)):
        close(o, case.want(r, 0, lens[r], scale), dtype, rough=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank, rot", [(72, 12), (120, 32), (512, 64)])
def test_a_far_key_stands_out_by_its_rotated_part_alone(dtype, rank, rot):
    """One key's rotated part outweighs every other score: all later queries take its value, whatever the page, tile or split."""
    n, H = 330, 3
    for j in (0, 15, 16, 63, 64, 200):
        case = RotatedCase((n,), H, rank, rot, dtype, seed=rot)
        for t in (case.c[0], case.q[0], case.kr[0], case.qr[0]):
            t.mul_(0.1)
        case.c[0][:, 1] = 0.0
        case.c[0][j, 1] = 40.0
        case.qr[0][:, :, rot - 1] = 5.0
        case.kr[0][:, rot - 1] = 0.0
        case.kr[0][j, rot - 1] = 5.0
        case.fill()
        seen = torch.arange(n) >= j
        out = case.run([(0, 0, n)], 1.0)[0][:, :, 1].float().cpu()
        assert ((out > 30).all(1) == seen).all() and (out[~seen] == 0).all(), j
        for i in (j, n - 1):
            for splits in (None, 4):
                assert (case.run([(0, i, 1)], 1.0, splits=splits)[0][0, :, 1].float() > 30).all(), (j, i)


# ------------------------------------------------------------------ differential attention
class PairCase(GqaCase):
    """Keys of two maps and their values of several requests on shuffled pages of one cache; queries, gates."""

    def __init__(self, lens, H, G, d, e, dtype, seed=0):
        from cubic_serve_b200.models.layered import DifferentialSpec, RotarySpec
        spec = DifferentialSpec(H, G, d, e, 1.0, RotarySpec(0, 1.0), 0.5)
        spec.validate()
        super().__init__(lens, H, G, 1, dtype, seed)
        self.d, self.e, self.P = d, e, spec.width_padded
        g = torch.Generator().manual_seed(seed + 1)
        self.k, self.q = ([torch.randn(n, heads, 2, d, generator=g).to(dtype) for n in lens] for heads in (G, H))
        self.v, self.gate = ([torch.randn(n, heads, e, generator=g).to(dtype) for n in lens] for heads in (G, H))
        self.refill()

    def fill(self):
        pass

    def rows(self, t):
        """Both maps of a head in a row of P columns."""
        out = torch.zeros(*t.shape[:2], 2, self.P // 2, dtype=self.dtype)
        out[..., :self.d] = t
        return out.flatten(2)

    def refill(self):
        self.cache = torch.full((self.pages, self.G, 2, 16, self.P), 1e4, dtype=self.dtype)
        for r, n in enumerate(self.lens):
            k, v = self.rows(self.k[r]), torch.nn.functional.pad(self.v[r], (0, self.P - self.e))
            for p in range(-(-n // 16)):
                page, m = self.cache[self.table[r, p]], min(16, n - 16 * p)
                for which, t in ((0, k), (1, v)):
                    page[:, which, :m] = t[16 * p:16 * p + m].transpose(0, 1)

    def run(self, spans, chunk, scale, less, out_scale=0.6, eps=1e-4, splits=None, decode=None):
        from cubic_serve_b200.ops import kernels as K
        q = torch.cat([self.rows(self.q[r][a:a + n]) for r, a, n in spans])
        T, n = q.shape[0], self.H * self.e
        wide, out = padded(T, n, self.dtype, fill=3.0)
        gates, z = padded(T, n, self.dtype)
        z.copy_(torch.cat([self.gate[r][a:a + c] for r, a, c in spans]).view(T, n))
        K.gqa_attention(q.view(T, -1).to(DEV), self.cache.to(DEV), self.table.to(DEV), segs([(c, r, a) for r, a, c in spans]), out, self.H, self.e,
                        0, scale, out_scale=out_scale, chunk=chunk, pair=(z, less, eps), splits=splits,
                        decode=T == len(spans) if decode is None else decode)
        assert untouched(wide, n, fill=3.0)
        return out.reshape(T, self.H, self.e).split([c for _, _, c in spans])

    def want(self, r, first, n, chunk, scale, less, out_scale=0.6, eps=1e-4):
        q, k, v = self.q[r][first:first + n].double(), self.k[r][:first + n].double(), self.v[r][:first + n].double()
        seen = R.same_chunk(first, n, first + n, chunk or None)
        a1, a2 = (R.masked_attention(q[:, :, i], k[:, :, i], v, seen, scale) for i in range(2))
        return R.rms(a1 - less * a2, eps) * out_scale * R.sigmoid(self.gate[r][first:first + n].double())


PAIRS = [(6, 2, 24, 40, 37), (3, 1, 13, 9, 0), (32, 8, 64, 128, 130), (40, 1, 72, 136, 16), (4, 4, 100, 250, 100), (1, 1, 24, 16, 1), (70, 1, 32, 64, 50),
         (10, 5, 128, 256, 17), (9, 3, 64, 32, 0), (4, 2, 16, 128, 33), (18, 2, 40, 24, 48)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, d, e, chunk", PAIRS)
def test_differential_attention_prefill_portions_and_decode(dtype, H, G, d, e, chunk):
    lens = (150, 3, 61, 16)
    case = PairCase(lens, H, G, d, e, dtype, seed=H)
    # a factor far from one: where the maps nearly cancel, the norm would amplify rounding
    scale, less, rough = 1.5 / d ** 0.5, -0.7, 1.5e-2
    for r, o in enumerate(case.run([(r, 0, n) for r, n in enumerate(lens)], chunk, scale, less)):
        close(o, case.want(r, 0, lens[r], chunk, scale, less), dtype, rough=rough)
    spans = [(2, 40, 21), (0, 149, 1), (1, 1, 2), (3, 15, 1), (0, 20, 90)]
    for (r, first, n), o in zip(spans, case.run(spans, chunk, scale, less, out_scale=1.3)):
        close(o, case.want(r, first, n, chunk, scale, less, out_scale=1.3), dtype, rough=rough)
    spans = [(r, n - 1, 1) for r, n in enumerate(lens)] + [(0, 49, 1), (0, 50, 1), (2, 16, 1)]
    for splits in (None, 1, 2, 7):
        for (r, first, n), o in zip(spans, case.run(spans, chunk, scale, less, splits=splits)):
            close(o, case.want(r, first, n, chunk, scale, less), dtype, rough=rough)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("less", [0.0, 0.4, 1.3])
def test_the_second_map_is_taken_away(dtype, less):
    """Maps that look at different keys with values of their own: the difference, its sign, and nothing of the second with factor 0."""
    n, d, e = 40, 16, 24
    case = PairCase((n,), 2, 1, d, e, dtype, seed=2)
    case.q[0].zero_()
    case.k[0].zero_()
    case.q[0][:, :, :, 0] = 8.0
    case.k[0][3, :, 0, 0], case.k[0][7, :, 1, 0] = 4.0, 4.0
    case.refill()
    out = case.run([(0, 8, 32)], 0, 1.0, less)[0]
    v = case.v[0].double()
    want = (R.rms(v[3, 0] - less * v[7, 0], 1e-4) * 0.6).expand(32, 2, e) * R.sigmoid(case.gate[0][8:].double())
    close(out, want, dtype, exact=1e-5, rough=1.5e-2)
    for i in (8, 39):
        close(case.run([(0, i, 1)], 0, 1.0, less)[0], want[i - 8:i - 7], dtype, exact=1e-5, rough=1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("chunk", [1, 2, 15, 16, 17, 31, 33, 63, 64, 65, 129])
def test_chunk_edge_shows_one_key(dtype, chunk, which):
    """One key of one map carries a score that outweighs all others and a value nothing else has: it is seen by exactly the later
    queries of its chunk, in a prompt, in portions that start inside or at the edge of a chunk, and decoded."""
    n, H, d, e = 200, 4, 16, 32
    for j in (0, 15, 16, 47, 64, 130):
        case = PairCase((n,), H, 2, d, e, dtype, seed=chunk)
        for t in (case.q[0], case.k[0]):
            t.mul_(0.1)
        case.q[0][..., which, 0] = 6.0
        case.k[0][..., which, 0] = 0.0
        case.k[0][j, :, which, 0] = 6.0
        case.v[0].mul_(0.5)
        case.v[0][:, :, 1] = 0.0
        case.v[0][j, :, 1] = 60.0
        case.gate[0].zero_()
        case.refill()
        seen = torch.tensor([i >= j and i // chunk == j // chunk for i in range(n)])
        # the value's own channel is most of the normed difference when its key is seen; the other map sees one key of its chunk as any other
        less = 0.5 if which == 0 else 2.0
        show = lambda o: o[:, :, 1].float().cpu().abs() > 0.9                           # noqa: E731
        want = case.want(0, 0, n, chunk, 1.0, less)[:, :, 1].abs()
        assert ((want[seen] > 1.2).all() or chunk == 1) and (want[~seen] < 0.1).all()
        out = case.run([(0, 0, n)], chunk, 1.0, less)[0]
        if chunk > 1:
            assert (show(out).all(1) == seen).all() and (out[~seen.to(DEV)][:, :, 1].abs() < 0.1).all(), (chunk, j)
        close(out, case.want(0, 0, n, chunk, 1.0, less), dtype, exact=1e-4, rough=3e-2)
        edge = (j // chunk + 1) * chunk
        for a, b in ((max(0, edge - 2), min(n, edge + 3)), (min(edge, n - 2), min(n, edge + 20))):
            if b - a > 1:
                close(case.run([(0, a, b - a)], chunk, 1.0, less)[0], case.want(0, a, b - a, chunk, 1.0, less), dtype, exact=1e-4, rough=3e-2)
        for i in {j, edge - 1, edge}:
            if j <= i < n:
                for splits in (None, 4):
                    close(case.run([(0, i, 1)], chunk, 1.0, less, splits=splits)[0], case.want(0, i, 1, chunk, 1.0, less), dtype, exact=1e-4,
                          rough=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window, chunk", [(0, 30), (30, 0)])
def test_chunks_and_windows_of_one_map(dtype, window, chunk):
    """The same chunks in attention with one map, beside the window they replace."""
    from cubic_serve_b200.ops import kernels as K
    case = GqaCase((100, 40), 6, 2, 24, dtype, seed=3)
    for decode in (False, True):
        spans = [(0, 99, 1), (1, 30, 1)] if decode else [(0, 0, 100), (1, 13, 27)]
        q = torch.zeros(sum(n for _, _, n in spans), 6, case.P, dtype=dtype)
        q[:, :, :24] = torch.cat([case.q[r][a:a + n] for r, a, n in spans])
        out = torch.zeros(q.shape[0], 144, dtype=dtype, device=DEV)
        K.gqa_attention(q.flatten(1).to(DEV), case.cache.to(DEV), case.table.to(DEV), segs([(n, r, a) for r, a, n in spans]), out, 6, 24, window,
                        0.4, decode=decode, chunk=chunk)
        for (r, a, n), o in zip(spans, out.view(-1, 6, 24).split([n for _, _, n in spans])):
            k, v = case.k[r][:a + n].double(), case.v[r][:a + n].double()
            seen = R.same_chunk(a, n, a + n, chunk) if chunk else R.kept_window(a, n, a + n, window, 0)
            close(o, R.masked_attention(case.q[r][a:a + n].double(), k, v, seen, 0.4), dtype, rough=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [5, 40, 700])
@pytest.mark.parametrize("H, G, d, e, pairs, maps", [(6, 2, 24, 40, 6, 2), (3, 1, 13, 9, 3, 2), (32, 8, 64, 128, 32, 2), (5, 5, 100, 250, 20, 2), (1, 1, 7, 5, 0, 2),
                                                     (4, 2, 128, 256, 64, 2), (9, 3, 32, 64, 2, 2), (4, 2, 60, 60, 30, 1), (3, 1, 128, 96, 5, 1)])
def test_head_norms_and_rotated_halves(dtype, T, H, G, d, e, pairs, maps):
    from cubic_serve_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T + d)
    P = next(p for p in (64, 128, 256) if max(maps * d, e) <= p)
    r8 = lambda n: -(-n // 8) * 8                                                      # noqa: E731
    offs = (8, 8 + r8(H * maps * d), 8 + r8(H * maps * d) + r8(G * maps * d))
    x = torch.full((T, offs[2] + r8(G * e) + 8), 50.0).to(dtype)
    parts = [torch.randn(T, n, generator=g).to(dtype) for n in (H * maps * d, G * maps * d, G * e)]
    for o, t in zip(offs, parts):
        x[:, o:o + t.shape[1]] = t
    qw, kw = (1 + 0.3 * torch.randn(d, generator=g) for _ in range(2))
    base, eps = 300.0, 1e-3
    freq = split_freq(torch.tensor([base ** (-i / max(pairs, 1)) for i in range(pairs)], dtype=torch.float64))
    pos = torch.randint(0, 500, (T,), generator=g, dtype=torch.int32)
    pos[0], pos[1] = 0, 990000
    pages = T // 8 + 2
    slots = torch.randperm(16 * pages, generator=g)[:T].to(torch.int32)
    slots[T // 2] = -1
    q = torch.full((T, H * P), 9.0, dtype=dtype, device=DEV)
    cache = torch.full((pages, G, 2, 16, P), 3.0, dtype=dtype, device=DEV)
    K.head_qkv(x.to(DEV), offs, qw.to(DEV), kw.to(DEV), freq, pos.to(DEV), slots.to(DEV), q, cache, H, d, e, eps, maps)

    def turned(t, heads, w):
        y = R.rms(t.double().view(T, heads * maps, d), eps) * w.double()
        y = torch.stack([R.rotate_halves(y[i:i + 1], int(pos[i]), 2 * pairs, base)[0] for i in range(T)])
        out = torch.zeros(T, heads, maps, P // maps, dtype=torch.float64)
        out[..., :d] = y.view(T, heads, maps, d)
        return out.flatten(2)

    close(q.view(T, H, P), turned(parts[0], H, qw), dtype, exact=5e-6, rough=8e-3)
    rows = cache.permute(2, 0, 3, 1, 4).reshape(2, -1, G, P)
    live = slots >= 0
    at = slots[live].long()
    close(rows[0][at], turned(parts[1], G, kw)[live], dtype, exact=5e-6, rough=8e-3)
    close(rows[1][at], torch.nn.functional.pad(parts[2].double().view(T, G, e), (0, P - e))[live], dtype, exact=0, rough=4e-3)
    rest = torch.ones(rows.shape[1], dtype=torch.bool)
    rest[at] = False
    assert (rows[:, rest] == 3).all()


# ------------------------------------------------------------------ element-wise recurrence
def gru_oracle(z, x, g, bias, S):
    """The mechanism from the projections on, in fp64: (outputs, state).  The products of the mixer are identities."""
    n, c = z.shape
    eye = torch.eye(3 * c, dtype=torch.float64)
    w = {"p.z": eye[:c], "p.x": eye[c:2 * c], "p.g": eye[2 * c:], "p.z.b": bias[0].double(), "p.x.b": bias[1].double(), "p.o": torch.eye(c, dtype=torch.float64)}
    st = {} if S is None else {"S": S}
    out = R.mingru_mixer(w, "p", {"width": c}, torch.cat([z, x, g], 1).double(), st, 0.0)
    return out, st["S"]


class Gru:
    def __init__(self, width, dtype, slots=6, seed=0):
        self.g = torch.Generator().manual_seed(seed + width)
        self.width, self.dtype, self.ld = width, dtype, -(-width // 4) * 4
        self.bias = torch.stack([torch.randn(width, generator=self.g) - 2.0, torch.randn(width, generator=self.g)])
        self.state = torch.full((slots, self.ld), 50.0, device=DEV)        # stale contents: a fresh request must not read them

    def rows(self, n):
        return tuple((1.5 * torch.randn(n, self.width, generator=self.g)).to(self.dtype) for _ in range(3))

    def run(self, zxg, seg):
        from cubic_serve_b200.ops import kernels as K
        T, r8 = zxg[0].shape[0], -(-self.width // 8) * 8
        x = torch.full((T, 8 + 3 * r8), 50.0, dtype=self.dtype)
        offs = [8 + i * r8 for i in (2, 0, 1)]
        for o, t in zip(offs, zxg):
            x[:, o:o + self.width] = t
        wide, out = padded(T, self.width, self.dtype)
        K.mingru(x.to(DEV), *offs, self.bias.to(DEV), self.state, seg if not isinstance(seg, list) else segs(seg), out)
        assert untouched(wide, self.width)
        return out.clone()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [1, 16, 37, 72, 130, 1024])
@pytest.mark.parametrize("cuts", [(2, 37, 128, 17, 2, 1, 1, 300, 3), (129, 1, 256, 2), (7, 8, 9, 127)])
def test_recurrence_in_portions(dtype, width, cuts):
    """Portions around the lengths of runs and turns, down to one token, on a slot with stale contents; other slots stay."""
    c = Gru(width, dtype)
    zxg = c.rows(sum(cuts))
    want, S = gru_oracle(*zxg, c.bias, None)
    got, i = [], 0
    for n in cuts:
        got.append(c.run([t[i:i + n] for t in zxg], [(n, 2, i)]))
        i += n
    close(torch.cat(got), want, dtype, exact=1e-5, rough=8e-3)
    close(c.state[2, :width], S, torch.float32, exact=1e-5)
    assert (c.state[[0, 1, 3, 4, 5]] == 50).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [31, 64, 200])
def test_long_prompts_share_a_segment_among_blocks(dtype, width):
    """Prompts long enough for clusters of 2, 4 and 8 blocks, alone, behind earlier tokens and beside shorter ones."""
    c = Gru(width, dtype)
    for cuts in ((256, 3), (700, 513), (2100,), (1, 1025)):
        zxg = c.rows(sum(cuts))
        want, S = gru_oracle(*zxg, c.bias, None)
        got, i = [], 0
        for n in cuts:
            got.append(c.run([t[i:i + n] for t in zxg], [(n, 3, i)]))
            i += n
        close(torch.cat(got), want, dtype, exact=1e-5, rough=8e-3)
        close(c.state[3, :width], S, torch.float32, exact=1e-5)
    lens = (5, 900, 0, 130)
    rows = [c.rows(n) for n in lens]
    out = c.run([torch.cat([r[i] for r in rows]) for i in range(3)], [(n, s, 0) for s, n in enumerate(lens)])
    for s, (r, o) in enumerate(zip(rows, out.split(lens))):
        if lens[s]:
            want, S = gru_oracle(*r, c.bias, None)
            close(o, want, dtype, exact=1e-5, rough=8e-3)
            close(c.state[s, :width], S, torch.float32, exact=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 37, 260])
def test_recurrence_batches(dtype, width):
    """Unequal requests in one step equal each alone; decode steps with a padding segment; a slot that is used again."""
    c = Gru(width, dtype)
    lens, slots = (33, 1, 2, 150, 16), (4, 0, 3, 1, 2)
    for turn in range(2):
        rows = [c.rows(n + 1) for n in lens]
        oracle = [gru_oracle(*(t[:n] for t in r), c.bias, None) for r, n in zip(rows, lens)]
        out = c.run([torch.cat([r[i][:n] for r, n in zip(rows, lens)]) for i in range(3)], [(n, s, 0) for n, s in zip(lens, slots)])
        for o, (want, _) in zip(out.split(lens), oracle):
            close(o, want, dtype, exact=1e-5, rough=8e-3)
        order = [0, 1, None, 2, 3, 4]
        bucket = segs([(1, slots[i], lens[i]) if i is not None else (0, 0, 0) for i in order])
        bucket.row0 = torch.arange(len(order), dtype=torch.int32, device=DEV)
        step = [torch.cat([rows[i][k][lens[i]:] if i is not None else torch.zeros(1, width, dtype=dtype) for i in order]) for k in range(3)]
        idle = c.state[5].clone()
        out = decode_rows(c, step, bucket)
        for j, i in enumerate(order):
            if i is None:
                continue
            want, S = gru_oracle(*(t[lens[i]:] for t in rows[i]), c.bias, oracle[i][1])
            close(out[j:j + 1], want, dtype, exact=1e-5, rough=8e-3)
            close(c.state[slots[i], :width], S, torch.float32, exact=1e-5)
        assert torch.equal(c.state[5], idle)


def decode_rows(c, step, bucket):
    """One token per segment; the padding segment's row is left as it was."""
    from cubic_serve_b200.ops import kernels as K
    r8 = -(-c.width // 8) * 8
    x = torch.zeros(step[0].shape[0], 3 * r8, dtype=c.dtype)
    for i, t in enumerate(step):
        x[:, i * r8:i * r8 + c.width] = t
    out = torch.zeros(x.shape[0], r8, dtype=c.dtype, device=DEV)[:, :c.width]
    K.mingru(x.to(DEV), 0, r8, 2 * r8, c.bias.to(DEV), c.state, bucket, out)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
def test_candidates_meet_at_zero_and_gates_saturate(dtype):
    """The candidate's two branches, a gate that takes everything, one that keeps everything over many tokens."""
    c = Gru(4, dtype)
    c.bias = torch.zeros(2, 4)
    z = torch.tensor([[60.0, 60.0, 60.0, 60.0]]).expand(400, 4).clone()
    z[1:] = -60.0
    x = torch.tensor([[0.0, -1e-3, 1e-3, -8.0]]).expand(400, 4).clone()
    g = torch.full((400, 4), 1.0)
    zxg = [t.to(dtype) for t in (z, x, g)]
    want, S = gru_oracle(*zxg, c.bias, None)
    got = c.run(zxg, [(400, 0, 0)])
    close(got, want, dtype, exact=1e-6, rough=8e-3)
    close(c.state[0], S, torch.float32, exact=1e-6)
    assert abs(float(c.state[0, 0]) - 0.5) < 1e-6
