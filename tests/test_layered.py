"""Layered decoders on the CPU: configuration and inventory, packing, the oracle's mechanisms, imposed steps, the eager mode."""
import copy
import io
import json
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
from layered_cases import CASES, LOW_RANKS, channel, config, delta, latent, prompt, tensors, write  # noqa: E402

from cubic_serve_b200.models import layered as L  # noqa: E402
from cubic_serve_b200.models import layered_reference as R  # noqa: E402
from cubic_serve_b200.models.checkpoint import CheckpointError, admit_checkpoint, inspect_checkpoint  # noqa: E402


def parsed(name):
    w = tensors(CASES[name])
    return L.parse_layered_config(CASES[name], {n: tuple(t.shape) for n, t in w.items()}), w


# ------------------------------------------------------------------ configuration and inventory
@pytest.mark.parametrize("name", list(CASES))
def test_config_and_inventory(name):
    cfg, w = parsed(name)
    L.check_inventory(cfg, {n: tuple(t.shape) for n, t in w.items()})
    back = L.parse_layered_config(cfg.to_config(), {n: tuple(t.shape) for n, t in w.items()}, name=cfg.name)
    assert back == cfg
    loop = CASES[name]["loop"]
    runs = len(cfg.layers) + ((loop["times"] - 1) * (loop["stop"] - loop["start"]) if loop else 0)
    assert len(cfg.runs) == runs == len(R.layer_schedule(CASES[name]))
    assert [i for i, _ in cfg.runs] == [i for i, _ in R.layer_schedule(CASES[name])]
    assert sum(enters for _, enters in cfg.runs) == (loop["times"] if loop else 0)


def test_low_ranks_come_from_the_tensors():
    cfg, _ = parsed("all")
    m = cfg.layers[2].mixer
    assert (m.decay_rank, m.gate_rank) == LOW_RANKS
    with pytest.raises(L.LayeredConfigError, match="stated by the checkpoint's tensors"):
        L.parse_layered_config(CASES["all"])


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda c: c.update(architecture="Other"), "not one of"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "grouped evenly"),
    (lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}), "at least the token itself"),
    (lambda c: c["loop"].update(stop=9), "loop needs"),
    (lambda c: c["layers"][0]["mixer"].update(dim=400), "key width"),
])
def test_bad_configurations_are_refused(change, message):
    c = copy.deepcopy(CASES["all"])
    change(c)
    with pytest.raises(L.LayeredConfigError, match=message):
        L.parse_layered_config(c, {n: tuple(t.shape) for n, t in tensors(CASES["all"]).items()})


def test_checkpoint_admission(tmp_path):
    w = tensors(CASES["all"])
    ck = admit_checkpoint(write(tmp_path / "good", CASES["all"], w))
    assert ck.cfg.family == "layered" and ck.cfg.vocab_size == 200 and ck.raw_config == CASES["all"]
    info = inspect_checkpoint(tmp_path / "good")
    assert info["layer_runs"] == 6 and info["mixers"] == {"channel_delta": 1, "delta": 1, "latent": 2}
    with pytest.raises(CheckpointError, match="missing tensor l0.mix.b"):
        admit_checkpoint(write(tmp_path / "missing", CASES["all"], {n: t for n, t in w.items() if n != "l0.mix.b"}))
    with pytest.raises(CheckpointError, match="does not own"):
        admit_checkpoint(write(tmp_path / "extra", CASES["all"], {**w, "l9.norm1": w["l0.norm1"].clone()}))
    with pytest.raises(CheckpointError, match="expected"):
        admit_checkpoint(write(tmp_path / "shape", CASES["all"], {**w, "head": w["head"][:5].clone()}))


def test_registry_and_memory_plan(tmp_path):
    from cubic_serve_b200.contracts.model import ModelSpec
    from cubic_serve_b200.contracts.plan import decoder_step_operators
    from cubic_serve_b200.models import registry
    defn = registry.for_architecture("Bumodra")
    assert defn.family == "layered"
    cfg = defn.parse_config(write(tmp_path, CASES["all"], tensors(CASES["all"])))
    # every run of a looped layer has a cache or a state of its own: 3 attention runs, 3 delta runs
    spec = ModelSpec.from_layered(cfg)
    assert spec.cache.runs == 3 and spec.state.runs == 3
    assert spec.cache.page_bytes == 3 * 16 * 64 * 2
    pages = spec.kv_pages(1 << 20, 0, 4096, 4)
    assert pages == ((1 << 20) - 4 * cfg.state_bytes_per_request) // spec.cache.page_bytes
    assert {o.semantic_op for o in decoder_step_operators(cfg, 8)} >= {"attention.latent", "delta_rule.head", "delta_rule.channel"}


# ------------------------------------------------------------------ packing
@pytest.mark.parametrize("H, n, k", [(5, 64, 16), (3, 128, 24), (6, 24, 64), (4, 32, 128), (7, 20, 64), (1, 16, 64), (9, 96, 64)])
def test_block_diagonal_operand_is_the_per_head_product(H, n, k):
    w = torch.randn(H, n, k).to(torch.bfloat16)
    b = L.BlockDiagonal.pack(w)
    assert b.rows == 0 and b.heads == H or b.rows == b.heads * n and b.rows % 128 == 0
    kg = b.w.k
    x = torch.randn(3, H, k)
    cols = torch.zeros(3, -(-H // b.heads) * kg)              # heads where their group reads them
    for h in range(H):
        c = (h // b.heads) * kg + (h % b.heads) * k
        cols[:, c:c + k] = x[:, h]
    dense = b.w.codes.float()
    out = torch.empty(3, H * n)
    for r in range(H * n):
        g = r // b.rows if b.rows else 0
        out[:, r] = cols[:, g * kg:(g + 1) * kg] @ dense[r]
    want = torch.einsum("thk,hnk->thn", x, w.float()).reshape(3, H * n)
    assert torch.allclose(out, want, atol=1e-4)


def test_projection_sections_are_aligned_and_complete():
    cfg, w = parsed("all")
    for i, l in enumerate(cfg.layers):
        p = L.pack_layer(cfg, i, w.__getitem__)
        rows, m = p.proj.codes.float()[:, :cfg.hidden_size], p.mixer
        assert p.split % 8 == 0 and p.proj.n == p.split + l.ff and p.out.n == cfg.hidden_size
        if l.ff:
            assert torch.equal(rows[p.split:], w[f"l{i}.mlp.up"].float())
            assert torch.equal(p.out.codes.float()[:, p.out_off:p.out_off + l.ff], w[f"l{i}.mlp.down"].float())
        assert torch.equal(p.out.codes.float()[:, :m.spec.out_width], w[f"l{i}.mix.o"].float())
        at = {"l0.mix.b": (0, "b_off"), "l0.mix.a": (0, "a_off"), "l0.mix.g": (0, "z_off"), "l1.mix.dkv": (1, "c_off"),
              "l1.mix.g": (1, "g_off"), "l2.mix.a1": (2, "a_off")}
        for name, (layer, attr) in at.items():
            if layer == i:
                off, t = getattr(m, attr), w[name]
                assert off % 8 == 0 and torch.equal(rows[off:off + t.shape[0]], t.float())


# ------------------------------------------------------------------ the oracle's mechanisms, against element-wise loops
def test_oracle_norms_and_activations():
    x, w = torch.randn(3, 5, dtype=torch.float64), torch.randn(5, dtype=torch.float64)
    for r in range(3):
        ms = sum(float(v) ** 2 for v in x[r]) / 5
        for c in range(5):
            assert abs(float(R.rms_around_zero(x, w, 1e-3)[r, c]) - float(x[r, c]) / (ms + 1e-3) ** 0.5 * (1 + float(w[c]))) < 1e-12
    u = R.unit(x)
    assert torch.allclose((u * u).sum(-1), (x * x).sum(-1) / ((x * x).sum(-1) + 1e-6))
    assert torch.allclose(R.softplus(x), torch.log(1 + torch.exp(x)))
    assert R.squared_relu(torch.tensor([-2.0, 0.0, 3.0])).tolist() == [0.0, 0.0, 9.0]


@pytest.mark.parametrize("taps", [1, 2, 4])
def test_oracle_convolution(taps):
    x, w = torch.randn(6, 3), torch.randn(3, taps)
    y, past = R.short_conv(x, w, torch.zeros(taps - 1, 3))
    for t in range(6):
        for c in range(3):
            s = sum(float(w[c, taps - 1 - d] * x[t - d, c]) for d in range(taps) if t - d >= 0)
            assert abs(float(y[t, c]) - s / (1 + np.exp(-s))) < 1e-5
    assert torch.equal(past, x[6 - (taps - 1):])
    a, p1 = R.short_conv(x[:1], w, torch.zeros(taps - 1, 3))
    b, p2 = R.short_conv(x[1:], w, p1)
    assert torch.allclose(torch.cat([a, b]), y, atol=1e-6) and torch.equal(p2, past)


def test_oracle_delta_step():
    H, d, e = 2, 3, 4
    S, q, k, v = torch.randn(H, d, e), torch.randn(H, d), torch.randn(H, d), torch.randn(H, e)
    beta, decay = torch.rand(H), torch.rand(H, d)
    o, S2 = R.delta_step(S, q, k, v, beta, decay)
    for h in range(H):
        for j in range(e):
            col = [float(decay[h, i] * S[h, i, j]) for i in range(d)]
            u = float(beta[h]) * (float(v[h, j]) - sum(col[i] * float(k[h, i]) for i in range(d)))
            col = [col[i] + float(k[h, i]) * u for i in range(d)]
            assert np.allclose(col, S2[h, :, j].numpy(), atol=1e-5)
            assert abs(sum(col[i] * float(q[h, i]) for i in range(d)) - float(o[h, j])) < 1e-5      # reads its own write


@pytest.mark.parametrize("window", [1, 4, None])
def test_oracle_window_edges(window):
    n, H, d = 9, 2, 4
    q, k, v = torch.randn(n, H, d), torch.randn(n, H, d), torch.randn(n, H, 3)
    base = R.windowed_attention(q, k, v, 0, window, 0.7)
    for j in range(n):                                      # which queries notice that key j changed
        k2 = k.clone()
        k2[j] += 3.0
        moved = (R.windowed_attention(q, k2, v, 0, window, 0.7) - base).abs().amax((1, 2)) > 1e-6
        seen = [i for i in range(n) if 0 <= i - j and (window is None or i - j < window)]
        if window == 1:
            assert not moved.any()                          # a single visible key has weight one whatever its score is
        else:
            first = j if j else 1                           # the first token sees only itself
            assert [i for i in range(n) if moved[i]] == [i for i in seen if i >= first]


@pytest.mark.parametrize("name", list(CASES))
def test_oracle_portions_equal_one_pass(name):
    o = R.Oracle(CASES[name], tensors(CASES[name]), torch.float64)
    ids = prompt(CASES[name], 61, 0)
    whole, _ = o.forward(ids)
    for cuts in ([1] * 61, [2, 2, 57], [40, 1, 20], [16, 16, 16, 13]):
        st, parts, i = None, [], 0
        for c in cuts:
            lg, st = o.forward(ids[i:i + c], st)
            parts.append(lg)
            i += c
        assert torch.allclose(torch.cat(parts), whole, atol=1e-9)
    last, _ = o.forward(ids, last_only=True)
    assert torch.allclose(last[0], whole[-1], atol=1e-9)


# ------------------------------------------------------------------ imposed steps through scheduler and pool
class RecordingExecutor:
    """Answers imposed steps from the oracle and records where the scheduler put things."""
    keeps_request_state = True

    def __init__(self, cfg, raw, w):
        self.cfg, self.oracle, self.states, self.calls = cfg, R.Oracle(raw, w), {}, []

    def execute(self, segs):
        raise AssertionError("imposed steps sample nothing")

    def copy_pages(self, pairs):
        raise AssertionError("nothing is shared")

    def execute_logits(self, segs):
        self.calls.append([(s.request_slot, s.start, len(s.token_ids), list(s.pages)) for s in segs])
        out = []
        for s in segs:
            if s.start == 0:
                self.states[s.request_slot] = self.oracle.new_state()
            st = self.states[s.request_slot]
            assert st.length == s.start and len(s.pages) * 16 >= s.start + len(s.token_ids)
            lg, _ = self.oracle.forward(s.token_ids, st)
            out.append(lg[s.logit_offsets].float().numpy())
        return out


def imposed(name="small", pages=9, requests=2):
    from cubic_serve_b200.runtime.engine import LLMEngine
    from cubic_serve_b200.runtime.imposed import ImposedSession
    from cubic_serve_b200.runtime.scheduler import SchedulerConfig
    cfg, w = parsed(name)
    ex = RecordingExecutor(cfg, CASES[name], w)
    eng = LLMEngine(ex, num_pages=pages, scheduler_config=SchedulerConfig(
        max_running_requests=requests, max_model_len=(pages - 1) * 16, max_batched_tokens=(pages - 1) * 16, enable_prefix_cache=False))
    return ImposedSession(eng), ex, R.Oracle(CASES[name], w)


def test_imposed_steps_reuse_pages_and_slots():
    s, ex, oracle = imposed(pages=10)
    for turn in range(3):                                   # 9 pages, 2 slots: the second and third turns reuse all of them
        a, b = prompt(CASES["small"], 70, turn), prompt(CASES["small"], 50, 10 + turn)
        la, _ = oracle.forward(a)
        lb, _ = oracle.forward(b)
        out = s.step([("a", a[:33], [0, 32])])
        assert np.allclose(out[0], la[[0, 32]].numpy(), atol=1e-5)
        out = s.step([("a", a[33:34], [0]), ("b", b[:49], [])])
        assert np.allclose(out[0], la[[33]].numpy(), atol=1e-5) and out[1].shape == (0, 70)
        out = s.step([("b", b[49:], [0]), ("a", a[34:], [35])])
        assert np.allclose(out[0], lb[[49]].numpy(), atol=1e-5) and np.allclose(out[1], la[[69]].numpy(), atol=1e-5)
        assert {p for _, _, _, pages in ex.calls[-1] for p in pages} == set(range(1, 10))      # 5 + 4 pages: all of them
        s.end(["a", "b"])
        assert s.engine.pool.num_used == 0
    assert {c[0] for call in ex.calls for c in call} == {0, 1}


def test_imposed_steps_refuse_what_does_not_fit():
    from cubic_serve_b200.runtime.cache.pool import OutOfPages
    from cubic_serve_b200.runtime.scheduler import AdmissionError
    s, _, _ = imposed(pages=5)
    s.step([("a", [1] * 33, []), ("b", [2], [])])
    with pytest.raises(OutOfPages):
        s.step([("b", [3] * 20, [])])
    s, _, _ = imposed(pages=5)
    s.step([("a", [1], []), ("b", [2], [])])
    with pytest.raises(AdmissionError, match="slot"):
        s.step([("c", [3], [])])
    s, _, _ = imposed(pages=5)
    for bad in ([("a", [], [])], [("a", [70], [])], [("a", [1], [1])], [("a", [1], []), ("a", [2], [])]):
        with pytest.raises(ValueError):
            s.step(bad)
    with pytest.raises(ValueError, match="not live"):
        s.end(["zz"])
    # a request may fill the pool to its last position
    s, _, _ = imposed(pages=5)
    assert s.step([("a", [1] * 64, [63])])[0].shape == (1, 70)


def test_trace_lines_and_files(tmp_path):
    from cubic_serve_b200.utils.trace_run import run
    s, _, oracle = imposed()
    a = prompt(CASES["small"], 20, 3)
    la, _ = oracle.forward(a)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:], "want": [1, 0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": a[:2], "want": [1]}], "end": ["b"]}]
    out = io.StringIO()
    run(s, (json.dumps(l) + "\n" for l in lines), tmp_path, stdout=out)
    assert out.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    assert sorted(p.name for p in tmp_path.iterdir()) == ["1.f32", "2.f32"]
    got = np.fromfile(tmp_path / "1.f32", "<f4").reshape(2, 70)
    assert np.allclose(got, la[[19, 18]].numpy(), atol=1e-5)
    assert np.allclose(np.fromfile(tmp_path / "2.f32", "<f4"), la[1].numpy(), atol=1e-5)


def test_segments_carry_wanted_rows_without_sampling():
    """The batch builder of a step whose rows are not sampled lists none of them for the sampler."""
    from cubic_serve_b200.executor.gpu_executor import BatchBuilder, Segment
    b = BatchBuilder(4, 64, 128, 1, 1, "cpu")
    batch, rows = b.fill([Segment(0, [1, 2, 3], 30, [1, 2, 3], sample=False, logit_offsets=[0, 2]), Segment(1, [4], 0, [5], sample=False)])
    b.stage.upload()
    assert rows == 0 and batch.num_tokens == 4 and batch.segments.num == 2
    assert batch.segments.row0[:2].tolist() == [0, 3] and batch.segments.pos0[:2].tolist() == [30, 0]
    assert batch.slots[:4].tolist() == [2 * 16 + 14, 2 * 16 + 15, 3 * 16, 5 * 16]


# ------------------------------------------------------------------ serving
def serve_args(model, *more):
    from cubic_serve_b200.cli import build_parser
    return build_parser().parse_args(["serve", str(model), *more])


def backend_of(args, tp=1):
    from cubic_serve_b200.cli import parse_speculative_config
    from cubic_serve_b200.runtime.serving import build_backend
    return build_backend(args, list(range(tp)), tp, parse_speculative_config(args.speculative_config), 8, 8)


def test_eager_mode_generates_like_the_oracle(tmp_path):
    from cubic_serve_b200.runtime.scheduler import SamplingParams
    raw = config(300, 64, [delta(2, 1, 16, 16, 3, 64), latent(2, 16, 16, 24, 32, 20, 0.25, 0), channel(2, 2, 16, 16, 2, 48)], (0, 2, 2))
    w = tensors(raw, 5)
    backend, _ = backend_of(serve_args(write(tmp_path, raw, w), "--execution-mode", "eager", "--prefill-chunk-tokens", "16",
                                       "--token-budget", "32"))
    eng = backend.engine
    backend.close()
    prompts = [prompt(raw, n, n) for n in (1, 17, 50)]
    got = eng.generate(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
    oracle = R.Oracle(raw, w)
    for ids, out in zip(prompts, got):
        lg, st = oracle.forward(ids, last_only=True)
        want = []
        for _ in range(6):
            want.append(int(lg[0].argmax()))
            lg, st = oracle.forward([want[-1]], st, last_only=True)
        assert out == want


@pytest.mark.parametrize("flags, tp, message", [
    (("--speculative-config", '{"method":"ngram","num_speculative_tokens":2}'), 1, "speculative"),
    ((), 2, "one GPU"),
])
def test_serving_refusals(flags, tp, message):
    with pytest.raises(SystemExit, match=message):
        backend_of(serve_args("random:layered-tiny", *flags), tp)


def test_float32_is_refused_for_the_quantized_decoders():
    with pytest.raises(SystemExit, match="float32"):
        backend_of(serve_args("random:toy", "--dtype", "float32"))


def test_reference_and_inspect_commands(tmp_path, capsys):
    from cubic_serve_b200.cli import main
    w = tensors(CASES["small"])
    path = write(tmp_path, CASES["small"], w)
    assert main(["reference", str(path), "--prompt-ids", "3,1,4", "--max-tokens", "3"]) == 0
    got = json.loads(capsys.readouterr().out)
    lg, _ = R.Oracle(CASES["small"], w).forward([3, 1, 4], last_only=True)
    assert got["family"] == "layered" and got["output_ids"][0] == int(lg[0].argmax())
    assert main(["inspect-model", str(path), "--json", "--tp", "2"]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Bumodra" and "one GPU" in info["partition_error"]
