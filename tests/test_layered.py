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
from layered_cases import (ALL, CASES, GATED, LOW_RANKS, SEQUENTIAL, STREAMS, channel, clamped, config, delta, differential,  # noqa: E402
                           far, gated, latent, mamba2, mingru, near, parallel, prompt, rotated, routed, sequential, streams, tensors,
                           write)

from cubic_serve_b200.models import layered as L  # noqa: E402
from cubic_serve_b200.models import layered_reference as R  # noqa: E402
from cubic_serve_b200.models.checkpoint import CheckpointError, admit_checkpoint, inspect_checkpoint  # noqa: E402


def parsed(name):
    w = tensors(ALL[name])
    return L.parse_layered_config(ALL[name], {n: tuple(t.shape) for n, t in w.items()}), w


# ------------------------------------------------------------------ configuration and inventory
@pytest.mark.parametrize("name", list(ALL))
def test_config_and_inventory(name):
    cfg, w = parsed(name)
    L.check_inventory(cfg, {n: tuple(t.shape) for n, t in w.items()})
    back = L.parse_layered_config(cfg.to_config(), {n: tuple(t.shape) for n, t in w.items()}, name=cfg.name)
    assert back == cfg
    loop = ALL[name].get("loop")
    runs = len(cfg.layers) + ((loop["times"] - 1) * (loop["stop"] - loop["start"]) if loop else 0)
    assert len(cfg.runs) == runs == len(R.layer_schedule(ALL[name]))
    assert [i for i, _ in cfg.runs] == [i for i, _ in R.layer_schedule(ALL[name])]
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


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=8), "values of this attention are its keys"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "grouped evenly"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "inside a head"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 0}), "at least the token itself"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0), "tau are positive"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "cut evenly"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "grouped evenly"),
    (lambda c: c["layers"][1]["mixer"].update(state=300), "state width"),
    (lambda c: c.update(loop={"start": 0, "stop": 1, "times": 2}), "run once"),
])
def test_bad_sequential_configurations_are_refused(change, message):
    c = copy.deepcopy(SEQUENTIAL["seq"])
    change(c)
    with pytest.raises(L.LayeredConfigError, match=message):
        L.parse_layered_config(c, {n: tuple(t.shape) for n, t in tensors(SEQUENTIAL["seq"]).items()})


def test_sequential_checkpoint_admission(tmp_path):
    from cubic_serve_b200.contracts.model import ModelSpec
    from cubic_serve_b200.contracts.plan import decoder_step_operators
    from cubic_serve_b200.models import registry
    raw, w = SEQUENTIAL["seq"], tensors(SEQUENTIAL["seq"])
    ck = admit_checkpoint(write(tmp_path / "good", raw, w))
    assert ck.cfg.family == "layered" and registry.for_architecture("Loduzen").family == "layered" and ck.cfg.side_dim == 12
    info = inspect_checkpoint(tmp_path / "good")
    assert info["mixers"] == {"attention+gated_linear": 2, "mamba2": 2} and info["architecture"] == "Loduzen"
    # a second norm without a feed-forward behind it is tolerated, anything else is not
    admit_checkpoint(write(tmp_path / "spare", raw, {**w, "l2.norm2": w["l1.norm2"].clone()}))
    with pytest.raises(CheckpointError, match="does not own"):
        admit_checkpoint(write(tmp_path / "head", raw, {**w, "head": w["embed"].clone()}))
    with pytest.raises(CheckpointError, match="missing tensor side.embed"):
        admit_checkpoint(write(tmp_path / "missing", raw, {n: t for n, t in w.items() if n != "side.embed"}))
    # caches and states of the parts: 2 attentions (keys and values of 64 padded channels), 2 gated linear and 2 mamba2 states
    spec = ModelSpec.from_layered(ck.cfg)
    assert spec.cache.runs == 2 and spec.state.runs == 4 and spec.cache.page_bytes == (2 + 4) * 2 * 16 * 64 * 2
    conv = (3 * (96 + 80) + 2 * (80 + 32)) * 2
    assert ck.cfg.state_bytes_per_request == 4 * (3 * 28 * 20 + 2 * 16 * 32 + 4 * 24 * 20 + 2 * 40 * 16) + conv
    assert {o.semantic_op for o in decoder_step_operators(ck.cfg, 8)} >= {"attention.gqa", "linear_recurrence.head",
                                                                          "linear_recurrence.channel", "token_side"}


def test_random_weights_of_all_designs_are_admitted(tmp_path):
    for name in ("layered-tiny", "layered-seq-tiny", "layered-streams-tiny", "layered-gated-tiny"):
        cfg = L.NAMED[name]()
        back = admit_checkpoint(L.write_checkpoint(tmp_path / name, cfg, L.random_tensors(cfg, 3))).cfg
        assert (back.layers, back.side_dim, back.loop) == (cfg.layers, cfg.side_dim, cfg.loop)
        assert (back.streams, back.embed_scale) == (cfg.streams, cfg.embed_scale)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="latent_attention"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "grouped evenly"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=300), "up to 256 channels"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "convolution taps"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "inside a head"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "at least the token itself"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "not negative"),
    (lambda c: c["layers"][1]["mixer"].update(bias_max=4), "behind their first half"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "positive number of positions"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "no more routes than outputs"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=255), "256 outputs"),
    (lambda c: c.update(streams=9), "residual streams"),
])
def test_bad_stream_configurations_are_refused(change, message):
    c = copy.deepcopy(STREAMS["str"])
    change(c)
    with pytest.raises(L.LayeredConfigError, match=message):
        L.parse_layered_config(c, {n: tuple(t.shape) for n, t in tensors(STREAMS["str"]).items()})


def test_routed_feed_forwards_belong_to_designs_with_streams():
    c = copy.deepcopy(SEQUENTIAL["seq"])
    c["layers"][0]["mlp"] = routed(4, 2, 16)
    with pytest.raises(L.LayeredConfigError, match="unknown feed-forward"):
        L.parse_layered_config(c, {n: tuple(t.shape) for n, t in tensors(SEQUENTIAL["seq"]).items()})


def test_stream_checkpoint_admission(tmp_path):
    from cubic_serve_b200.contracts.model import ModelSpec
    from cubic_serve_b200.contracts.plan import decoder_step_operators
    from cubic_serve_b200.models import registry
    raw, w = STREAMS["str"], tensors(STREAMS["str"])
    ck = admit_checkpoint(write(tmp_path / "good", raw, w))
    assert ck.cfg.family == "layered" and registry.for_architecture("Vimelorn").family == "layered" and ck.cfg.streams == 2
    info = inspect_checkpoint(tmp_path / "good")
    assert info["mixers"] == {"biased_attention": 2, "conv_attention": 3} and info["residual_streams"] == 2 and info["routed_layers"] == 3
    # what a missing feed-forward would need is tolerated, anything else is not
    admit_checkpoint(write(tmp_path / "spare", raw, {**w, "l2.norm2": w["l1.norm2"].clone(), "l2.hc2.in": w["l1.hc2.in"].clone()}))
    with pytest.raises(CheckpointError, match="does not own"):
        admit_checkpoint(write(tmp_path / "extra", raw, {**w, "l1.mlp.e5.up": w["l1.mlp.e0.up"].clone()}))
    with pytest.raises(CheckpointError, match="missing tensor l0.hc2.mix"):
        admit_checkpoint(write(tmp_path / "missing", raw, {n: t for n, t in w.items() if n != "l0.hc2.mix"}))
    with pytest.raises(CheckpointError, match="l1.mix.rel is stated"):
        admit_checkpoint(write(tmp_path / "rel", raw, {n: t for n, t in w.items() if n != "l1.mix.rel"}))
    # keys and values of 64 padded channels for every layer; convolution inputs of the three convolved ones
    spec = ModelSpec.from_layered(ck.cfg)
    assert spec.cache.runs == 5 and spec.cache.page_bytes == (2 + 2 + 4 + 1 + 1) * 2 * 16 * 64 * 2
    conv = (2 * (144 + 48 + 80), 1 * (128 + 128 + 64), 3 * (48 + 16 + 24))
    assert spec.state.runs == 3 and ck.cfg.state_bytes_per_request == 2 * sum(conv) and ck.cfg.is_hybrid
    assert {o.semantic_op for o in decoder_step_operators(ck.cfg, 8)} >= {"attention.gqa", "moe.route", "residual.streams"}
    plain, _ = parsed("str_small")
    assert not plain.is_hybrid and ModelSpec.from_layered(plain).state is None          # one tap: nothing to remember


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0), "positive limit"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rotated as a whole"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=1020), "with their rotated part"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=0), "come together"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "grouped evenly"),
    (lambda c: c["layers"][2]["mixer"].update(dim=129), "128 channels"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=257), "256 channels"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26), "inside a head"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "at least the token itself"),
    (lambda c: c["layers"][1]["mixer"].update(width=0), "positive width"),
    (lambda c: c["loop"].update(start=3), "loop needs"),
])
def test_bad_gated_configurations_are_refused(change, message):
    c = copy.deepcopy(GATED["gat"])
    change(c)
    with pytest.raises(L.LayeredConfigError, match=message):
        L.parse_layered_config(c, {n: tuple(t.shape) for n, t in tensors(GATED["gat"]).items()})


def test_gated_checkpoint_admission(tmp_path):
    from cubic_serve_b200.contracts.model import ModelSpec
    from cubic_serve_b200.contracts.plan import decoder_step_operators
    from cubic_serve_b200.models import registry
    raw, w = GATED["gat"], tensors(GATED["gat"])
    ck = admit_checkpoint(write(tmp_path / "good", raw, w))
    assert ck.cfg.family == "layered" and registry.for_architecture("Fovunex").family == "layered" and ck.cfg.embed_scale == 0.7
    info = inspect_checkpoint(tmp_path / "good")
    assert info["mixers"] == {"differential": 1, "latent": 2, "mingru": 2} and tuple(info["loop"]) == (1, 3, 2) and info["layer_runs"] == 7
    # what a missing feed-forward would need is tolerated, anything else is not
    admit_checkpoint(write(tmp_path / "spare", raw, {**w, "l3.norm2": w["l1.norm2"].clone(), "l3.rg2": w["l1.rg2"].clone()}))
    with pytest.raises(CheckpointError, match="does not own"):
        admit_checkpoint(write(tmp_path / "extra", raw, {**w, "loop.in": w["l0.rg1"].clone()}))
    with pytest.raises(CheckpointError, match="missing tensor l1.rg1.b"):
        admit_checkpoint(write(tmp_path / "missing", raw, {n: t for n, t in w.items() if n != "l1.rg1.b"}))
    with pytest.raises(CheckpointError, match="expected \\(\\)"):
        admit_checkpoint(write(tmp_path / "norm", raw, {**w, "l0.norm1": torch.ones(96).to(torch.bfloat16)}))
    # rows of [72 | 12] and [40 | 8] in 128 and 64 columns, keys of two maps and values of 64; the looped layers' states and caches twice
    spec = ModelSpec.from_layered(ck.cfg)
    assert spec.cache.runs == 4 and spec.cache.page_bytes == 16 * 2 * (128 + 64 + 2 * 2 * 2 * 64)
    assert spec.state.runs == 3 and ck.cfg.state_bytes_per_request == 4 * (2 * 72 + 132) and ck.cfg.is_hybrid
    assert {o.semantic_op for o in decoder_step_operators(ck.cfg, 8)} >= {"attention.latent", "attention.differential", "residual.gate",
                                                                          "linear_recurrence.elementwise"}


@pytest.mark.parametrize("rank, rot, widths", [(72, 12, (128, 128)), (120, 8, (128, 128)), (121, 6, (192, 128)), (128, 64, (192, 128)), (129, 8, (256, 256)),
                                               (256, 64, (320, 256)), (256, 66, (512, 512)), (512, 64, (576, 512)), (512, 66, (1024, 1024)),
                                               (44, 16, (64, 64)), (449, 8, (512, 512))])
def test_widths_of_rotated_rows(rank, rot, widths):
    m = L.LatentSpec(1, 8, 8, 0, rank, 1.0, 0, rot, L.RotarySpec(rot, 10.0), False)
    m.validate()
    assert (m.row_padded, m.rank_padded) == widths and m.rot_col % 8 == 0 and m.rot_col >= rank


def test_passes_of_a_loop_add_the_embedding_before_all_but_the_first():
    cfg, _ = parsed("gat")
    assert [i for i, _ in cfg.runs] == [0, 1, 2, 1, 2, 3, 4] and [r for r in range(7) if cfg.reenters(r)] == [3]
    first, _ = parsed("gat_odd")
    assert [r for r in range(len(first.runs)) if first.reenters(r)] == [4, 8]
    once, _ = parsed("gat_small")
    assert not any(once.reenters(r) for r in range(3)) and not any(parsed("all")[0].reenters(r) for r in range(6))


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


def test_sequential_packing():
    """Sections of the joint projection and of the joint output product, gated rows in the GEMM's order, folded scales."""
    from cubic_serve_b200.ops import wq_pack
    cfg, w = parsed("seq")
    W = cfg.hidden_size
    p = L.pack_layer(cfg, 0, w.__getitem__)
    left, right = p.mixer.left, p.mixer.right
    rows = p.proj.codes.float()[:, :W]
    for name, off in (("left.q", left.q_off), ("left.k", left.k_off), ("right.q", right.q_off), ("right.k", right.k_off),
                      ("right.v", right.v_off), ("right.g", right.g_off), ("right.a1", right.a_off)):
        t = w[f"l0.mix.{name}"]
        assert off % 8 == 0 and torch.equal(rows[off:off + t.shape[0]], t.float())
    assert right.a_off + right.low.k <= p.split == p.proj.n and p.ff == 0
    out = p.out.codes.float()
    assert torch.equal(out[:, :144], w["l0.mix.left.o"].float()) and torch.equal(out[:, 144:228], w["l0.mix.right.o"].float())
    assert left.out_scale == 0.7 and torch.allclose(right.norm_w, 1.3 * w["l0.mix.right.norm"].float())
    assert torch.equal(p.norm, w["l0.norm1"].float()) and torch.equal(p.norm2, w["l0.norm2"].float())
    order = wq_pack.swiglu_row_order(80)
    both = torch.cat([w["l0.mlp.gate"], w["l0.mlp.up"]]).float()
    assert torch.equal(p.gate_up.codes.float()[:, :W], both[order]) and p.gate_up.act_interleaved
    assert torch.equal(p.down.codes.float()[:, :80], w["l0.mlp.down"].float()) and p.down.k == 128
    assert p.side.col == 0 and L.pack_layer(cfg, 3, w.__getitem__).side.col == 36
    m = L.pack_layer(cfg, 1, w.__getitem__)
    rows, s = m.proj.codes.float()[:, :W], m.mixer
    for off, (a, b) in ((s.z_off, (0, 96)), (s.x_off, (96, 96 + 176)), (s.dt_off, (272, 276))):
        assert off % 8 == 0 and torch.equal(rows[off:off + b - a], w["l1.mix.in"].float()[a:b])
    assert torch.equal(s.conv_w[:, :176].t(), w["l1.mix.conv"].float()) and (s.conv_w[:, 176:] == 0).all()
    # a feed-forward width that is no multiple of the activation's block gets zero features
    odd, wo = parsed("seq_odd")
    q = L.pack_layer(odd, 0, wo.__getitem__)
    assert q.gate_up.n == 96 and q.down.k == 64 and (q.down.codes.float()[:, 44:] == 0).all()
    assert L.pack_layer(cfg, 2, w.__getitem__).down is None
    packed = L.pack_weights(cfg, w.__getitem__)
    assert torch.equal(packed.lm_head.codes.float()[:, :W], w["embed"].float()) and packed.embed_norm is None


def test_stream_packing():
    """Sections of the projection and the convolution's columns, distance biases, the routed feed-forward's joint matrix."""
    cfg, w = parsed("str")
    W = cfg.hidden_size
    p = L.pack_layer(cfg, 0, w.__getitem__)
    rows, s = p.proj.codes.float()[:, :W], p.mixer.spec
    for t, off in zip("qkv", s.offsets):
        n = w[f"l0.mix.{t}"].shape[0]
        assert off % 8 == 0 and torch.equal(rows[p.mixer.q_off + off:p.mixer.q_off + off + n], w[f"l0.mix.{t}"].float())
        assert torch.equal(p.mixer.conv_w[:, off:off + n].t(), w[f"l0.mix.{t}.conv"].float())
    assert torch.equal(p.out.codes.float()[:, :s.out_width], w["l0.mix.o"].float())
    exact = torch.tensor([1000.0 ** (-i / 6) for i in range(6)], dtype=torch.float64)
    assert torch.equal(p.mixer.freq[0].double(), exact.float().double())
    assert (p.mixer.freq.double().sum(0) - exact).abs().max() < 1e-14
    assert p.streams[0].read.tolist() == w["l0.hc1.in"].float().tolist() and torch.equal(p.streams[1].mix, w["l0.hc2.mix"].float())
    assert p.gate_up.act_interleaved and p.gate_up.n == 160 and p.routed is None
    q = L.pack_layer(cfg, 1, w.__getitem__)
    bias, rel = q.mixer.bias, w["l1.mix.rel"].float()
    assert bias.shape == (31, 4) and all(torch.equal(bias[n], rel[R.distance_bucket(n, 8, 30)]) for n in range(31))
    r, head = q.routed, q.routed.head.codes.float()[:, :W]
    assert r.split == 16 and torch.equal(head[:8], w["l1.mlp.router"].float()) and torch.equal(head[8:9], w["l1.mlp.shared.sg"].float())
    assert torch.equal(head[16:80], w["l1.mlp.shared.up"].float()) and head.shape[0] == 80
    assert r.up.codes.shape == (5, 48, 128) and r.down.codes.shape == (5, 96, 64) and q.gate_up is None
    assert all(torch.equal(r.down.codes[e, :, :48].float(), w[f"l1.mlp.e{e}.down"].float()) for e in range(5))
    last = L.pack_layer(cfg, 2, w.__getitem__)
    assert last.norm2 is None and len(last.streams) == 1 and last.routed is None
    packed = L.pack_weights(cfg, w.__getitem__)
    assert torch.equal(packed.lm_head.codes.float()[:, :W], w["head"].float()) and packed.nbytes() > 0


def test_gated_packing():
    """Sections of the projection, where the absorbed queries are read, gate rows behind both products that read a norm."""
    from cubic_serve_b200.ops import wq_pack
    cfg, w = parsed("gat")
    W = cfg.hidden_size
    p = L.pack_layer(cfg, 0, w.__getitem__)
    m, rows = p.mixer, p.proj.codes.float()[:, :W]
    q = w["l0.mix.q"].float().view(5, 28, W)
    hp, kg = m.absorb.heads, m.absorb.w.k
    for h in range(5):
        c = m.q_off + h // hp * kg + h % hp * 16
        assert torch.equal(rows[c:c + 16], q[h, :16])
    assert torch.equal(rows[m.qr_off:m.qr_off + 60], q[:, 16:].reshape(60, W)) and m.qr_off >= -(-5 // hp) * kg
    down = w["l0.mix.dkv"].float()
    assert torch.equal(rows[m.c_off:m.c_off + 72], down[:72]) and torch.equal(rows[m.r_off:m.r_off + 12], down[72:])
    assert torch.equal(rows[p.rg_off:p.rg_off + W], w["l0.rg1"].float()) and p.split == p.proj.n
    assert all(o % 8 == 0 for o in (m.q_off, m.qr_off, m.c_off, m.r_off, p.rg_off))
    freq, mult = R.rotary_frequencies(cfg.to_config()["layers"][0]["mixer"]["rot"])
    assert (m.freq.double().sum(0) - freq).abs().max() < 1e-14 and m.rot_mult == mult
    assert m.absorb.w.n == 5 * 128 and (m.absorb.w.codes.float().view(5, 128, -1)[:, 72:] == 0).all()
    assert torch.equal(p.norm, w["l0.norm1"].float().expand(W)) and torch.equal(p.rg[1], w["l0.rg2.b"].float()) and p.limit == 1.2
    # a width of 80 features takes two tiles of the activation, the gate follows
    assert p.ff_rows == 256 and p.gate_up.n == 256 + W and p.gate_up.act_interleaved
    both = torch.zeros(256, W)
    both[:80], both[128:208] = w["l0.mlp.gate"].float(), w["l0.mlp.up"].float()
    codes = p.gate_up.codes.float()[:, :W]
    assert torch.equal(codes[:256], both[wq_pack.swiglu_row_order(128)]) and torch.equal(codes[256:], w["l0.rg2"].float())
    g = L.pack_layer(cfg, 1, w.__getitem__)
    rows = g.proj.codes.float()[:, :W]
    for t, off in zip("zxg", (g.mixer.z_off, g.mixer.x_off, g.mixer.g_off)):
        assert torch.equal(rows[off:off + 72], w[f"l1.mix.{t}"].float())
    assert torch.equal(g.mixer.bias, torch.stack([w["l1.mix.z.b"], w["l1.mix.x.b"]]).float())
    d = L.pack_layer(cfg, 2, w.__getitem__)
    rows = d.proj.codes.float()[:, :W]
    for t, off in zip("qkv", d.mixer.spec.offsets):
        t = w[f"l2.mix.{t}"].float()
        assert torch.equal(rows[d.mixer.q_off + off:d.mixer.q_off + off + t.shape[0]], t)
    assert torch.equal(rows[d.mixer.g_off:d.mixer.g_off + 240], w["l2.mix.g"].float())
    dots = [float((w[f"l2.mix.lq{i}"].double() * w[f"l2.mix.lk{i}"].double()).sum()) for i in (1, 2)]
    assert abs(d.mixer.less - (np.exp(dots[0]) - np.exp(dots[1]) + 0.4)) < 1e-12
    last = L.pack_layer(cfg, 3, w.__getitem__)
    assert last.gate_up is None and len(last.rg) == 1 and L.pack_weights(cfg, w.__getitem__).loop_in is None


@pytest.mark.parametrize("rows, most", [(2, 2), (2, 50), (3, 9), (8, 30), (9, 128), (11, 70), (16, 120), (16, 128), (32, 512), (33, 100)])
def test_distance_buckets(rows, most):
    """The product's table and the oracle's buckets: the formula wherever floating point decides it, every row up to the last."""
    half = rows // 2
    spec = L.BiasedAttentionSpec(1, 1, 8, 8, 1.0, rows, most)
    table = spec.bucket_of_distance().tolist()
    assert table == [R.distance_bucket(n, rows, most) for n in range(most + 1)]
    assert table[:half] == list(range(half)) and table[-1] == rows - 1 and sorted(table) == table
    assert R.distance_bucket(most * 7, rows, most) == rows - 1
    for n in range(half, most + 1):
        at = np.log(n / half) / np.log(most / half) * (rows - half)
        if abs(at - round(at)) > 1e-9:
            assert table[n] == min(rows - 1, half + int(np.floor(at)))
        else:
            assert table[n] == min(rows - 1, half + round(at))                          # a border is the next row's


# ------------------------------------------------------------------ the oracle's mechanisms, against element-wise loops
def test_oracle_chunks():
    for size in (1, 3, 4, None):
        seen = R.same_chunk(6, 5, 11, size)
        for i in range(5):
            for j in range(11):
                assert bool(seen[i, j]) == (j <= 6 + i and (size is None or j // size == (6 + i) // size))


def test_oracle_differential_attention():
    """Both maps, the factor, the norm without a weight and the gate, score by score."""
    raw = gated(30, 24, [differential(4, 2, 6, 5, 0.7, 4, 20.0, 0.3, 4, None)])
    w = {n: t.double() for n, t in tensors(raw, 1).items()}
    m, h, eps = raw["layers"][0]["mixer"], torch.randn(9, 24, dtype=torch.float64), 1e-3
    got = R.differential_attention(w, "l0.mix", m, h, {}, eps)
    q, k = ((h @ w[f"l0.mix.{t}"].T).view(9, -1, 2, 6) for t in "qk")
    q, k = (torch.stack([R.rotate_halves(R.rms(t[i:i + 1, :, j], eps) * w[f"l0.mix.{n}.norm"], i, 4, 20.0)[0] for i in range(9) for j in range(2)])
            .view(9, 2, -1, 6) for t, n in ((q, "q"), (k, "k")))
    v = (h @ w["l0.mix.v"].T).view(9, 2, 5)
    less = float(torch.exp(w["l0.mix.lq1"] @ w["l0.mix.lk1"]) - torch.exp(w["l0.mix.lq2"] @ w["l0.mix.lk2"]) + 0.3)
    out = torch.empty(9, 4, 5, dtype=torch.float64)
    for i in range(9):
        for n in range(4):
            maps = []
            for j in range(2):
                keys = range(i // 4 * 4, i + 1)
                e = np.exp([0.7 * float(q[i, j, n] @ k[t, j, n // 2]) for t in keys])
                maps.append(sum(a * v[t, n // 2] for a, t in zip(e / e.sum(), keys)))
            o = maps[0] - less * maps[1]
            out[i, n] = o / torch.sqrt((o * o).mean() + eps) * 0.7
    want = (out.view(9, 20) / (1 + torch.exp(-(h @ w["l0.mix.g"].T)))) @ w["l0.mix.o"].T
    assert torch.allclose(got, want, atol=1e-9)


def test_oracle_rotated_latent_attention():
    raw = gated(30, 24, [rotated(3, 6, 4, 5, 7, 0.6, 20.0, (2.0, 30, 4.0, 1.0), None)])
    w = {n: t.double() for n, t in tensors(raw, 2).items()}
    m, h, eps = raw["layers"][0]["mixer"], torch.randn(8, 24, dtype=torch.float64), 1e-3
    got = R.rotated_latent_attention(w, "l0.mix", m, h, {}, eps)
    freq, mult = R.rotary_frequencies(m["rot"])
    q, down = (h @ w["l0.mix.q"].T).view(8, 3, 10), h @ w["l0.mix.dkv"].T

    def turn(x, i):
        return R.rotate_pairs(x.view(1, 1, 4), i, freq, mult).view(4)

    c = [down[t, :7] / torch.sqrt((down[t, :7] ** 2).mean() + eps) * w["l0.mix.dkv.norm"] for t in range(8)]
    out = torch.empty(8, 3, 5, dtype=torch.float64)
    for i in range(8):
        for n in range(3):
            uk, uv = w["l0.mix.uk"].view(3, 6, 7)[n], w["l0.mix.uv"].view(3, 5, 7)[n]
            e = np.exp([0.6 * float(q[i, n, :6] @ (uk @ c[t]) + turn(q[i, n, 6:], i) @ turn(down[t, 7:], t)) for t in range(i + 1)])
            out[i, n] = sum(a * (uv @ c[t]) for t, a in enumerate(e / e.sum()))
    assert torch.allclose(got, out.view(8, 15) @ w["l0.mix.o"].T, atol=1e-9)


def test_oracle_elementwise_recurrence_and_clamped_feed_forward():
    raw = gated(30, 12, [mingru(5, clamped(6, 0.8))])
    w = {n: t.double() for n, t in tensors(raw, 3).items()}
    h = torch.randn(7, 12, dtype=torch.float64)
    st, S, sig = {}, np.zeros(5), lambda v: 1 / (1 + np.exp(-v))                        # noqa: E731
    got = torch.cat([R.mingru_mixer(w, "l0.mix", raw["layers"][0]["mixer"], part, st, 0.0) for part in h.split([2, 1, 4])])
    for t in range(7):
        z, x, g = ((w[f"l0.mix.{n}"] @ h[t]).numpy() for n in "zxg")
        z, x = z + w["l0.mix.z.b"].numpy(), x + w["l0.mix.x.b"].numpy()
        for c in range(5):
            S[c] = (1 - sig(z[c])) * S[c] + sig(z[c]) * (x[c] + 0.5 if x[c] >= 0 else sig(x[c]))
        assert torch.allclose(got[t], w["l0.mix.o"] @ torch.from_numpy(S * g * sig(g)), atol=1e-9)
    y = R.clamped_feed_forward(w, "l0.mlp", 3 * h, 0.8)
    for t in range(7):
        act = [min(a, 0.8) * sig(1.702 * min(a, 0.8)) * (max(-0.8, min(b, 0.8)) + 1)
               for a, b in zip((w["l0.mlp.gate"] @ (3 * h[t])).tolist(), (w["l0.mlp.up"] @ (3 * h[t])).tolist())]
        assert torch.allclose(y[t], w["l0.mlp.down"] @ torch.tensor(act, dtype=torch.float64), atol=1e-9)


def test_oracle_gated_residuals_and_the_loop():
    """A model of one looped recurrence, layer by layer: gates that read the normed input, the embedding added between passes."""
    raw = gated(30, 12, [mingru(5, clamped(6, 0.8))], (0, 1, 3), 0.4)
    w = tensors(raw, 4)
    got, _ = R.Oracle(raw, w, torch.float64).forward([3, 7, 7, 1])
    f = {n: t.double() for n, t in w.items()}
    m, eps = raw["layers"][0]["mixer"], 1e-5
    x0 = 0.4 * f["embed"][[3, 7, 7, 1]]
    x = x0
    for turn in range(3):
        if turn:
            x = x + x0
        for q, sub in ((1, lambda h: R.mingru_mixer(f, "l0.mix", m, h, {}, eps)), (2, lambda h: R.clamped_feed_forward(f, "l0.mlp", h, 0.8))):
            h = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * float(f[f"l0.norm{q}"])
            x = x + sub(h) / (1 + torch.exp(-(h @ f[f"l0.rg{q}"].T + f[f"l0.rg{q}.b"])))
    want = (x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * float(f["final.norm"])) @ f["head"].T
    assert torch.allclose(got, want, atol=1e-9)


def test_oracle_rotation_of_halves_and_kept_window():
    x = torch.randn(4, 2, 7, dtype=torch.float64)
    y = R.rotate_halves(x, 5, 6, 50.0)
    for t in range(4):
        for h in range(2):
            for i in range(3):
                a = (5 + t) * 50.0 ** (-2 * i / 6)
                u, v = float(x[t, h, i]), float(x[t, h, i + 3])
                assert abs(float(y[t, h, i]) - (u * np.cos(a) - v * np.sin(a))) < 1e-12
                assert abs(float(y[t, h, i + 3]) - (v * np.cos(a) + u * np.sin(a))) < 1e-12
    assert torch.equal(y[:, :, 6:], x[:, :, 6:]) and torch.equal(R.rotate_halves(x, 5, 0, 9.0), x)
    for size, keep in ((3, 2), (1, 0), (None, 0), (4, 20)):
        seen = R.kept_window(6, 5, 11, size, keep)
        for i in range(5):
            for j in range(11):
                p = 6 + i
                assert bool(seen[i, j]) == (j <= p and (size is None or p - j < size or j < keep))


def test_oracle_masked_attention_with_bias():
    q, k, v, b = torch.randn(5, 4, 3), torch.randn(5, 2, 3), torch.randn(5, 2, 6), torch.randn(4, 5, 5)
    seen = R.kept_window(0, 5, 5, 2, 1)
    o = R.masked_attention(q, k, v, seen, 0.8, b)
    for i in range(5):
        for h in range(4):
            js = [j for j in range(5) if j <= i and (i - j < 2 or j < 1)]
            e = [np.exp(0.8 * float(q[i, h] @ k[j, h // 2]) + float(b[h, i, j])) for j in js]
            assert torch.allclose(o[i, h], sum(w * v[j, h // 2] for w, j in zip(e, js)) / sum(e), atol=1e-5)


def test_oracle_routing():
    """Choice by score plus correction, weights by score alone, ties to the first; an expert that returns the token."""
    z, corr = torch.tensor([[1.0, 1.0, 0.0, 2.0], [0.0, 0.0, 0.0, 0.0]], dtype=torch.float64), torch.tensor([0.0, 0.0, 0.6, 0.0])
    chosen, weight = R.route(z, corr, 2)
    s = torch.exp(z[0]) / torch.exp(z[0]).sum()
    assert chosen.tolist() == [[2, 3], [2, 0]]
    assert torch.allclose(weight[0], s[[2, 3]] / s[[2, 3]].sum()) and torch.allclose(weight[1], torch.tensor([0.5, 0.5], dtype=torch.float64))
    w = {"p.router": torch.zeros(3, 4), "p.correction": torch.tensor([0.0, 0.2, 0.1]), "p.e0.up": torch.randn(5, 4), "p.e0.down": torch.randn(4, 5),
         "p.e1.up": torch.randn(5, 4), "p.e1.down": torch.randn(4, 5), "p.shared.up": torch.randn(3, 4), "p.shared.down": torch.randn(4, 3),
         "p.shared.sg": torch.randn(1, 4)}
    h = torch.randn(2, 4)
    out = R.routed_feed_forward(w, "p", routed(2, 2, 5, 1, 3), h)
    for t in range(2):
        e1 = w["p.e1.down"] @ (w["p.e1.up"] @ h[t]).clamp_min(0) ** 2
        sh = w["p.shared.down"] @ (w["p.shared.up"] @ h[t]).clamp_min(0) ** 2
        want = 0.5 * e1 + 0.5 * h[t] + sh / (1 + torch.exp(-(w["p.shared.sg"] @ h[t])))
        assert torch.allclose(out[t], want, atol=1e-5)


def test_oracle_streams():
    xs, w_in, mix, out, y = torch.randn(3, 2, 4), torch.randn(3), torch.randn(3, 3), torch.randn(3), torch.randn(2, 4)
    assert torch.allclose(R.stream_read(xs, w_in), sum(w_in[s] * xs[s] for s in range(3)), atol=1e-6)
    new = R.stream_write(xs, mix, out, y)
    for t in range(3):
        assert torch.allclose(new[t], sum(mix[s, t] * xs[s] for s in range(3)) + out[t] * y, atol=1e-6)


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_oracle_plain_convolution(taps):
    x, w = torch.randn(6, 3), torch.randn(3, taps)
    y, past = R.plain_short_conv(x, w, torch.zeros(taps - 1, 3))
    for t in range(6):
        assert torch.allclose(y[t], sum(w[:, taps - 1 - d] * x[t - d] for d in range(taps) if t - d >= 0), atol=1e-5)
    a, p1 = R.plain_short_conv(x[:1], w, torch.zeros(taps - 1, 3))
    b, p2 = R.plain_short_conv(x[1:], w, p1)
    assert torch.allclose(torch.cat([a, b]), y, atol=1e-6) and torch.equal(p2, past)


def test_oracle_query_factor():
    """The factor steps where the position after a token is a multiple of ``every``; a query scaled alone moves the weights."""
    raw = streams(30, 16, [far(1, 1, 8, 8, 2.0, 4, (0.7, 3), 0, 2)], 1)
    w = {n: t.double() for n, t in tensors(raw, 1).items()}
    m, h = raw["layers"][0]["mixer"], torch.randn(9, 16, dtype=torch.float64)
    got = R.biased_attention(w, "l0.mix", m, h, {}, 1e-5)
    q, k = (R.rms(h @ w[f"l0.mix.{t}"].T, 1e-5) * w[f"l0.mix.{t}.norm"] for t in "qk")
    v = h @ w["l0.mix.v"].T
    for i in range(9):
        f = 1 + 0.7 * np.log((i + 1) // 3 + 1)
        sc = [2.0 * f * float(q[i] @ k[j]) + float(w["l0.mix.rel"][min(i - j, 1), 0]) for j in range(i + 1)]
        e = np.exp(np.array(sc) - max(sc))
        assert torch.allclose(got[i], w["l0.mix.o"] @ sum(a * v[j] for j, a in enumerate(e / e.sum())), atol=1e-9)


def test_rotary_table_equals_the_oracle():
    """Frequencies of the product and of the oracle, stretched and plain; the ramp's ends, also where it has no width."""
    for raw in (*SEQUENTIAL.values(),):
        for l in raw["layers"]:
            if l["type"] == "parallel":
                rot = l["mixer"]["left"]["rot"]
                f, mult = L._read_rotary(rot).table()
                g, m2 = R.rotary_frequencies(rot)
                assert torch.allclose(f.double(), g, rtol=1e-7) and abs(mult - m2) < 1e-12
    for fast, slow in ((32, 1), (1, 1), (1000, 0.001), (0.01, 0.001), (5000, 4000)):
        rot = {"dims": 16, "base": 700.0, "scaling": {"factor": 5.0, "original": 90, "fast": fast, "slow": slow}}
        f, _ = L._read_rotary(rot).table()
        g, _ = R.rotary_frequencies(rot)
        assert torch.allclose(f.double(), g, rtol=1e-7), (fast, slow)
        plain = torch.tensor([700.0 ** (-i / 8) for i in range(8)], dtype=torch.float64)
        ratio = g / plain
        assert ((ratio <= 1 + 1e-12) & (ratio >= 0.2 - 1e-12)).all() and (ratio[1:] <= ratio[:-1] + 1e-12).all()


def test_oracle_rotation_and_sink():
    x = torch.randn(4, 2, 7, dtype=torch.float64)
    freq = torch.tensor([0.9, 0.05], dtype=torch.float64)
    y = R.rotate_pairs(x, 5, freq, 1.3)
    for t in range(4):
        for h in range(2):
            for i in range(2):
                a = (5 + t) * float(freq[i])
                u, v = float(x[t, h, 2 * i]), float(x[t, h, 2 * i + 1])
                assert abs(float(y[t, h, 2 * i]) - 1.3 * (u * np.cos(a) - v * np.sin(a))) < 1e-12
                assert abs(float(y[t, h, 2 * i + 1]) - 1.3 * (v * np.cos(a) + u * np.sin(a))) < 1e-12
    assert torch.equal(y[:, :, 4:], x[:, :, 4:])
    q, k, v = torch.randn(6, 4, 3), torch.randn(6, 2, 3), torch.randn(6, 2, 5)
    o = R.sink_attention(q, k, v, 0, 3, 0.8)
    for i in range(6):
        for h in range(4):
            js = [j for j in range(6) if 0 <= i - j < 3]
            e = [np.exp(0.8 * float(q[i, h] @ k[j, h // 2])) for j in js]
            want = sum(w * v[j, h // 2] for w, j in zip(e, js)) / (1 + sum(e))
            assert torch.allclose(o[i, h], want, atol=1e-5)


def test_oracle_linear_step_and_parts_norm():
    H, d, e = 2, 3, 4
    S, q, k, v, decay = torch.randn(H, d, e), torch.randn(H, d), torch.randn(H, d), torch.randn(H, e), torch.rand(H, d)
    o, S2 = R.linear_step(S, q, k, v, decay)
    for h in range(H):
        for j in range(e):
            col = [float(decay[h, i] * S[h, i, j] + k[h, i] * v[h, j]) for i in range(d)]
            assert np.allclose(col, S2[h, :, j].numpy(), atol=1e-5)
            assert abs(sum(c * float(q[h, i]) for i, c in enumerate(col)) - float(o[h, j])) < 1e-5
    y, z, w = torch.randn(2, 6, dtype=torch.float64), torch.randn(2, 6, dtype=torch.float64), torch.randn(6, dtype=torch.float64)
    out = R.gated_parts_norm(y, z, w, 3, 0.01)
    for t in range(2):
        u = [float(y[t, c] * z[t, c]) / (1 + np.exp(-float(z[t, c]))) for c in range(6)]
        for c in range(6):
            part = u[c // 2 * 2:c // 2 * 2 + 2]
            assert abs(float(out[t, c]) - u[c] / (sum(p * p for p in part) / 2 + 0.01) ** 0.5 * float(w[c])) < 1e-9
    x = torch.linspace(-4, 4, 9, dtype=torch.float64)
    assert torch.allclose(R.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))


def test_oracle_convolution_bias():
    x, w, b = torch.randn(5, 3), torch.randn(3, 2), torch.randn(3)
    y, past = R.short_conv(x, w, torch.zeros(1, 3), b)
    for t in range(5):
        s = b + w[:, 1] * x[t] + (w[:, 0] * x[t - 1] if t else 0)
        assert torch.allclose(y[t], s / (1 + torch.exp(-s)), atol=1e-6)
    assert torch.equal(past, x[4:])


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


def _swapped(name, change):
    """A mistake planted in one of the oracle's functions."""
    right = getattr(R, name)

    def plant(monkeypatch):
        wrong = lambda *a: change(right, *a)                                            # noqa: E731
        monkeypatch.setattr(R, name, wrong)
        for kind, fn in R.GATED_MIXERS.items():
            if fn is right:
                monkeypatch.setitem(R.GATED_MIXERS, kind, wrong)
    return plant


def _first_turned(x, first, freq, mult):
    return x if x.shape[1] == 1 else RIGHT_ROTATE(x, first, freq, mult)


RIGHT_ROTATE = R.rotate_pairs


@pytest.mark.parametrize("mistake", [
    _swapped("same_chunk", lambda f, a, n, m, size: f(a, n, m, size and size + 1)),
    _swapped("same_chunk", lambda f, a, n, m, size: f(a, n, m, None)),
    _swapped("same_chunk", lambda f, a, n, m, size: R.kept_window(a, n, m, size, 0)),
    _swapped("rotary_frequencies", lambda f, rot: (f(rot)[0], 1.0)),
    _swapped("rotary_frequencies", lambda f, rot: f({**rot, "scaling": None})),
    _swapped("rotate_pairs", lambda f, x, a, fr, mult: _first_turned(x, a, fr, mult)),
    _swapped("rotate_halves", lambda f, x, a, dims, base: f(x, a, dims, 1.02 * base)),
    _swapped("rotate_halves", lambda f, x, a, dims, base: f(x, a + 1, dims, base) if x.shape[1] == 12 else f(x, a, dims, base)),
    _swapped("clamped_feed_forward", lambda f, w, p, h, limit: f(w, p, h, 1.01 * limit)),
    _swapped("mingru_mixer", lambda f, w, p, m, h, st, eps: f(w, p, m, h, {}, eps) if h.shape[0] == 40 else f(w, p, m, h, st, eps)),
    _swapped("differential_attention", lambda f, w, p, m, h, st, eps: f(w, p, {**m, "diff": m["diff"] + 1e-3}, h, st, eps)),
    _swapped("layer_schedule", lambda f, cfg: [(i, False) for i, _ in f(cfg)]),
], ids=["chunk + 1", "no chunk", "window", "factor", "stretch", "shared key", "base", "query position", "limit", "lost state", "constant", "entry"])
def test_mistakes_show_in_the_logits(monkeypatch, mistake):
    """What the comparisons with the oracle allow in 32-bit is far below what a mistake in one mechanism changes."""
    raw = GATED["gat"]
    w, ids = tensors(raw, 1), prompt(raw, 90, 4)

    def logits():
        o, st, out = R.Oracle(raw, w, torch.float64), None, []
        for part in (ids[:50], ids[50:]):
            lg, st = o.forward(part, st)
            out.append(lg)
        return torch.cat(out)

    right = logits()
    mistake(monkeypatch)
    err = (logits() - right).pow(2).mean(-1).sqrt() / right.pow(2).mean(-1).sqrt()
    assert (err > 10 * 2e-5).sum() > 3, float(err.max())


@pytest.mark.parametrize("name", list(ALL))
def test_oracle_portions_equal_one_pass(name):
    o = R.Oracle(ALL[name], tensors(ALL[name]), torch.float64)
    ids = prompt(ALL[name], 61, 0)
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


@pytest.mark.parametrize("raw", [
    config(300, 64, [delta(2, 1, 16, 16, 3, 64), latent(2, 16, 16, 24, 32, 20, 0.25, 0), channel(2, 2, 16, 16, 2, 48)], (0, 2, 2)),
    sequential(300, 64, [mamba2(2, 16, 8, 1, 3, 2, 48), parallel((4, 2, 16, 20, 0.3, 8, 90.0, (2.0, 50, 4.0, 1.0)), (2, 12, 16, 8.0), (0.9, 0.8), 64)], 8),
    streams(300, 64, [near(4, 2, 16, 24, 3, 0.5, 8, 90.0, 20, 3, routed(4, 2, 32, 1, 24)), far(2, 1, 16, 16, 0.3, 20, (0.4, 8), 48)], 2, 3.0),
    gated(300, 64, [rotated(2, 16, 8, 16, 32, 0.3, 90.0, (2.0, 50, 4.0, 1.0), clamped(64)), mingru(48, None),
                    differential(4, 2, 16, 24, 0.3, 8, 90.0, 0.4, 20, clamped(48))], (1, 3, 2), 0.5),
], ids=["Bumodra", "Loduzen", "Vimelorn", "Fovunex"])
def test_eager_mode_generates_like_the_oracle(tmp_path, raw):
    from cubic_serve_b200.runtime.scheduler import SamplingParams
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
