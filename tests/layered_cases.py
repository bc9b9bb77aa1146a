"""Configurations and weights of the layered-decoder tests: raw ``config.json`` dictionaries and seeded tensors, made here
without the product's own helpers."""
from __future__ import annotations

import math

import torch


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def channel(heads, kv_heads, dim, vdim, conv, ff):
    return {**delta(heads, kv_heads, dim, vdim, conv, ff), "type": "channel_delta"}


def latent(heads, dim, vdim, q_rank, kv_rank, size, scale, ff):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": size} if size else None},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(vocab, width, layers, loop=None, eps=1e-5):
    return {"architecture": "Bumodra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


CASES = {
    # every mixer, a loop in the middle, a layer without a feed-forward
    "all": config(200, 96, [delta(4, 2, 24, 40, 4, 96), latent(5, 16, 24, 40, 48, 19, 0.3, 72), channel(3, 3, 32, 16, 2, 0),
                            latent(2, 32, 16, 32, 64, 33, 0.2, 64)], (1, 3, 2), 1e-6),
    # no loop; one head; equal and unit sizes; a single tap; a window of one token
    "small": config(70, 64, [latent(1, 16, 16, 16, 16, 1, 0.25, 64), delta(1, 1, 16, 16, 1, 64), channel(2, 1, 8, 12, 3, 48)],
                    None, 1e-5),
    # odd widths, many taps, the whole model looped three times, full attention
    "odd": config(123, 68, [channel(2, 2, 7, 9, 5, 44), delta(6, 3, 20, 13, 3, 36), latent(3, 12, 20, 24, 20, 0, 0.35, 40)],
                  (0, 3, 3), 1e-4),
    # wide heads, a loop that runs once, many heads of attention, window over several pages
    "wide": config(256, 128, [delta(2, 1, 128, 144, 4, 128), latent(40, 8, 8, 64, 136, 50, 0.35, 0),
                              channel(2, 1, 160, 64, 4, 96)], (2, 3, 1), 1e-6),
}


# ------------------------------------------------------------------ sequential layers (Loduzen)
def parallel(left, right, scales, ff):
    """``left``: (heads, kv heads, dim, window, scale, rotary dims, base, yarn (factor, original, fast, slow) or None);
    ``right``: (heads, dim, vdim, tau)."""
    H, G, d, size, scale, dims, base, yarn = left
    rot = {"dims": dims, "base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None}
    return {"type": "parallel",
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": scale, "rot": rot,
                               "mask": {"size": size} if size else None},
                      "right": dict(zip(("heads", "dim", "vdim", "tau"), right)),
                      "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba2(heads, vdim, state, groups, conv, norm_groups, ff):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def sequential(vocab, width, layers, side=0, eps=1e-5):
    return {"architecture": "Loduzen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "token_side": {"dim": side} if side else None}


SEQUENTIAL = {
    # both mixers, grouped heads, stretched rotary pairs, parts of the norm, a layer without a feed-forward
    "seq": sequential(210, 96, [parallel((6, 2, 24, 21, 0.3, 12, 1000.0, (3.0, 40, 4.0, 0.5)), (3, 20, 28, 8.0), (0.7, 1.3), 80),
                                mamba2(4, 24, 20, 2, 4, 3, 96),
                                parallel((4, 4, 32, 40, 0.25, 32, 5000.0, (2.0, 64, 8.0, 1.0)), (2, 32, 16, 16.0), (1.1, 0.6), 0),
                                mamba2(2, 40, 16, 1, 3, 1, 64)], 12, 1e-6),
    # single heads, a window of one token, one tap, no side input, plain rotation
    "seq_small": sequential(71, 64, [mamba2(1, 16, 16, 1, 1, 1, 48),
                                     parallel((1, 1, 16, 1, 0.25, 16, 100.0, None), (1, 16, 16, 1.0), (1.0, 1.0), 64)]),
    # odd widths, many taps, three query heads per key head, every earlier token, no rotated channel in one layer
    "seq_odd": sequential(123, 68, [parallel((9, 3, 13, 0, 0.4, 6, 50.0, (4.0, 30, 2.0, 1.0)), (2, 7, 9, 3.0), (0.5, 1.5), 44),
                                    mamba2(6, 5, 7, 3, 6, 5, 36),
                                    parallel((5, 1, 18, 33, 0.3, 0, 10.0, None), (3, 10, 12, 5.0), (1.2, 0.8), 20)], 5, 1e-4),
    # wide heads, more query heads than a block has rows, windows over several pages
    "seq_wide": sequential(256, 128, [parallel((40, 1, 72, 50, 0.15, 64, 10000.0, (8.0, 100, 32.0, 1.0)), (1, 144, 72, 16.0), (0.9, 1.2), 0),
                                      mamba2(4, 130, 136, 1, 4, 4, 128),
                                      parallel((3, 1, 200, 19, 0.1, 40, 300.0, None), (2, 96, 200, 4.0), (1.0, 0.5), 96)], 40),
}


# ------------------------------------------------------------------ several residual streams (Vimelorn)
def ff_of(mlp):
    """``mlp``: width of a dense feed-forward, 0 for none, or ``routed(...)``."""
    return mlp if isinstance(mlp, dict) else {"kind": "dense", "ff": mlp} if mlp else None


def routed(experts, top, ff, identity=0, shared=0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top},
            "shared": {"ff": shared} if shared else None}


def near(heads, kv_heads, dim, vdim, conv, scale, dims, base, size, keep, mlp):
    """Convolved attention with rotary halves; ``size`` 0: no window."""
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
                      "rot": {"dims": dims, "base": base}, "mask": {"size": size, "keep_first": keep} if size else None},
            "mlp": ff_of(mlp)}


def far(heads, kv_heads, dim, vdim, scale, bias_max, temp, mlp, rows=8):
    """Attention with a bias by distance (a table of ``rows`` rows); ``temp``: (coef, every) or None."""
    return {"type": "attention_2", "rows": rows,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
                      "q_temp": dict(zip(("coef", "every"), temp)) if temp else None},
            "mlp": ff_of(mlp)}


class StreamConfig(dict):
    """A configuration with the rows of its layers' bias tables, which only the tensors state."""
    bias_rows: list[int]
    close_calls = False          # the choice of experts may hang on rounding


def streams(vocab, width, layers, count, scale=1.0, eps=1e-5, close_calls=False):
    rows = [l.pop("rows", 0) for l in layers]
    cfg = StreamConfig(architecture="Vimelorn", vocab=vocab, width=width, layers=layers, norm={"eps": eps}, streams=count,
                       embedding={"scale": scale})
    cfg.bias_rows, cfg.close_calls = rows, close_calls
    return cfg


STREAMS = {
    # both attentions and both feed-forwards, grouped heads, key and value widths that differ, a layer without a feed-forward
    "str": streams(210, 96, [near(6, 2, 24, 40, 3, 0.5, 12, 1000.0, 21, 5, 80), far(4, 2, 20, 28, 0.3, 30, (0.5, 16), routed(5, 3, 48, 3, 64)),
                             near(4, 4, 32, 16, 2, 0.4, 32, 5000.0, 40, 18, 0), far(2, 1, 32, 32, 0.25, 70, None, routed(7, 2, 40), 11),
                             near(3, 1, 16, 24, 4, 0.5, 8, 100.0, 17, 0, routed(3, 2, 56, 1, 32))], 2, 9.5, 1e-6),
    # one stream, single heads, a window of one token, one tap, no rotated channel, the smallest table, a single expert
    "str_small": streams(71, 64, [near(1, 1, 16, 16, 1, 0.5, 0, 10.0, 1, 0, routed(1, 1, 32)),
                                  far(1, 1, 16, 16, 0.25, 2, (1.0, 1), 48, 2), near(2, 1, 16, 16, 1, 0.4, 16, 100.0, 1, 1, routed(2, 1, 16, 1, 16))], 1),
    # a choice of experts per token
    "str_select": streams(150, 64, [near(4, 2, 16, 16, 3, 0.5, 16, 200.0, 30, 4, routed(9, 3, 32, 3, 32)), far(2, 2, 16, 16, 0.3, 40, (0.3, 20), routed(6, 2, 24, 2), 10),
                                    near(4, 1, 16, 24, 2, 0.4, 8, 200.0, 25, 2, routed(16, 4, 16, 0, 16))], 2, 2.0, close_calls=True),
    # odd widths, more taps than the unrolled forms have, three query heads per key head, every earlier token, three streams
    "str_odd": streams(123, 68, [near(9, 3, 13, 9, 6, 0.6, 6, 50.0, 0, 0, 44), far(6, 2, 7, 13, 0.5, 25, (0.2, 7), routed(4, 4, 20, 2, 36), 9),
                                 near(5, 1, 18, 21, 7, 0.5, 10, 300.0, 33, 7, routed(6, 5, 12, 4))], 3, 2.5, 1e-4),
    # wide heads, more query heads than a block has rows, kept tokens over several pages, many experts, four streams
    "str_wide": streams(256, 128, [near(40, 1, 72, 136, 4, 0.2, 64, 10000.0, 50, 35, routed(40, 6, 64, 9, 128)),
                                   far(20, 1, 200, 64, 0.1, 60, (0.3, 30), 96, 16), near(3, 1, 200, 256, 3, 0.1, 40, 300.0, 19, 65, 0)], 4, 3.0),
}


# ------------------------------------------------------------------ gated residuals (Fovunex)
def clamped(ff, limit=2.0):
    return {"kind": "dense", "ff": ff, "limit": limit} if ff else None


def rotated(heads, dim, rot_dim, vdim, kv_rank, scale, base, yarn, mlp):
    """Latent attention with a rotated key part; ``yarn``: (factor, original, fast, slow) or None."""
    rot = {"dims": rot_dim, "base": base}
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": rot}, "mlp": mlp}


def differential(heads, kv_heads, dim, vdim, scale, dims, base, diff, size, mlp):
    """``size`` 0: every earlier token."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff,
                                           "rot": {"dims": dims, "base": base}, "mask": {"size": size} if size else None}, "mlp": mlp}


def mingru(width, mlp):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def gated(vocab, width, layers, loop=None, scale=1.0, eps=1e-5):
    return {"architecture": "Fovunex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


GATED = {
    # every mixer, a loop in the middle, grouped heads, stretched pairs, a layer without a feed-forward
    "gat": gated(210, 96, [rotated(5, 16, 12, 40, 72, 0.3, 1000.0, (3.0, 40, 4.0, 0.5), clamped(80, 1.2)), mingru(72, clamped(96, 3.0)),
                           differential(6, 2, 24, 40, 0.3, 12, 5000.0, 0.4, 37, clamped(72)), mingru(130, None),
                           rotated(3, 24, 8, 16, 40, 0.25, 300.0, None, None)], (1, 3, 2), 0.7, 1e-6),
    # single heads, unit sizes, a chunk of one token, a loop that runs once from the first layer on
    "gat_small": gated(71, 64, [differential(1, 1, 16, 16, 0.25, 16, 100.0, 0.2, 1, clamped(48)), rotated(1, 16, 2, 16, 16, 0.25, 50.0, None, clamped(64, 0.5)),
                                mingru(16, None)], (0, 2, 1)),
    # odd widths, three query heads per key head, few rotated channels, every earlier token, the whole model looped three times
    "gat_odd": gated(123, 68, [differential(9, 3, 13, 9, 0.5, 6, 50.0, 0.7, 0, clamped(44)), rotated(3, 20, 6, 13, 19, 0.35, 80.0, (4.0, 30, 2.0, 1.0), clamped(36, 0.8)),
                               mingru(37, clamped(20)), differential(4, 1, 7, 21, 0.6, 0, 10.0, 0.1, 33, None)], (0, 4, 3), 2.5, 1e-4),
    # wide heads, more query heads than a block has rows, latents of several widths, chunks over several pages
    "gat_wide": gated(256, 128, [differential(40, 1, 72, 136, 0.15, 64, 10000.0, 0.5, 50, clamped(128)), rotated(40, 24, 64, 16, 512, 0.1, 10000.0, (8.0, 100, 32.0, 1.0), None),
                                 rotated(2, 32, 100, 40, 500, 0.1, 500.0, None, clamped(96)), mingru(300, None),
                                 differential(3, 3, 100, 250, 0.1, 40, 300.0, 0.3, 19, clamped(64))], (2, 4, 2), 3.0),
    # a latent beside a rotated part that adds a group of columns, and one that fits in
    "gat_latent": gated(150, 64, [rotated(4, 16, 32, 24, 120, 0.2, 700.0, None, clamped(40)), rotated(33, 8, 40, 8, 250, 0.2, 90.0, (2.0, 64, 8.0, 1.0), None),
                                  rotated(6, 48, 16, 8, 44, 0.2, 2000.0, None, clamped(32))], None, 1.5),
}
ALL = {**CASES, **SEQUENTIAL, **STREAMS, **GATED}
LOW_RANKS = (12, 20)          # inner sizes of the low-rank decay and gate projections


def tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        out[name] = (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, mean=0.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    mat("embed", cfg["vocab"], W, math.sqrt(W))
    if cfg["architecture"] == "Loduzen":
        _sequential_tensors(cfg, mat, vec)
        return out
    if cfg["architecture"] == "Vimelorn":
        _stream_tensors(cfg, mat, vec, out, g)
        return out
    if cfg["architecture"] == "Fovunex":
        _gated_tensors(cfg, mat, vec, out, g)
        return out
    vec("embed.norm", W)
    vec("final.norm", W)
    mat("head", cfg["vocab"], W)
    if cfg["loop"]:
        mat("loop.in", W, 2 * W)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        vec(f"l{i}.norm1", W)
        H, e = m["heads"], m["vdim"]
        if l["type"] == "latent_attention":
            mat(f"{p}.dq", m["q_rank"], W)
            vec(f"{p}.dq.norm", m["q_rank"], 1.0)
            mat(f"{p}.uq", H * m["dim"], m["q_rank"], 2.0)
            mat(f"{p}.dkv", m["kv_rank"], W)
            vec(f"{p}.dkv.norm", m["kv_rank"], 1.0)
            mat(f"{p}.uk", H * m["dim"], m["kv_rank"], 2.0)
            mat(f"{p}.uv", H * e, m["kv_rank"])
            mat(f"{p}.g", H, W)
        else:
            for t, c in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", H * e)):
                mat(f"{p}.{t}", c, W)
                mat(f"{p}.{t}.conv", c, m["conv"])
            mat(f"{p}.b", H, W)
            vec(f"{p}.A_log", H, -1.5, 0.5)
            vec(f"{p}.norm", e, 1.0)
            if l["type"] == "channel_delta":
                ra, rg = LOW_RANKS
                mat(f"{p}.a1", ra, W)
                mat(f"{p}.a2", H * m["dim"], ra)
                vec(f"{p}.dt_bias", H * m["dim"], 0.0, 0.5)
                mat(f"{p}.g1", rg, W)
                mat(f"{p}.g2", H * e, rg)
            else:
                mat(f"{p}.a", H, W)
                vec(f"{p}.dt_bias", H, 0.0, 0.5)
                mat(f"{p}.g", H * e, W)
        mat(f"{p}.o", W, H * e)
        if l["mlp"]:
            mat(f"l{i}.mlp.up", l["mlp"]["ff"], W)
            mat(f"l{i}.mlp.down", W, l["mlp"]["ff"])
    return out


def _sequential_tensors(cfg: dict, mat, vec) -> None:
    W = cfg["width"]
    side = (cfg["token_side"] or {}).get("dim", 0)
    vec("final.norm", W, 1.0)
    if side:
        mat("side.embed", cfg["vocab"], len(cfg["layers"]) * side, math.sqrt(len(cfg["layers"]) * side))
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        vec(f"l{i}.norm1", W, 1.0)
        if l["type"] == "mamba2":
            H, inner = m["heads"], m["heads"] * m["vdim"]
            C = inner + 2 * m["groups"] * m["state"]
            mat(f"{p}.in", inner + C + H, W)
            mat(f"{p}.conv", C, m["conv"], 1.5)
            vec(f"{p}.conv.b", C, 0.1, 0.3)
            vec(f"{p}.dt_bias", H, -1.0, 0.7)
            vec(f"{p}.A_log", H, -1.0, 0.7)
            vec(f"{p}.D", H, 0.5, 0.5)
            vec(f"{p}.norm", inner, 1.0)
            mat(f"{p}.o", W, inner)
        else:
            a, g = m["left"], m["right"]
            for t, n in (("q", a["heads"]), ("k", a["kv_heads"])):
                mat(f"{p}.left.{t}", n * a["dim"], W)
                vec(f"{p}.left.{t}.norm", a["dim"], 1.0, 0.3)
            mat(f"{p}.left.o", W, a["heads"] * a["dim"])
            H, d, e = g["heads"], g["dim"], g["vdim"]
            for t, n in (("q", d), ("k", d), ("v", e), ("g", e)):
                mat(f"{p}.right.{t}", H * n, W)
            mat(f"{p}.right.o", W, H * e)
            vec(f"{p}.right.norm", e, 1.0)
            mat(f"{p}.right.a1", LOW_RANKS[0], W)
            mat(f"{p}.right.a2", H * d, LOW_RANKS[0], 1.5)
            vec(f"{p}.right.a2.b", H * d, 1.0, 0.5)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            vec(f"l{i}.norm2", W, 1.0)
            mat(f"l{i}.mlp.gate", ff, W)
            mat(f"l{i}.mlp.up", ff, W)
            mat(f"l{i}.mlp.down", W, ff)
        if side:
            mat(f"l{i}.side.gate", side, W)
            mat(f"l{i}.side.proj", W, side)
            vec(f"l{i}.side.norm", W, 0.3, 0.1)


def _stream_tensors(cfg: dict, mat, vec, out: dict, g) -> None:
    W, S = cfg["width"], cfg["streams"]
    rows = cfg.bias_rows
    out["embed"] = (out["embed"].float() / cfg["embedding"]["scale"]).to(torch.bfloat16)
    vec("final.norm", W, 1.0)
    mat("head", cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        m, p, mlp = l["mixer"], f"l{i}.mix", l["mlp"]
        vec(f"l{i}.norm1", W, 1.0)
        sizes = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        for t, n in sizes.items():
            mat(f"{p}.{t}", n, W)
            if l["type"] == "attention":
                mat(f"{p}.{t}.conv", n, m["conv"])
            elif t != "v":
                vec(f"{p}.{t}.norm", n, 1.0, 0.3)
        if l["type"] == "attention_2":
            out[f"{p}.rel"] = torch.randn(rows[i], m["heads"], generator=g).to(torch.bfloat16)
        mat(f"{p}.o", W, m["heads"] * m["vdim"])
        for q in (1, 2) if mlp else (1,):
            vec(f"l{i}.hc{q}.in", S, 1.0 / S, 0.2)
            vec(f"l{i}.hc{q}.out", S, 1.0, 0.3)
            out[f"l{i}.hc{q}.mix"] = (torch.eye(S) + 0.15 * torch.randn(S, S, generator=g)).to(torch.bfloat16)
        if not mlp:
            continue
        p = f"l{i}.mlp"
        vec(f"l{i}.norm2", W, 1.0)
        if mlp["kind"] == "dense":
            for t in ("gate", "up"):
                mat(f"{p}.{t}", mlp["ff"], W)
            mat(f"{p}.down", W, mlp["ff"])
            continue
        r = mlp["router"]
        n = r["experts"] + r["identity"]
        for e in range(r["experts"]):
            mat(f"{p}.e{e}.up", mlp["expert"]["ff"], W)
            mat(f"{p}.e{e}.down", W, mlp["expert"]["ff"])
        # corrections farther apart than any two scores: the choice of a token's experts does not hang on rounding, their weights
        # follow the scores; or close together: every token has experts of its own, and some tokens a close call
        mat(f"{p}.router", n, W, 3.0)
        out[f"{p}.correction"] = ((0.3 / n if cfg.close_calls else 1.5) * torch.randperm(n, generator=g)).to(torch.bfloat16)
        if mlp["shared"]:
            mat(f"{p}.shared.up", mlp["shared"]["ff"], W)
            mat(f"{p}.shared.down", W, mlp["shared"]["ff"])
            mat(f"{p}.shared.sg", 1, W)


def _gated_tensors(cfg: dict, mat, vec, out: dict, g) -> None:
    W = cfg["width"]

    def one(name):
        out[name] = (1.0 + 0.3 * torch.randn((), generator=g)).to(torch.bfloat16)

    out["embed"] = (out["embed"].float() / cfg["embedding"]["scale"]).to(torch.bfloat16)
    one("final.norm")
    mat("head", cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        m, p, mlp = l["mixer"], f"l{i}.mix", l["mlp"]
        for q in (1, 2) if mlp else (1,):
            one(f"l{i}.norm{q}")
            mat(f"l{i}.rg{q}", W, W, 1.5)
            vec(f"l{i}.rg{q}.b", W, 0.3, 0.7)
        if l["type"] == "latent_attention":
            H, R = m["heads"], m["kv_rank"]
            mat(f"{p}.q", H * (m["dim"] + m["rot_dim"]), W, 2.0)
            mat(f"{p}.dkv", R + m["rot_dim"], W, 2.0)
            vec(f"{p}.dkv.norm", R, 1.0, 0.3)
            mat(f"{p}.uk", H * m["dim"], R, 2.0)
            mat(f"{p}.uv", H * m["vdim"], R)
            mat(f"{p}.o", W, H * m["vdim"])
        elif l["type"] == "attention":
            d = m["dim"]
            for t, n in (("q", m["heads"] * 2 * d), ("k", m["kv_heads"] * 2 * d), ("v", m["kv_heads"] * m["vdim"]), ("g", m["heads"] * m["vdim"])):
                mat(f"{p}.{t}", n, W)
            for t in ("q", "k"):
                vec(f"{p}.{t}.norm", d, 1.2, 0.4)
            for t in ("lq1", "lk1", "lq2", "lk2"):
                vec(f"{p}.{t}", d, 0.0, 0.7 / d ** 0.25)
            mat(f"{p}.o", W, m["heads"] * m["vdim"])
        else:
            for t in "zxg":
                mat(f"{p}.{t}", m["width"], W)
            vec(f"{p}.z.b", m["width"], -2.0, 1.0)
            vec(f"{p}.x.b", m["width"], 0.0, 0.5)
            mat(f"{p}.o", W, m["width"])
        if mlp:
            for t in ("gate", "up"):
                mat(f"l{i}.mlp.{t}", mlp["ff"], W, 1.5)
            mat(f"l{i}.mlp.down", W, mlp["ff"])


def write(path, cfg: dict, weights: dict[str, torch.Tensor]):
    import json

    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    save_file(weights, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(cfg))
    return path


def prompt(cfg: dict, n: int, seed: int) -> list[int]:
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
