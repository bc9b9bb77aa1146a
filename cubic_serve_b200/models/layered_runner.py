"""Layered decoders on the native sm_100a kernels.

``LayeredRunner`` is the model body of ``models/layered.py`` checkpoints: it owns the packed weights, fixed-address
buffers, one paged cache per attention run and the per-request state of every recurrent run, and serves the executor
through the same surface as ``DecoderRunner`` (``forward_hidden`` / ``forward_logits`` / ``run_step``, all capturable in a
CUDA graph).  A run of a parallel layer is

    norm(x) -> h                          fp32 residual in, activation type out
    [mixer inputs | relu^2(up)] = h W     one product; the up columns leave as the right half of the output's operand
    mixer -> left half of that operand
    x += [o | relu^2(up)] [W_o | W_down]  one product, accumulated into the fp32 residual

and a sequential layer, whose h comes from the step before it,

    mixer inputs = h W;  mixer -> operand;  x += operand W_o
    norm2(x) -> h;  act = gelu(h W_gate) (h W_up), one product;  x += act W_down
    side = gelu(x W_side) e, one kernel;  y = side W_proj;  x += norm(y) and h = norm1 of the next layer, one kernel

with gated residuals the matrices that read a norm also make the logits of the gate, which the products that join the residual
take in their epilogue (and the feed-forward's product is [act | gate] = h [W_gate, W_up ; W_rg]),

    x += sigmoid(gate) (operand W_o);  x += sigmoid(gate) (act W_down)

and a pass of a loop that adds the embedding output starts with x += scale E and h = norm1 of its first layer, one kernel.  A layer on
several residual streams x_s, whose h is the norm of their weighted sum, runs

    mixer inputs = h W;  mixer -> operand;  y = operand W_o
    x_t <- sum_s mix[s, t] x_s + out[t] y and h = norm2 of the next weighted sum, one kernel
    dense:   act = silu(h W_gate) (h W_up), one product;  y = act W_down
    routed:  [router, gate | relu^2(shared up)] = h W, one product;  routes, rows to their experts
             relu^2(rows W_up), rows W_down, one product each over all experts;  y = shared W_down
    the same kernel as above puts a routed y together from the places of the token's routes

``cfg.dtype`` "float32" runs the same steps with fp32 activations and fp32 products.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from .layered import (AttentionWeights, BiasedAttentionWeights, ConvAttentionWeights, DeltaWeights, DifferentialWeights,
                      GatedLinearWeights, LatentWeights, LayeredConfig, LayeredWeights, MinGruWeights, PairWeights, RoutedWeights,
                      SsdWeights, round_up)
from .step_runner import StepRunner


_PAGED = (AttentionWeights, ConvAttentionWeights, BiasedAttentionWeights, DifferentialWeights)      # keys and values in pages


class _StateRun:
    """Per-request state of one run of a layer: recurrence state (fp32; none with ``heads`` 0) and, with a convolution, its last
    inputs (activation type)."""

    def __init__(self, rows: int, heads: int, vdim: int, stride: int, device, taps: int = 0, conv_width: int = 0,
                 act: torch.dtype = torch.bfloat16) -> None:
        # a row is a multiple of 16 bytes (whole-row copies); the history's layout inside it is [taps - 1, channels]
        self.conv = torch.zeros(rows, max(1, taps - 1), conv_width, dtype=act, device=device) if taps else None
        self.state = torch.zeros(rows, heads, vdim, stride, dtype=torch.float32, device=device) if heads else None

    def copy(self, src, dst) -> None:
        if self.conv is not None:
            K.copy_rows(self.conv, src, dst)
        if self.state is not None:
            K.copy_rows(self.state, src, dst)


def _parts(m) -> tuple:
    """The mixers a layer's weights consist of."""
    return (m.left, m.right) if isinstance(m, PairWeights) else (m,)


class LayeredRunner(StepRunner):
    def __init__(self, cfg: LayeredConfig, weights: LayeredWeights, num_pages: int, max_tokens: int, device=None,
                 max_requests: int = 256, state_checkpoints: int = 0) -> None:
        """``max_requests``: request slots (rows of the recurrent state and of the page table); ``state_checkpoints``: further
        state rows for snapshots at page boundaries of prompts (prefix cache)."""
        self.cfg, self.w = cfg, weights
        self.device = dev = device or weights.embed.device
        self.tp_size = 1
        self.hq = self.hkv = 1                 # the batch builder's row blocks are not used: kernels read the segments
        self.max_tokens, self.num_pages, self.max_requests = max_tokens, num_pages, max_requests
        self.state_checkpoint_rows = tuple(range(max_requests, max_requests + state_checkpoints))
        self.act = act = torch.float32 if cfg.dtype == "float32" else torch.bfloat16
        self.logits_dtype = act
        self.ws = K.workspace(dev)
        self.sequential = cfg.design.sequential
        T, W = max_tokens, cfg.hidden_size

        def buf(cols: int, dtype=act) -> torch.Tensor:
            # zero-filled: padding columns are multiplied by zero weights, and must be finite for that
            return torch.zeros(T, cols, dtype=dtype, device=dev)

        self.x = buf(cfg.streams * W, torch.float32)      # residual stream, or streams
        project = cfg.loop is not None and cfg.design.loop == "project"
        self.x0 = buf(W, torch.float32) if project else None
        self.h = buf(round_up(W, 64))
        self.entry = buf(round_up(2 * W, 64)) if project else None
        # logits of the feed-forward's gate
        self.rg = buf(round_up(W, 8))[:, :W] if cfg.design.gated else None
        self.side = buf(round_up(cfg.side_dim, 64)) if cfg.side_dim else None
        self.side_y = buf(round_up(W, 8)) if cfg.side_dim else None
        self.y = buf(round_up(W, 8))[:, :W] if cfg.design.streams else None       # a sublayer's result
        self.kv = []                           # paged caches (copied page by page on copy-on-write)
        self.states = []                       # recurrent states (copied row by row)
        # per layer run: the cache or state of every mixer it consists of
        self.runs = [tuple(self._store(p) for p in _parts(weights.layers[i].mixer)) for i, _ in cfg.runs]
        # operands of the products by layout, scratch by width: layers share them
        self._operands: dict = {}
        self._scratch: dict = {}
        recurrent = []
        for l in weights.layers:
            self._operands.setdefault(self._layout(l), buf(l.out.k))
            self._need("proj", l.split)
            if l.down is not None:
                self._operands.setdefault(("act", l.ff_rows, l.down.k), buf(l.down.k))
            for m in _parts(l.mixer):
                s = m.spec
                if isinstance(m, LatentWeights):
                    if m.uq is not None:
                        self._need("cq%d" % s.q_rank, round_up(s.q_rank, 64))
                        self._need("q", m.uq.n)
                    self._need("ql", s.heads * s.row_padded)
                    self._need("ol", s.heads * s.rank_padded)
                elif isinstance(m, _PAGED):
                    self._need("q", s.heads * s.width_padded)
                elif not isinstance(m, MinGruWeights):
                    if isinstance(m, DeltaWeights):
                        recurrent.append((s.heads, s.kv_heads, s.dim, s.vdim, s.per_channel))
                    elif isinstance(m, SsdWeights):
                        recurrent.append((s.heads, s.groups, s.state, s.vdim, False))
                    else:
                        recurrent.append((s.heads, s.heads, s.dim, s.vdim, True))
                    if getattr(m, "low", None) is not None and (isinstance(m, DeltaWeights) or act == torch.float32):
                        self._need("low", m.low.n)
        self._routing()
        self._scratch = {n: torch.zeros(T * c, dtype=act, device=dev) for n, c in self._scratch.items()}
        self.recurrence = K.RecurrenceScratch(T, recurrent, act, dev) if recurrent else None
        self.trace: list | None = None         # a list here receives a copy of the residual after every layer run

    def _store(self, m):
        """Cache or state of one run of a mixer."""
        s, dev, rows = m.spec, self.device, self.max_requests + len(self.state_checkpoint_rows)
        if isinstance(m, LatentWeights):
            self.kv.append(torch.zeros(self.num_pages, 16, s.row_padded, dtype=self.act, device=dev))
            return self.kv[-1]
        if isinstance(m, MinGruWeights):
            self.states.append(_StateRun(rows, 1, 1, s.padded, dev))
            return self.states[-1]
        if isinstance(m, _PAGED):
            self.kv.append(torch.zeros(self.num_pages, s.kv_heads, 2, 16, s.width_padded, dtype=self.act, device=dev))
            if not isinstance(m, ConvAttentionWeights):
                return self.kv[-1]
            if s.conv == 1:
                return self.kv[-1], None
            self.states.append(_StateRun(rows, 0, 0, 0, dev, taps=s.conv, conv_width=s.conv_width, act=self.act))
            return self.kv[-1], self.states[-1].conv
        conv = {} if isinstance(m, GatedLinearWeights) else dict(taps=s.conv, conv_width=s.conv_width, act=self.act)
        self.states.append(_StateRun(rows, s.heads, s.vdim, s.state_stride, dev, **conv))
        return self.states[-1]

    def _routing(self) -> None:
        """Buffers of routed feed-forwards; layers of equal sizes share them."""
        T, W, dev = self.max_tokens, self.cfg.hidden_size, self.device
        routed = [l.routed for l in self.w.layers if l.routed is not None]
        self._z = torch.zeros(T * max((r.split for r in routed), default=0), dtype=torch.float32, device=dev)
        self._routes: dict = {}
        for r in routed:
            key = (r.spec.top, r.spec.experts)
            if key not in self._routes:
                self._routes[key] = K.ScoredScratch(T, r.spec.top, r.spec.experts, W, r.up.k, self.act, dev)
            for name, rows, m, used in (("expert", T * r.spec.top, r.down, r.spec.ff), ("shared", T, r.shared_down, r.spec.shared_ff)):
                if m is not None and (name, used, rows, m.k) not in self._operands:
                    self._operands[(name, used, rows, m.k)] = torch.zeros(rows, m.k, dtype=self.act, device=dev)

    def _layout(self, l) -> tuple:
        """What an operand of a layer's output product is shared by: every column keeps its role."""
        return (*(m.spec.out_width for m in _parts(l.mixer)), l.out_off, l.ff, l.out.k)

    def _need(self, name: str, cols: int) -> None:
        self._scratch[name] = max(self._scratch.get(name, 0), cols)

    def _rows(self, name: str, T: int, cols: int) -> torch.Tensor:
        return self._scratch[name][:T * cols].view(T, cols)

    def copy_state(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        """Whole recurrent-state rows ``src[i] -> dst[i]`` of every recurrent run."""
        for r in self.states:
            r.copy(src, dst)

    # ---------------------------------------------------------------- forward
    def forward_hidden(self, b) -> torch.Tensor:
        if b.segments is None:
            raise RuntimeError("layered decoders need the step's request segments (StepBatch.segments)")
        if self.cfg.design.streams:
            return self._streams(b)
        return self._sequential(b) if self.sequential else self._parallel(b)

    def _parallel(self, b) -> torch.Tensor:
        cfg, w, T = self.cfg, self.w, b.num_tokens
        decode = T == b.segments.num           # every segment has at most one row
        x, x0, h = self.x[:T], None if self.x0 is None else self.x0[:T], self.h[:T]
        K.embed_norm(b.token_ids[:T], w.embed, w.embed_norm, x, cfg.rms_eps, x0)
        n = 1
        for (i, enters), run in zip(cfg.runs, self.runs):
            l = w.layers[i]
            if enters:
                entry = self.entry[:T]
                K.concat_rows(x, x0, entry)
                K.wide_gemm(entry, w.loop_in, x, ws=self.ws)
                n += 2
            K.row_norm(x, l.norm, h, cfg.rms_eps)
            operand = self._operands[self._layout(l)][:T]
            proj = self._rows("proj", T, l.split)
            up = operand[:, l.out_off:l.out_off + l.ff] if l.ff else None
            K.wide_gemm(h, l.proj, proj, relu2=up, split=l.split, ws=self.ws)
            n += 3 + self._mix(l.mixer, proj, run, b, operand, decode)
            K.wide_gemm(operand, l.out, x, residual=x, ws=self.ws)
            self._after_layer(x)
        self.launches_per_step = n
        return x

    def _sequential(self, b) -> torch.Tensor:
        cfg, w, T, eps = self.cfg, self.w, b.num_tokens, self.cfg.rms_eps
        decode = T == b.segments.num
        x, h, W = self.x[:T], self.h[:T], cfg.hidden_size
        K.embed_rows(b.token_ids[:T], w.embed, w.layers[0].norm, x, h, eps, cfg.embed_scale)
        n, last = 1, len(cfg.runs) - 1
        for at, ((i, enters), run) in enumerate(zip(cfg.runs, self.runs)):
            l = w.layers[i]
            operand, proj = self._operands[self._layout(l)][:T], self._rows("proj", T, l.split)
            K.wide_gemm(h, l.proj, proj, ws=self.ws)
            n += 2 + self._mix(l.mixer, proj, run, b, operand, decode)
            K.wide_gemm(operand, l.out, x, residual=x, gate=(proj[:, l.rg_off:l.rg_off + W], l.rg[0]) if l.rg else None, ws=self.ws)
            if l.down is not None:
                act = self._operands[("act", l.ff_rows, l.down.k)][:T]
                rest = dict(rest=self.rg[:T], split=l.ff_rows, limit=l.limit) if l.rg else {}
                K.row_norm(x, l.norm2, h, eps)
                K.wide_gemm(h, l.gate_up, act[:, :l.ff_rows // 2], glu=cfg.design.ff[:-len("_glu")], ws=self.ws, **rest)
                K.wide_gemm(act, l.down, x, residual=x, gate=(self.rg[:T], l.rg[1]) if l.rg else None, ws=self.ws)
                n += 3
            follow = None if at == last else w.layers[cfg.runs[at + 1][0]].norm      # the final norm reads the wanted rows only
            if l.side is not None:
                n += K.side_input(x, l.side.gate, b.token_ids[:T], w.side_embed, l.side.col, l.side.proj, l.side.norm_w, eps, follow,
                                  None if follow is None else h, self.side[:T], self.side_y[:T, :W], self.ws)
            self._after_layer(x)
            if l.side is None and follow is not None:
                if cfg.reenters(at + 1):
                    K.embed_rows(b.token_ids[:T], w.embed, follow, x, h, eps, cfg.embed_scale, add=True)
                else:
                    K.row_norm(x, follow, h, eps)
                n += 1
        self.launches_per_step = n
        return x

    def _streams(self, b) -> torch.Tensor:
        cfg, w, T, eps = self.cfg, self.w, b.num_tokens, self.cfg.rms_eps
        decode = T == b.segments.num
        x, h, y = self.x[:T].view(T, cfg.streams, cfg.hidden_size), self.h[:T], self.y[:T]
        # what every sublayer reads: its weights of the streams and its norm; nothing behind the last
        reads = [(s.read, norm) for l in w.layers for s, norm in zip(l.streams, (l.norm, l.norm2))] + [(None, None)]
        K.stream_embed(b.token_ids[:T], w.embed, cfg.embed_scale, x, *reads[0], h, eps)
        n, at = 1, 0
        for l, run in zip(w.layers, self.runs):
            operand, proj = self._operands[self._layout(l)][:T], self._rows("proj", T, l.split)
            K.wide_gemm(h, l.proj, proj, ws=self.ws)
            n += 3 + self._mix(l.mixer, proj, run, b, operand, decode)
            K.wide_gemm(operand, l.out, y, ws=self.ws)
            for q, s in enumerate(l.streams):
                result, routes = y, None
                if q and l.routed is not None:
                    result, routes, made = self._routed(l.routed, h, y)
                    n += 1 + made
                elif q:
                    act = self._operands[("act", l.ff_rows, l.down.k)][:T]
                    K.wide_gemm(h, l.gate_up, act[:, :l.ff_rows // 2], glu=cfg.design.ff[:-len("_glu")], ws=self.ws)
                    K.wide_gemm(act, l.down, y, ws=self.ws)
                    n += 3
                at += 1
                K.stream_step(x, result, s.mix, s.write, h, eps, *reads[at], routes)
            self._after_layer(x.sum(1) if self.trace is not None else x)
        self.launches_per_step = n
        return self.x[:T]

    def _routed(self, m: RoutedWeights, h, y) -> tuple:
        """A routed feed-forward of ``h`` up to its combination: (shared expert's result, what the experts left, launches made)."""
        s, T = m.spec, h.shape[0]
        sc = self._routes[(s.top, s.experts)]
        z = self._z[:T * m.split].view(T, m.split)
        shared = None
        if s.shared_ff:
            shared = self._operands[("shared", s.shared_ff, self.max_tokens, m.shared_down.k)][:T]
            K.wide_gemm(h, m.head, z, relu2=shared[:, :s.shared_ff], split=m.split, ws=self.ws)
        else:
            K.wide_gemm(h, m.head, z, ws=self.ws)
        mb = K.scored_route(z, m.correction, h, self.cfg.hidden_size, s.experts, s.top, sc)
        rows = T * s.top
        act = self._operands[("expert", s.ff, self.max_tokens * s.top, m.down.k)]
        out = sc.ys[:, :self.cfg.hidden_size]
        K.grouped_gemm(sc.xs, m.up, act[:, :s.ff], sc, rows, mb, relu2=True, ws=self.ws)
        K.grouped_gemm(act, m.down, out, sc, rows, mb, ws=self.ws)
        if shared is not None:
            K.wide_gemm(shared, m.shared_down, y, ws=self.ws)
        gate = z[:, s.outputs:s.outputs + 1] if s.shared_ff else None
        routes = K.RoutedResult(out, sc.pos, sc.weight, sc.self_weight if s.identity else None, gate, s.top)
        return (None if shared is None else y), routes, 5 + (shared is not None)

    def _after_layer(self, x: torch.Tensor) -> None:
        if self.trace is not None:
            self.trace.append(x.clone())

    # ---------------------------------------------------------------- mixers: columns of ``proj`` -> columns of the operand
    def _mix(self, m, proj, run, b, operand, decode: bool) -> int:
        """Runs a layer's mixer; returns the launches made."""
        if isinstance(m, PairWeights):
            off = (0, m.spec.right_off)
            return sum(self._one(p, proj, store, b, operand[:, c:c + p.spec.out_width], decode)
                       for p, store, c in zip(_parts(m), run, off))
        return self._one(m, proj, run[0], b, operand[:, :m.spec.out_width], decode)

    def _one(self, m, proj, store, b, out, decode: bool) -> int:
        return _MIXERS[type(m)](self, m, proj, store, b, out, decode)

    def _delta(self, m: DeltaWeights, proj, run: _StateRun, b, out, decode: bool) -> int:
        s, T = m.spec, proj.shape[0]
        n = 1
        if m.low is not None:
            low = self._rows("low", T, m.low.n)
            K.wide_gemm(proj[:, m.a_off:m.a_off + m.low.k], m.low, low, ws=self.ws)
            a, z = low[:, :s.heads * s.dim], low[:, m.low_z:]
            n += 1
        else:
            a, z = proj[:, m.a_off:m.a_off + s.heads], proj[:, m.z_off:m.z_off + s.out_width]
        K.delta_prepare(proj[:, :s.conv_width], proj[:, m.b_off:m.b_off + s.heads], a, m.conv_w, run.conv, m.a_log, m.dt_bias,
                        b.segments, self.recurrence, s.heads, s.kv_heads, s.dim, s.vdim)
        return n + K.delta_walk(z, m.norm_w, run.state, b.segments, out, self.recurrence, s.kv_heads, s.dim, self.cfg.rms_eps,
                                s.per_channel, s.per_channel, decode)

    def _latent(self, m: LatentWeights, proj, cache: torch.Tensor, b, out, decode: bool) -> int:
        s, T, eps = m.spec, proj.shape[0], self.cfg.rms_eps
        ql, ol = self._rows("ql", T, s.heads * s.row_padded), self._rows("ol", T, s.heads * s.rank_padded)
        if m.uq is not None:
            cq, q = self._rows("cq%d" % s.q_rank, T, round_up(s.q_rank, 64)), self._rows("q", T, m.uq.n)
            K.latent_prepare(proj, m.c_off, s.kv_rank, m.c_norm, cache, b.slots, eps, low=(m.q_off, s.q_rank, m.q_norm, cq))
            K.wide_gemm(cq, m.uq, q, ws=self.ws)
            K.wide_gemm(q, m.absorb.w, ql, diag_rows=m.absorb.rows, ws=self.ws)
        else:                                  # the product writes zeros where the rotated part follows
            K.wide_gemm(proj[:, m.q_off:m.qr_off], m.absorb.w, ql, diag_rows=m.absorb.rows, ws=self.ws)
            K.latent_prepare(proj, m.c_off, s.kv_rank, m.c_norm, cache, b.slots, eps,
                             rotated=(m.qr_off, m.r_off, s.rot_col, m.freq, m.rot_mult, b.positions[:T], ql, s.heads))
        K.latent_attention(ql, proj[:, m.g_off:m.g_off + s.heads] if s.gated else None, cache, b.page_table, b.segments, ol, s.heads,
                           s.window, s.scale, decode=decode, ws=self.ws)
        K.wide_gemm(ol, m.value.w, out, diag_rows=m.value.rows, ws=self.ws)
        return 5 if m.uq is not None else 4

    def _attention(self, m: AttentionWeights, proj, cache: torch.Tensor, b, out, decode: bool) -> int:
        s, T = m.spec, proj.shape[0]
        q = self._rows("q", T, s.heads * s.width_padded)
        K.gqa_prepare(proj, m.q_off, m.k_off, m.q_norm, m.k_norm, m.freq, m.rot_mult, b.positions[:T], b.slots[:T], q, cache, s.heads,
                      s.dim, self.cfg.rms_eps)
        return 1 + K.gqa_attention(q, cache, b.page_table, b.segments, out, s.heads, s.dim, s.window, s.scale, s.sink, m.out_scale,
                                   decode=decode, ws=self.ws)

    def _conv_attention(self, m: ConvAttentionWeights, proj, store, b, out, decode: bool) -> int:
        s, T, (cache, history) = m.spec, proj.shape[0], store
        q = self._rows("q", T, s.heads * s.width_padded)
        K.conv_qkv(proj, tuple(m.q_off + o for o in s.offsets), m.conv_w, history, m.freq, b.positions[:T], b.slots[:T], b.segments, q,
                   cache, s.heads, s.dim, s.vdim, self.cfg.rms_eps)
        return 1 + K.gqa_attention(q, cache, b.page_table, b.segments, out, s.heads, s.vdim, s.window, s.scale, decode=decode, ws=self.ws,
                                   keep=s.keep)

    def _biased_attention(self, m: BiasedAttentionWeights, proj, cache: torch.Tensor, b, out, decode: bool) -> int:
        s, T = m.spec, proj.shape[0]
        q = self._rows("q", T, s.heads * s.width_padded)
        K.norm_qkv(proj, tuple(m.q_off + o for o in s.offsets), m.q_norm, m.k_norm, b.positions[:T], b.slots[:T], q, cache, s.heads,
                   s.dim, s.vdim, self.cfg.rms_eps, (s.temp_coef, s.temp_every))
        return 1 + K.gqa_attention(q, cache, b.page_table, b.segments, out, s.heads, s.vdim, s.window, s.scale, decode=decode, ws=self.ws,
                                   bias=m.bias)

    def _differential(self, m: DifferentialWeights, proj, cache: torch.Tensor, b, out, decode: bool) -> int:
        s, T = m.spec, proj.shape[0]
        q = self._rows("q", T, s.heads * s.width_padded)
        K.head_qkv(proj, tuple(m.q_off + o for o in s.offsets), m.q_norm, m.k_norm, m.freq, b.positions[:T], b.slots[:T], q, cache,
                   s.heads, s.dim, s.vdim, self.cfg.rms_eps, maps=2)
        return 1 + K.gqa_attention(q, cache, b.page_table, b.segments, out, s.heads, s.vdim, 0, s.scale, out_scale=1.0 - s.diff,
                                   decode=decode, ws=self.ws, chunk=s.chunk,
                                   pair=(proj[:, m.g_off:m.g_off + s.out_width], m.less, self.cfg.rms_eps))

    def _mingru(self, m: MinGruWeights, proj, run: _StateRun, b, out, decode: bool) -> int:
        K.mingru(proj, m.z_off, m.x_off, m.g_off, m.bias, run.state[:, 0, 0], b.segments, out)
        return 1

    def _gated_linear(self, m: GatedLinearWeights, proj, run: _StateRun, b, out, decode: bool) -> int:
        s, T, n = m.spec, proj.shape[0], 1
        low, a = m.low, proj[:, m.a_off:m.a_off + m.low.k]
        if proj.dtype != torch.bfloat16:       # bf16: the preparation makes the decay logits itself
            z = self._rows("low", T, low.n)
            K.wide_gemm(a, low, z, ws=self.ws)
            low, a, n = None, z, 2
        K.gated_linear_prepare(proj, m.q_off, m.k_off, m.v_off, a, m.bias, 1.0 / s.tau, b.segments, self.recurrence, s.heads, s.dim,
                               s.vdim, low, s.decay_rank)
        return n + K.gated_linear_walk(proj[:, m.g_off:m.g_off + s.out_width], m.norm_w, run.state, b.segments, out, self.recurrence,
                                       s.dim, self.cfg.rms_eps, decode)

    def _ssd(self, m: SsdWeights, proj, run: _StateRun, b, out, decode: bool) -> int:
        s = m.spec
        K.ssd_prepare(proj[:, m.x_off:m.x_off + s.conv_width], proj[:, m.dt_off:m.dt_off + s.heads], m.conv_w, m.conv_b, run.conv,
                      m.a_log, m.dt_bias, b.segments, self.recurrence, s.heads, s.groups, s.state, s.vdim)
        return 1 + K.ssd_walk(proj[:, m.z_off:m.z_off + s.out_width], m.d, m.norm_w, s.norm_groups, run.state, b.segments, out,
                              self.recurrence, s.groups, s.state, self.cfg.rms_eps, decode)

    def forward_logits(self, b, hidden: torch.Tensor, logits_out: torch.Tensor) -> torch.Tensor:
        """Final norm and output head of the selected rows."""
        R = b.num_logit_rows
        h = self.h[:R]                         # free once the last layer has run
        if self.cfg.design.streams:
            K.stream_norm(hidden.view(-1, self.cfg.streams, self.cfg.hidden_size), self.w.final_norm, h, self.cfg.rms_eps,
                          rows=b.logit_rows[:R])
        else:
            K.row_norm(hidden, self.w.final_norm, h, self.cfg.rms_eps, rows=b.logit_rows[:R])
        K.wide_gemm(h, self.w.lm_head, logits_out[:R], ws=self.ws)
        self.launches_per_step += 2
        return logits_out[:R]


_MIXERS = {DeltaWeights: LayeredRunner._delta, LatentWeights: LayeredRunner._latent, AttentionWeights: LayeredRunner._attention,
           GatedLinearWeights: LayeredRunner._gated_linear, SsdWeights: LayeredRunner._ssd,
           ConvAttentionWeights: LayeredRunner._conv_attention, BiasedAttentionWeights: LayeredRunner._biased_attention,
           DifferentialWeights: LayeredRunner._differential, MinGruWeights: LayeredRunner._mingru}
