"""Layered decoders on the native sm_100a kernels.

``LayeredRunner`` is the model body of ``models/layered.py`` checkpoints: it owns the packed weights, fixed-address
buffers, one paged latent cache per attention run and the per-request state of every delta run, and serves the executor
through the same surface as ``DecoderRunner`` (``forward_hidden`` / ``forward_logits`` / ``run_step``, all capturable in a
CUDA graph).  A layer run is

    norm(x) -> h                          fp32 residual in, activation type out
    [mixer inputs | relu^2(up)] = h W     one product; the up columns leave as the right half of the output's operand
    mixer -> left half of that operand
    x += [o | relu^2(up)] [W_o | W_down]  one product, accumulated into the fp32 residual

``cfg.dtype`` "float32" runs the same steps with fp32 activations and fp32 products.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from .layered import DeltaWeights, LatentWeights, LayeredConfig, LayeredWeights, round_up
from .step_runner import StepRunner


class _DeltaRun:
    """Per-request state of one run of a delta layer: convolution history (activation type) and delta-rule state (fp32)."""

    def __init__(self, spec, rows: int, act: torch.dtype, device) -> None:
        # a row is a multiple of 16 bytes (whole-row copies); the history's layout inside it is [taps - 1, channels]
        self.conv = torch.zeros(rows, max(1, spec.conv - 1), spec.conv_width, dtype=act, device=device)
        self.state = torch.zeros(rows, spec.heads, spec.vdim, spec.state_stride, dtype=torch.float32, device=device)

    def copy(self, src, dst) -> None:
        K.copy_rows(self.conv, src, dst)
        K.copy_rows(self.state, src, dst)


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
        T, W = max_tokens, cfg.hidden_size

        def buf(cols: int, dtype=act) -> torch.Tensor:
            # zero-filled: padding columns are multiplied by zero weights, and must be finite for that
            return torch.zeros(T, cols, dtype=dtype, device=dev)

        self.x = buf(W, torch.float32)         # residual stream
        self.x0 = buf(W, torch.float32) if cfg.loop is not None else None
        self.h = buf(round_up(W, 64))
        self.entry = buf(round_up(2 * W, 64)) if cfg.loop is not None else None
        self.runs = []                         # per layer run: _DeltaRun or the latent cache of the run
        self.kv = []                           # latent caches (copied page by page on copy-on-write)
        for i, _ in cfg.runs:
            m = cfg.layers[i].mixer
            if isinstance(weights.layers[i].mixer, DeltaWeights):
                self.runs.append(_DeltaRun(m, max_requests + state_checkpoints, act, dev))
            else:
                self.runs.append(torch.zeros(num_pages, 16, m.rank_padded, dtype=act, device=dev))
                self.kv.append(self.runs[-1])
        # operands of the output products ([mixer output | feed-forward]) by layout, scratch by width: layers share them
        self._operands: dict = {}
        self._scratch: dict = {}
        delta = []
        for l in weights.layers:
            key = (l.mixer.spec.out_width, l.out_off, l.ff, l.out.k)
            self._operands.setdefault(key, buf(l.out.k))
            self._need("proj", l.split)
            if isinstance(l.mixer, DeltaWeights):
                m = l.mixer.spec
                delta.append((m.heads, m.kv_heads, m.dim, m.vdim, m.per_channel))
                if l.mixer.low is not None:
                    self._need("low", l.mixer.low.n)
            else:
                m, mw = l.mixer.spec, l.mixer
                self._need("cq%d" % m.q_rank, round_up(m.q_rank, 64))
                self._need("q", mw.uq.n)
                self._need("ql", m.heads * m.rank_padded)
                self._need("ol", m.heads * m.rank_padded)
        self._scratch = {n: torch.zeros(T * c, dtype=act, device=dev) for n, c in self._scratch.items()}
        self.delta = K.DeltaScratch(T, delta, act, dev) if delta else None
        self.trace: list | None = None         # a list here receives a copy of the residual after every layer run

    def _need(self, name: str, cols: int) -> None:
        self._scratch[name] = max(self._scratch.get(name, 0), cols)

    def _rows(self, name: str, T: int, cols: int) -> torch.Tensor:
        return self._scratch[name][:T * cols].view(T, cols)

    def copy_state(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        """Whole recurrent-state rows ``src[i] -> dst[i]`` of every delta run."""
        for r in self.runs:
            if isinstance(r, _DeltaRun):
                r.copy(src, dst)

    # ---------------------------------------------------------------- forward
    def forward_hidden(self, b) -> torch.Tensor:
        cfg, w, T = self.cfg, self.w, b.num_tokens
        if b.segments is None:
            raise RuntimeError("layered decoders need the step's request segments (StepBatch.segments)")
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
            m = l.mixer
            operand = self._operands[(m.spec.out_width, l.out_off, l.ff, l.out.k)][:T]
            proj = self._rows("proj", T, l.split)
            up = operand[:, l.out_off:l.out_off + l.ff] if l.ff else None
            K.wide_gemm(h, l.proj, proj, relu2=up, split=l.split, ws=self.ws)
            mixed = operand[:, :m.spec.out_width]
            n += 3 + (self._delta(m, proj, run, b, mixed, decode) if isinstance(m, DeltaWeights)
                      else self._latent(m, proj, run, b, mixed, decode))
            K.wide_gemm(operand, l.out, x, residual=x, ws=self.ws)
            if self.trace is not None:
                self.trace.append(x.clone())
        self.launches_per_step = n
        return x

    def _delta(self, m: DeltaWeights, proj, run: _DeltaRun, b, out, decode: bool) -> int:
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
                        b.segments, self.delta, s.heads, s.kv_heads, s.dim, s.vdim)
        return n + K.delta_walk(z, m.norm_w, run.state, b.segments, out, self.delta, s.kv_heads, s.dim, self.cfg.rms_eps,
                                s.per_channel, s.per_channel, decode)

    def _latent(self, m: LatentWeights, proj, cache: torch.Tensor, b, out, decode: bool) -> int:
        s, T = m.spec, proj.shape[0]
        wide = s.heads * s.rank_padded
        cq = self._rows("cq%d" % s.q_rank, T, round_up(s.q_rank, 64))
        q, ql, ol = self._rows("q", T, m.uq.n), self._rows("ql", T, wide), self._rows("ol", T, wide)
        K.latent_prepare(proj, s.q_rank, m.c_off, s.kv_rank, m.q_norm, m.c_norm, cq, cache, b.slots, self.cfg.rms_eps)
        K.wide_gemm(cq, m.uq, q, ws=self.ws)
        K.wide_gemm(q, m.absorb.w, ql, diag_rows=m.absorb.rows, ws=self.ws)
        K.latent_attention(ql, proj[:, m.g_off:m.g_off + s.heads], cache, b.page_table, b.segments, ol, s.heads, s.window,
                           s.scale, decode=decode, ws=self.ws)
        K.wide_gemm(ol, m.value.w, out, diag_rows=m.value.rows, ws=self.ws)
        return 5

    def forward_logits(self, b, hidden: torch.Tensor, logits_out: torch.Tensor) -> torch.Tensor:
        """Final norm and output head of the selected rows."""
        R = b.num_logit_rows
        h = self.h[:R]                         # free once the last layer has run
        K.row_norm(hidden, self.w.final_norm, h, self.cfg.rms_eps, rows=b.logit_rows[:R])
        K.wide_gemm(h, self.w.lm_head, logits_out[:R], ws=self.ws)
        self.launches_per_step += 2
        return logits_out[:R]
