"""What every native model body does after its layers: logits of the wanted rows, sampling, token agreement between ranks
and the thinking-budget state machine.  ``models.decoder.DecoderRunner`` and ``models.layered_runner.LayeredRunner`` derive
from it and supply ``forward_hidden`` and ``forward_logits``.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K


class StepRunner:
    # set by the subclass
    tp = None
    pp = None
    device = None
    max_requests = 0
    reasoning = None                 # K.ReasoningBudget once enable_reasoning_budget() was called
    launches_per_step = 0
    logits_dtype = torch.bfloat16

    def _dummy_val(self) -> torch.Tensor:
        if not hasattr(self, "_cand_val"):
            self._cand_val = torch.zeros(1, dtype=torch.float32, device=self.device)
            self._cand_id = torch.zeros(1, dtype=torch.int32, device=self.device)
        return self._cand_val

    def _dummy_id(self) -> torch.Tensor:
        self._dummy_val()
        return self._cand_id

    def enable_reasoning_budget(self, end_token_id: int, forced_tokens: list[int]) -> None:
        """Enforce thinking-token budgets on the device (before the decode graphs are captured): after the budget of
        a request is used up its sampled ids are replaced by ``forced_tokens`` (1-4 tokens, ending the reasoning
        block); sampling ``end_token_id`` on its own ends the phase.  Every rank and stage runs the same state
        machine on the same ids."""
        self.reasoning = K.ReasoningBudget(self.max_requests, end_token_id, forced_tokens, self.device)

    def run_step(self, b, d: dict, logits_buf: torch.Tensor, out_ids: torch.Tensor) -> None:
        """Whole step: layers, final norm, lm_head, sampling (and the cross-rank token agreement under TP), then the
        thinking-budget state machine on the sampled ids when it is enabled."""
        self._run_step(b, d, logits_buf, out_ids)
        if self.reasoning is not None and b.num_logit_rows:
            self.reasoning.apply(out_ids, d["row_slot"], d["budget_init"], b.num_logit_rows)
            self.launches_per_step += 1

    def _run_step(self, b, d: dict, logits_buf: torch.Tensor, out_ids: torch.Tensor) -> None:
        R = b.num_logit_rows
        fused = self.tp is not None and self.tp.fused is not None
        pp = self.pp
        if not fused:
            hidden = self.forward_hidden(b)
            if not R:
                return
            if pp is not None and not pp.is_last:
                pp.share_token_ids(out_ids[:R])        # receive what the last stage sampled
                return
            logits = self.forward_logits(b, hidden, logits_buf)
        else:
            f = self.tp.fused
            s = self.forward_hidden_fused(b)
            if R == b.num_tokens:
                logits = f.gemm_gather(self.w.lm_head, logits_buf[:R], s)
            else:
                x = f.wait_gather(s)
                if R:
                    rows = torch.index_select(x, 0, b.logit_rows[:R])
                    logits = K.wq_gemm(rows, self.w.lm_head, out=logits_buf[:R], ws=self.ws)
            self.launches_per_step += 2
        mask = d.get("mask")             # allowed-token bitmask rows [R, ceil(V / 32)] (structured output) or None
        if mask is not None:
            mask = mask[:R, self.w.vocab_start // 32:]       # this rank's vocabulary shard starts at a word boundary
        if self.tp is None:
            K.sample(logits, out_ids[:R], temperature=d["temperature"][:R], top_p=d["top_p"][:R], top_k=d["top_k"][:R],
                     seeds=d["seeds"][:R], counters=d["draws"][:R], vocab=logits.shape[1], mask=mask)
            self.launches_per_step += 1
            if pp is not None:
                pp.share_token_ids(out_ids[:R])
            return
        # vocab-sharded: rank-local candidates (one for a greedy row, up to 20 for a sampled one), exchanged
        # between the ranks, then the same merge + draw on every rank
        if fused:
            if R:
                self.tp.fused.sample_sharded(logits, R, out_ids, d, self.w.vocab_start, mask)
            else:
                self.tp.fused.argmax_merge(self._dummy_val(), self._dummy_id(), out_ids, 0)   # step barrier only
        elif R:
            self.tp.sample_sharded_nccl(logits, R, out_ids, d, self.w.vocab_start, mask)
        self.launches_per_step += 3
        if pp is not None and R:
            pp.share_token_ids(out_ids[:R])
