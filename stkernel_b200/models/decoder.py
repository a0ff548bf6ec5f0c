"""What every model family's decoder shares with the engine: sampling from head hidden states, selection of the sampling
rows, pipeline-stage hand-over of tokens and log-probabilities.

A family implements `build_meta`, `forward_hidden`, `head_hidden` and `compute_logits`; the engine calls `forward_sample`
(and `forward_hidden` alone for a prompt portion that samples nothing, `score` for logits at given rows).
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ..ops import functional as Fn


class Decoder:
    recurrent = False          # running a step twice changes more than running it once (a state advances)

    def __init__(self, device, comm=None, tp_rank: int = 0, tp_size: int = 1):
        self.device = torch.device(device)
        self.comm = comm
        self.tp_rank, self.tp_size = tp_rank, tp_size
        self.vocab_start = 0                                 # first vocabulary row of this rank's head shard
        self.pipe = None                                     # parallel.pipeline.PipeStage when the model is one stage of several
        self.pipe_defer = False                              # the engine exchanges a step's tokens when it finishes the step
        self.want_logprobs: Optional[int] = None             # set by the engine for a step that reports log-probabilities
        self.last_logprobs = None                            # (sampled token's, top values, top ids) of that step
        self.load_recorder = None                            # parallel.eplb.LoadRecorder when expert load is being recorded

    # ---- what a family provides --------------------------------------------------
    def build_meta(self, buf, t_pad: int, n_req: int, max_comp_rows: int, pure_decode: bool = False,
                   spans: Tuple = (1, 1)):
        """Device-side description of the staged step.  spans = (shortest, longest[, all as (start, tokens)]) spans,
        known on the host."""
        raise NotImplementedError

    def decode_bucket(self, max_comp_rows: int) -> int:
        """Key of the captured decode graph that serves a step with contexts of up to 4 * max_comp_rows tokens, and the
        value `max_comp_rows` takes inside that graph."""
        return 0

    def forward_hidden(self, meta):
        raise NotImplementedError

    def head_hidden(self, X, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Input of the LM head for the selected token rows (all of them when rows is None)."""
        raise NotImplementedError

    def compute_logits(self, h: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def _ll_any(self, words: int):
        return None

    # ---- shared --------------------------------------------------------------------
    def local_logits(self, h: torch.Tensor) -> torch.Tensor:
        """This rank's vocabulary shard of the logits."""
        return self.compute_logits(h)

    def sample(self, h: torch.Tensor, temp: torch.Tensor, seed: torch.Tensor, pos: torch.Tensor,
               top_k: Optional[torch.Tensor] = None, top_p: Optional[torch.Tensor] = None,
               agreed_status: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Head hidden states [n, H] -> sampled tokens [n] (seeded Gumbel arg-max).  Under tensor parallelism the
        logits stay sharded: every rank takes the noisy arg-max of its vocabulary shard and the ranks exchange one
        candidate per row (no logits all-gather); truncated sampling (top-k / top-p) needs the whole row and gathers."""
        from ..ops import sampling as S
        n = h.shape[0]
        if self.want_logprobs is not None:
            # log-probabilities asked for: the whole rows are needed anyway (gathered across ranks); the token is the one
            # the sharded arg-max would pick (same noise, same logits)
            lg = self.compute_logits(h)
            toks, _ = S.gumbel_argmax(lg, temp, seed, pos, top_k=top_k, top_p=top_p)
            lp = torch.log_softmax(lg.float(), dim=-1)
            top_lp, top_ids = lp.topk(max(1, min(self.want_logprobs, lp.shape[1])), dim=-1)
            self.last_logprobs = (lp.gather(1, toks.view(-1, 1).long()).squeeze(1), top_lp, top_ids)
            return toks
        ll = None
        if self.tp_size > 1 and top_k is None and top_p is None and h.is_cuda and n <= 256:
            ll = self._ll_any(3 * n)
        if ll is not None:
            lg = self.local_logits(h)
            toks, _ = S.gumbel_argmax(lg, temp, seed, pos, vocab_start=self.vocab_start, ll=ll, agreed_status=agreed_status)
            return toks
        toks, _ = S.gumbel_argmax(self.compute_logits(h), temp, seed, pos, top_k=top_k, top_p=top_p)
        return toks

    def forward_sample(self, meta, logit_rows: Optional[torch.Tensor], temp, seed, pos, top_k=None, top_p=None,
                       agreed_status=None) -> torch.Tensor:
        """Sampled tokens for the selected token rows (all rows when logit_rows is None)."""
        X = self.forward_hidden(meta)
        pipe = self.pipe
        if pipe is not None and not pipe.last:
            # an earlier stage: the step's tokens come back from the last one (now, or when the engine finishes the
            # step if the exchange is deferred)
            n = logit_rows.shape[0] if logit_rows is not None else meta.token_ids.shape[0]
            toks = torch.zeros(n, dtype=torch.int64, device=meta.token_ids.device)
            return toks if self.pipe_defer else pipe.broadcast_from_last(toks)
        toks = self.sample(self.head_hidden(X, logit_rows), temp, seed, pos, top_k, top_p, agreed_status)
        if pipe is None or self.pipe_defer:
            return toks.contiguous() if pipe is not None else toks
        return pipe.broadcast_from_last(toks.contiguous())

    def forward(self, meta, logit_rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Logits for the selected token rows (all rows when logit_rows is None)."""
        return self.compute_logits(self.head_hidden(self.forward_hidden(meta), logit_rows))
