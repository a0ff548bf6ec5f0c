"""What a token takes from the one before it: the bigram embedding, and the shifted norm of "shifted" blocks, whose mixer reads
h + (h' - h) * shift with h' the previous token's norm output.

One kernel per layer (`csrc/token_shift.cu`) forms the residual after the layer before (both mixers' outputs, each RMS-normed, and the
feed-forward's, for experts their weighted sum), its norm h, the shifted row s that the mixer reads, and the blends
s + (s' - s) * mu_j that a time-mixing side projects.  The previous token of a span's first one comes from the request's state; what the
next step will find there is left beside it and moves in when the step is over (`commit`), so no kernel of the step can see it early.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from . import _lib
from .hybrid import HybridMeta, _is32, expert_sum
from .moe import ExpertRows
from .scratch import scratch

F32 = torch.float32


@dataclass
class Pending:
    """What a layer adds to the residual: up to two mixer outputs (fp32 rows, the weight of their RMS norm or None, a factor), and the
    feed-forward's rows (fp32, or `ExpertRows`)."""
    outs: List[Tuple[torch.Tensor, Optional[torch.Tensor], float]]
    ff: object = None


@dataclass
class ShiftState:
    """Per request row: the last token, and per layer the last norm output and the last shifted row (fp32).  `now` is what a step
    reads, `then` what it leaves for the next one."""
    token: torch.Tensor            # [rows] int64
    now: torch.Tensor              # [layers, rows, 2, W]
    then: torch.Tensor


def shift_state(layers: int, rows: int, width: int, device) -> ShiftState:
    z = lambda: torch.zeros(layers, rows, 2, width, dtype=F32, device=device)
    return ShiftState(torch.zeros(rows, dtype=torch.int64, device=device), z(), z())


def embed_bigram(meta: HybridMeta, embed: torch.Tensor, scale: float, table: Optional[torch.Tensor], bigram, st: ShiftState) -> torch.Tensor:
    """-> fp32 residual [T, W]: the token's embedding (times scale), plus the row of `table` that it and the token before it select."""
    ids, w = meta.token_ids, embed.shape[1]
    t = ids.shape[0]
    if not ids.is_cuda:
        ok = (ids >= 0) & (ids < embed.shape[0])
        x = torch.where(ok[:, None], embed[ids.clamp(0, embed.shape[0] - 1)].to(F32) * scale, torch.zeros(1))
        if table is None:
            return x
        for i in range(t):
            r, p = int(meta.tok_req[i]), int(meta.positions[i])
            if r < 0 or p < 0 or not ok[i]:
                continue
            row = bigram.buckets
            if p > 0:
                last = int(ids[i - 1]) if p > int(meta.first_pos[i]) else int(st.token[r])
                row = (last * bigram.mul_prev + int(ids[i]) * bigram.mul_cur) % bigram.buckets
            x[i] += table[row].to(F32)
        return x
    x = torch.empty(t, w, dtype=F32, device=ids.device)
    b = (bigram.buckets, bigram.mul_prev, bigram.mul_cur) if table is not None else (1, 0, 0)
    _lib.call("stk_embed_bigram", ids, embed, _is32(embed), float(scale), table, *b, meta.tok_req, meta.positions, meta.first_pos, st.token, x, t, w,
              embed.shape[0], _lib.status_buffer(), _lib.stream())
    return x


def _add_cpu(x: torch.Tensor, p: Pending, eps: float) -> torch.Tensor:
    x = x.clone()
    for y, w, f in p.outs:
        y = y[:, :x.shape[1]]
        x += (y if w is None else y * torch.rsqrt((y * y).mean(-1, keepdim=True) + eps) * w) * f
    if p.ff is not None:
        x += expert_sum(p.ff, x.shape[1])[:, :x.shape[1]]
    return x


def shifted_norm(x: torch.Tensor, p: Optional[Pending], norm: torch.Tensor, eps: float, width: int, dtype: torch.dtype,
                 shift: Optional[torch.Tensor] = None, mu: Optional[torch.Tensor] = None, st: Optional[ShiftState] = None, layer: int = 0,
                 meta: Optional[HybridMeta] = None, rows: Optional[torch.Tensor] = None):
    """x [T, W] fp32 plus what is pending -> (the sum, its RMS norm h, shifted s, blends): h and s in `dtype`, zero-padded to `width`
    columns; blends [T, len(mu) * width], one after the other.  Without `shift` only the sum and h; rows: only h, of these rows."""
    t, w_n = x.shape
    blends = mu.shape[0] if mu is not None else 0
    if not x.is_cuda:
        if p is not None:
            x = _add_cpu(x, p, eps)
        pad = lambda v: torch.nn.functional.pad(v, (0, width - w_n)).to(dtype)
        hf = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * norm
        if rows is not None:
            return None, pad(hf[rows]), None, None
        if shift is None:
            return x, pad(hf), None, None
        sf, mf = torch.zeros_like(hf), torch.zeros(t, blends, w_n)
        for i in range(t):
            r, q = int(meta.tok_req[i]), int(meta.positions[i])
            if r < 0 or q < 0:
                continue
            zero = torch.zeros(w_n)
            if q > int(meta.first_pos[i]):
                hp, sp = hf[i - 1], sf[i - 1]
            else:
                hp, sp = st.now[layer, r] if q > 0 else (zero, zero)
            sf[i] = hf[i] + (hp - hf[i]) * shift
            if blends:
                mf[i] = sf[i] + (sp - sf[i]) * mu
            if q == int(meta.last_pos[i]):
                st.then[layer, r, 0], st.then[layer, r, 1] = hf[i], sf[i]
        return x, pad(hf), pad(sf), pad(mf).flatten(1) if blends else None
    n = t if rows is None else rows.shape[0]
    dev = x.device
    h = torch.empty(n, width, dtype=dtype, device=dev)
    s = torch.empty(n, width, dtype=dtype, device=dev) if shift is not None else None
    mix = torch.empty(n, blends * width, dtype=dtype, device=dev) if blends else None
    out = torch.empty_like(x) if p is not None and rows is None else None
    outs = (p.outs if p is not None else []) + [(None, None, 0.0)] * 2
    args = []
    for y, w, f in outs[:2]:
        args += [y, y.stride(0) if y is not None else 0, w, float(f)]
    ff = p.ff if p is not None else None
    pairs = ff if isinstance(ff, ExpertRows) else None
    plain = ff if pairs is None else None
    _lib.call("stk_shifted_norm", x, out, *args, plain, plain.stride(0) if plain is not None else 0, pairs.y if pairs is not None else None,
              pairs.y.stride(0) if pairs is not None else 0, pairs.pair_row if pairs is not None else None,
              pairs.weights if pairs is not None else None, pairs.weights.shape[1] if pairs is not None else 0, norm, float(eps), shift, mu, blends,
              h, s, mix, width, _is32(h), st.now[layer] if shift is not None else None, st.then[layer] if shift is not None else None,
              meta.tok_req if shift is not None else None, meta.positions if shift is not None else None,
              meta.first_pos if shift is not None else None, meta.last_pos if shift is not None else None, rows,
              scratch("shift.inv", (n,), F32, dev) if shift is not None else None, n, w_n,
              1 if meta is not None and meta.pure_decode else 0, _lib.sm_count(), _lib.stream())
    return (out if out is not None else x if rows is None else None), h, s, mix


def commit(st: ShiftState, meta: HybridMeta) -> None:
    """The step's last tokens and rows become what the next step finds."""
    if not st.now.is_cuda:
        for i in range(meta.n_req):
            a, b = int(meta.query_start[i]), int(meta.query_start[i + 1])
            if b > a:
                r = int(meta.req_rows[i])
                st.token[r] = meta.token_ids[b - 1]
                st.now[:, r] = st.then[:, r]
        return
    layers, n_rows, _, w = st.now.shape
    _lib.call("stk_shift_commit", meta.query_start, meta.req_rows, meta.n_req, meta.token_ids, st.token, st.then, st.now, layers, n_rows,
              2 * w, _lib.stream())
