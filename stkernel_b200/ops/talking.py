"""Grouped-query attention whose heads' scores are mixed before the softmax ("talking heads"): score_h <- sum_g T[h, g] score_g.

A mixed score is linear in the queries, so it is one product of a mixed query with the keys of all key/value heads side by side:
the part of head h's mixed query that meets key/value head c is sum of T[h, g] q_g over the heads g that read c.  The mixed queries are
formed once per token (`talking_prep`), and every head then attends with keys [kv_heads * dim] that all heads share.

A cached row is [values of all key/value heads | keys of all key/value heads], every head's part zero-padded to 16 columns
(`talking_row`).  Chunks restrict a position to the keys of its own chunk.  Norms, rotation, mixing, scores, softmax, sinks and gates are
fp32; queries are rounded once, after they are mixed.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from . import reference as R
from .cache import PAGE
from .hybrid import HybridMeta, _is32
from .latent import PROMPT_ROWS, PROMPT_SPAN, _up
from .scratch import scratch

F32 = torch.float32


def talking_row(kv_heads: int, dim: int, vdim: int) -> Tuple[int, int, int, int]:
    """(elements of a cached row, column where the keys start, columns per key, columns per value)."""
    kp, vp = _up(dim, 16), _up(vdim, 16)
    return kv_heads * (kp + vp), kv_heads * vp, kp, vp


@dataclass
class TalkingParams:
    """One layer on the device."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                             # positions per chunk; 0: the full context
    eps: float
    bias: Optional[torch.Tensor]           # fp32 [heads * dim | kv_heads * dim | kv_heads * vdim]
    q_norm: Optional[torch.Tensor]         # fp32 [dim]; None: as projected
    k_norm: Optional[torch.Tensor]
    freq: torch.Tensor                     # [2, pairs] (`latent.split_frequencies`): dimension 2 i turns with 2 i + 1
    talk: torch.Tensor                     # fp32 [heads, heads]
    sink: Optional[torch.Tensor]           # fp32 [heads]
    gated: bool


def talking_prep(p: torch.Tensor, q_off: int, k_off: int, v_off: int, g_off: int, a: TalkingParams, meta: HybridMeta, table: torch.Tensor,
                 cache: torch.Tensor) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """Inserts the tokens' rows into the paged cache; -> (mixed queries [heads, T, kv_heads * kp], gate logits [T, heads] fp32)."""
    t = p.shape[0]
    h, g, d, v = a.heads, a.kv_heads, a.dim, a.vdim
    row, k_col, kp, vp = talking_row(g, d, v)
    if not p.is_cuda:
        b = a.bias if a.bias is not None else torch.zeros(h * d + g * (d + v))
        q = (p[:, q_off:q_off + h * d].to(F32) + b[:h * d]).reshape(t, h, d)
        k = (p[:, k_off:k_off + g * d].to(F32) + b[h * d:(h + g) * d]).reshape(t, g, d)
        vv = (p[:, v_off:v_off + g * v].to(F32) + b[(h + g) * d:]).reshape(t, g, v)
        if a.q_norm is not None:
            q, k = R.unit_rms(q, a.eps) * a.q_norm, R.unit_rms(k, a.eps) * a.k_norm
        n = 2 * a.freq.shape[1]
        q = torch.cat([R.rotate_pairs(q[..., :n], meta.positions, a.freq), q[..., n:]], -1)
        k = torch.cat([R.rotate_pairs(k[..., :n], meta.positions, a.freq), k[..., n:]], -1)
        R.talking_kv_insert(k, vv, k_col, kp, vp, meta.positions, meta.tok_req, table, cache)
        out = torch.zeros(h, t, g, kp, dtype=p.dtype)
        out[..., :d] = torch.einsum("hcj,tcjd->htcd", a.talk.view(h, g, h // g), q.view(t, g, h // g, d)).to(p.dtype)
        return out.flatten(2), p[:, g_off:g_off + h].to(F32) if a.gated else None
    out = torch.empty(h, t, g * kp, dtype=p.dtype, device=p.device)
    gate = torch.empty(t, h, dtype=F32, device=p.device) if a.gated else None
    _lib.call("stk_talking_prep", p, p.stride(0), q_off, k_off, v_off, g_off, a.bias, a.q_norm, a.k_norm, float(a.eps), a.freq, a.freq.shape[1],
              a.talk, meta.positions, meta.tok_req, table, table.stride(0), cache, row, k_col, kp, vp, h, g, d, v, out, gate, _is32(p), t,
              _lib.stream())
    return out, gate


def talking_attention(q: torch.Tensor, gate: Optional[torch.Tensor], a: TalkingParams, meta: HybridMeta, table: torch.Tensor,
                      cache: torch.Tensor, out: torch.Tensor) -> None:
    """q, gate: `talking_prep` of the step.  Writes the gated heads' outputs into out[:, : heads * vdim], zeros behind them."""
    t = out.shape[0]
    h, g, d, v = a.heads, a.kv_heads, a.dim, a.vdim
    row, k_col, kp, vp = talking_row(g, d, v)
    if q.shape != (h, t, g * kp) or out.shape[1] < h * v:
        raise ValueError(f"mixed queries {tuple(q.shape)} do not fit outputs {tuple(out.shape)}")
    if not q.is_cuda:
        o = R.talking_attention(q.transpose(0, 1), v, vp, g, k_col, meta.positions, meta.tok_req, table, cache, a.scale, a.chunk, a.sink)
        if gate is not None:
            o = o * torch.sigmoid(gate)[..., None]
        out[:, h * v:] = 0
        out[:, :h * v] = o.flatten(1).to(out.dtype)
        return
    shape = (row, k_col, kp, vp, h, g, v, a.chunk, float(a.scale), out, out.stride(0), out.shape[1])
    common = (q, gate, a.sink, meta.positions, meta.tok_req, table, table.stride(0), cache, *shape)
    prompt = (not _is32(q) and meta.max_span >= PROMPT_SPAN and meta.spans is not None
              and _lib.query("stk_talking_prompt_ok", h, g, kp, vp, v) == 1)
    if not prompt or meta.min_span < PROMPT_SPAN:
        max_span = PROMPT_SPAN - 1 if prompt else meta.max_span
        if _is32(q) or _lib.query("stk_talking_tokens_ok", h, g, kp, vp, max_span) == 0:
            _lib.call("stk_talking_simt", *common, _is32(q), meta.first_pos, meta.last_pos, max_span, t, _lib.stream())
        else:
            context = min(meta.max_context, table.shape[1] * PAGE)
            keys = min(a.chunk, context) if a.chunk else context
            plan = _lib.query("stk_talking_tokens_plan", t, h, g, kp, vp, max_span, keys, _lib.sm_count())
            part = scratch("talking.part", ((plan & 255) * t * h * (v + 2),), F32, q.device)
            _lib.call("stk_talking_tokens", *common, meta.query_start, meta.req_rows, meta.start_pos, meta.n_req, meta.first_pos,
                      meta.last_pos, max_span, cache.shape[0], plan, part, t, _lib.status_buffer(), _lib.stream())
    if prompt:
        n_rows = sum(_up(start + n - _rows_base(a.chunk, start), PROMPT_ROWS) for start, n in meta.spans if n >= PROMPT_SPAN)
        rows = torch.empty(n_rows, row, dtype=q.dtype, device=q.device)
        _lib.call("stk_talking_rows", meta.query_start, meta.req_rows, meta.start_pos, meta.n_req, PROMPT_SPAN, a.chunk, table, table.stride(0),
                  cache, row, rows, n_rows, _lib.stream())
        _lib.call("stk_talking_prompt", q, gate, a.sink, rows, n_rows, *shape, meta.query_start, meta.start_pos, meta.n_req,
                  PROMPT_SPAN, t, _lib.sm_count(), _lib.status_buffer(), _lib.stream())


def _rows_base(chunk: int, start: int) -> int:
    """First position whose row a long span starting at `start` gathers."""
    return start // chunk * chunk // PROMPT_ROWS * PROMPT_ROWS if chunk else 0
