"""Grouped-query attention over the full context: keys and values of their own sizes, optional projection biases, unit-RMS queries and
keys, a query temperature that grows with the position, a null sink in the softmax, and an element-wise output gate.

The cached row of a token and key/value head is [value | zeros | key | zeros], both parts on 16-element borders (`grouped_row`): the
kernels of windowed attention (`csrc/window_attention.cu`) contract the key columns and sum the value columns of one row.  Long
spans of bf16 models gather their context's rows and run on the prompt kernel that latent attention uses as well.
Activations are bf16, or fp32 in a float32 model; norms, temperature, scores, softmax and gate are fp32 in either.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from . import reference as R
from .cache import PAGE
from .hybrid import ATTN_TOKEN_SPAN, HybridMeta, _is32
from .latent import PROMPT_ROWS, PROMPT_SPAN, _up
from .scratch import scratch

F32 = torch.float32
WHOLE = 1 << 30              # window of a kernel that sees every earlier position


def grouped_row(dim: int, vdim: int) -> Tuple[int, int]:
    """(elements of a cached row, column where the key starts)."""
    return _up(vdim, 16) + _up(dim, 16), _up(vdim, 16)


@dataclass
class GroupedParams:
    """One layer on the device."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias: Optional[torch.Tensor]           # fp32 [heads * dim | kv_heads * dim | kv_heads * vdim]
    eps: Optional[float]                   # unit-RMS queries and keys; None: as projected
    temp: Tuple[float, float]              # (coef, every); coef 0: none
    sink: Optional[torch.Tensor]           # fp32 [heads] scores without a value
    gated: bool
    out_scale: float                       # the output (after the gate) times this


def grouped_prep(p: torch.Tensor, q_off: int, k_off: int, v_off: int, a: GroupedParams, meta: HybridMeta, table: torch.Tensor,
                 cache: torch.Tensor) -> torch.Tensor:
    """Inserts the tokens' rows into the paged cache; -> queries [T, heads * pad(dim)] ready for the scores."""
    t = p.shape[0]
    h, g, d, v = a.heads, a.kv_heads, a.dim, a.vdim
    dp = _up(d, 64)
    row, k_col = grouped_row(d, v)
    if not p.is_cuda:
        b = a.bias if a.bias is not None else torch.zeros(h * d + g * (d + v))
        q = (p[:, q_off:q_off + h * d].to(F32) + b[:h * d]).reshape(t, h, d)
        k = (p[:, k_off:k_off + g * d].to(F32) + b[h * d:(h + g) * d]).reshape(t, g, d)
        vv = (p[:, v_off:v_off + g * v].to(F32) + b[(h + g) * d:]).reshape(t, g, v)
        if a.eps is not None:
            q, k = R.unit_rms(q, a.eps), R.unit_rms(k, a.eps)
        q = q * R.query_temperature(meta.positions, *a.temp)[:, None, None]
        R.grouped_kv_insert(k, vv, k_col, meta.positions, meta.tok_req, table, cache)
        out = torch.zeros(t, h, dp, dtype=p.dtype)
        out[:, :, :d] = q.to(p.dtype)
        return out.flatten(1)
    out = torch.empty(t, h * dp, dtype=p.dtype, device=p.device)
    _lib.call("stk_grouped_prep", p, p.stride(0), q_off, k_off, v_off, a.bias, 1 if a.eps is not None else 0, float(a.eps or 0.0),
              float(a.temp[0]), float(a.temp[1]), meta.positions, meta.tok_req, table, table.stride(0), cache, row, k_col, h, g, d, v,
              out, dp, _is32(p), t, _lib.stream())
    return out


def grouped_attention(p: torch.Tensor, q: torch.Tensor, g_off: int, a: GroupedParams, meta: HybridMeta, table: torch.Tensor,
                      cache: torch.Tensor, out: torch.Tensor) -> None:
    """q: `grouped_prep` of the step's projections p, whose column g_off starts the gate.  Writes the gated and scaled heads'
    outputs into out[:, : heads * vdim]."""
    t = p.shape[0]
    h, g, d, v = a.heads, a.kv_heads, a.dim, a.vdim
    dp = _up(d, 64)
    row, k_col = grouped_row(d, v)
    if not p.is_cuda:
        o = R.grouped_attention(q.view(t, h, dp)[:, :, :d], v, k_col, meta.positions, meta.tok_req, table, cache, a.scale,
                                a.sink is not None).flatten(1) * a.out_scale
        if a.gated:
            o = o * torch.sigmoid(p[:, g_off:g_off + h * v].to(F32))
        out[:, :h * v] = o.to(out.dtype)
        return
    gate = p[:, g_off:] if a.gated else None
    ldg = p.stride(0) if a.gated else 0
    common = (q, q.stride(0), 0, 0, meta.positions, meta.tok_req, table, table.stride(0), cache, row, None, 0, 1.0, h, g, d)
    tail = (k_col, v, dp, gate, ldg, float(a.out_scale), WHOLE, float(a.scale), 0.0, a.sink, out, out.stride(0))
    if _is32(p) or _lib.query("stk_window_attention_mma_ok", h, g, d, v, k_col, row) != 1:
        _lib.call("stk_window_attention_simt", *common, *tail, _is32(p), t, _lib.stream())
        return
    spans = (meta.query_start, meta.req_rows, meta.start_pos, meta.n_req)
    prompt = meta.max_span >= PROMPT_SPAN and meta.spans is not None and _lib.query("stk_prompt_attention_ok", d, dp, v, row, k_col) == 1
    token_span = ATTN_TOKEN_SPAN if meta.max_span > ATTN_TOKEN_SPAN else meta.max_span
    if meta.min_span <= token_span:
        keys = min(WHOLE, meta.max_context, table.shape[1] * PAGE)
        splits = _lib.query("stk_window_attention_splits", t, h, g, keys, _lib.sm_count())
        part = scratch("wattn.part", (splits * t * h * (v + 2),), F32, p.device) if splits > 1 else None
        _lib.call("stk_window_attention_tokens", *common, *tail, meta.first_pos, meta.last_pos, token_span, splits, part, t,
                  _lib.stream())
    if meta.max_span > token_span and not (prompt and meta.min_span >= PROMPT_SPAN):
        _lib.call("stk_window_attention_tiles", *common, *tail, *spans, token_span + 1, PROMPT_SPAN - 1 if prompt else 1 << 30, t,
                  _lib.stream())
    if prompt:
        n_rows = sum(_up(start + n, PROMPT_ROWS) for start, n in meta.spans if n >= PROMPT_SPAN)
        rows = torch.empty(n_rows, g * row, dtype=q.dtype, device=q.device)
        _lib.call("stk_latent_rows", *spans, PROMPT_SPAN, table, table.stride(0), cache, g, row, rows, n_rows, _lib.stream())
        _lib.call("stk_prompt_attention", q, q.stride(0), meta.query_start, meta.start_pos, meta.n_req, PROMPT_SPAN, rows, n_rows, row,
                  k_col, gate, ldg, float(a.out_scale), a.sink, h, g, d, dp, v, float(a.scale), out, out.stride(0), t,
                  _lib.status_buffer(), _lib.stream())
