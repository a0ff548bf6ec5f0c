"""Latent attention: per-token latents in a paged cache, queries brought into latent space (decoding, short spans, any size).

The cached row of a token is [normed latent | zeros | rotated key part shared by all heads | zeros] (`latent_row`).  Scores
contract a query row of the same layout, [q W_uk | rotated q], with it; the attention's read-out is in latent space too and goes
through the value expansion afterwards.  Long spans of bf16 models expand keys and values of their whole context instead and run
as ordinary attention per head.  Activations are bf16, or fp32 in a float32 model; norms, angles, scores and softmax are
fp32 in either.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from . import _lib
from . import reference as R
from . import functional as Fn
from .cache import PAGE
from .functional import LinearWeight
from .hybrid import HybridMeta, _is32
from .scratch import scratch

F32 = torch.float32

# spans of at least this many tokens expand keys and values of their context (where the kernel covers the layer)
PROMPT_SPAN = 64
# bound on the expanded keys and values of one launch; more heads than fit go one group after the other
EXPANDED_BYTES = 1 << 30
PROMPT_ROWS = 128


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def latent_row(kv_rank: int, rot_dim: int) -> Tuple[int, int]:
    """(elements of a cached row, column where the rotated part starts): both multiples of 8, so that rows and their parts
    stay 16-byte aligned in bf16."""
    off = _up(kv_rank, 8)
    return off + _up(rot_dim, 8), off


def head_pads(m) -> Tuple[int, int, int]:
    """(dp, cp, vp) of a `LatentAttentionMixer`: block-diagonal products want 64-element inputs and 128-row outputs a head."""
    return _up(m.dim, 64), _up(m.kv_rank, 128), _up(m.vdim, 128)


def split_frequencies(freq: Sequence[float], device) -> torch.Tensor:
    """[2, n] fp32: the frequencies' high parts and what those leave over."""
    f = torch.tensor(list(freq), dtype=torch.float64)
    hi = f.to(F32)
    return torch.stack([hi, (f - hi.double()).to(F32)]).contiguous().to(device)


@dataclass
class LatentParams:
    """One latent-attention layer on the device.  Head segments are padded so that block-diagonal products split on tile
    borders: dp (unrotated query part), cp (latent), vp (value)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    eps: float
    dp: int
    cp: int
    vp: int
    freq: torch.Tensor                     # [2, rot_dim / 2] (`split_frequencies`)
    q_norm: torch.Tensor                   # [q_rank] fp32
    kv_norm: Optional[torch.Tensor]        # [kv_rank] fp32; None: the layer attends over another layer's rows
    w_uq: LinearWeight                     # [heads * dp + pad(heads * rot_dim), pad(q_rank)]: unrotated parts, then rotated parts
    w_uk: LinearWeight                     # [heads * cp, dp]: per head the transposed key expansion
    w_uv: LinearWeight                     # [heads * vp, cp]: per head the value expansion
    w_ukv: Optional[LinearWeight] = None   # [heads * (dp + v64), row's latent columns]: per head key, then value expansion (prompts)


def latent_prep(p: torch.Tensor, q_off: int, kv_off: int, a: LatentParams, meta: HybridMeta, table: torch.Tensor,
                cache: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """p [T, *] fp32 holds the query latent at column q_off and, unless kv_off < 0, [latent | key part] at kv_off.  Inserts the
    tokens' rows into the paged cache [pages, PAGE, row] and returns the normed query latent [T, w_uq.in_features]."""
    t, width = p.shape[0], a.w_uq.in_features
    row, off = latent_row(a.kv_rank, a.rot_dim)
    if not p.is_cuda:
        cq = torch.zeros(t, width, dtype=dtype)
        cq[:, :a.q_rank] = R.rms_norm(p[:, q_off:q_off + a.q_rank], a.q_norm, a.eps).to(dtype)
        if kv_off >= 0:
            c = R.rms_norm(p[:, kv_off:kv_off + a.kv_rank], a.kv_norm, a.eps)
            k = R.rotate_pairs(p[:, kv_off + a.kv_rank:kv_off + a.kv_rank + a.rot_dim], meta.positions, a.freq)
            R.latent_insert(c, k, off, meta.positions, meta.tok_req, table, cache)
        return cq
    cq = torch.empty(t, width, dtype=dtype, device=p.device)
    _lib.call("stk_latent_prep", p, p.stride(0), q_off, kv_off, a.q_norm, a.kv_norm, float(a.eps), a.q_rank, width, a.kv_rank,
              a.rot_dim, meta.positions, meta.tok_req, table, table.stride(0), cache, row, off, a.freq, cq, cq.stride(0), _is32(cq),
              t, _lib.stream())
    return cq


def latent_attention(q: torch.Tensor, gate: Optional[torch.Tensor], a: LatentParams, meta: HybridMeta, table: torch.Tensor,
                     cache: torch.Tensor) -> torch.Tensor:
    """q [T, heads * dp | heads * rot_dim]: unrotated parts, then rotated parts before their rotation; gate [T, heads] fp32
    logits (None: ungated).  -> gated head outputs [T, heads * vp] (columns vdim..vp of a head are zero)."""
    t = q.shape[0]
    qc, qr = q[:, :a.heads * a.dp], q[:, a.heads * a.dp:]
    row, off = latent_row(a.kv_rank, a.rot_dim)
    if not q.is_cuda:
        qa = Fn.linear(qc, a.w_uk, groups=a.heads, tag="uk")
        o = R.latent_attention(qa.reshape(t, a.heads, a.cp)[:, :, :a.kv_rank],
                               qr[:, :a.heads * a.rot_dim].reshape(t, a.heads, a.rot_dim), off, meta.positions, meta.tok_req, table,
                               cache, a.freq, a.scale)
        if gate is not None:
            o = o * torch.sigmoid(gate.to(F32))[..., None]
        lat = torch.zeros(t, a.heads, a.cp, dtype=q.dtype)
        lat[:, :, :a.kv_rank] = o.to(q.dtype)
        return Fn.linear(lat.flatten(1), a.w_uv, groups=a.heads, tag="uv")
    spans = (meta.query_start, meta.req_rows, meta.start_pos, meta.n_req)
    prompt = a.w_ukv is not None and meta.max_span >= PROMPT_SPAN and meta.spans is not None
    if prompt and meta.min_span >= PROMPT_SPAN:
        out = torch.empty(t, a.heads * a.vp, dtype=q.dtype, device=q.device)
    else:
        qa = Fn.linear(qc, a.w_uk, groups=a.heads, tag="uk")
        lat = torch.empty(t, a.heads * a.cp, dtype=q.dtype, device=q.device)
        max_span = min(meta.max_span, PROMPT_SPAN - 1) if prompt else meta.max_span
        common = (qa, qa.stride(0), a.cp, qr, qr.stride(0), gate, gate.stride(0) if gate is not None else 0, meta.positions,
                  meta.tok_req, table, table.stride(0), cache, row, off, a.freq, a.heads, a.kv_rank, a.rot_dim, float(a.scale), lat,
                  lat.stride(0))
        if _is32(q) or _lib.query("stk_latent_tokens_columns", a.heads, a.kv_rank, row, max_span) == 0:
            _lib.call("stk_latent_attention_simt", *common, _is32(q), meta.first_pos, meta.last_pos, max_span, t, _lib.stream())
        else:
            splits = _lib.query("stk_latent_tokens_splits", t, a.heads, max_span, min(meta.max_context, table.shape[1] * PAGE),
                                _lib.sm_count())
            part = scratch("latent.part", (splits * t * a.heads * (a.kv_rank + 2),), F32, q.device)
            _lib.call("stk_latent_tokens", *common, *spans, meta.first_pos, meta.last_pos, max_span, cache.shape[0], splits, part, t,
                      _lib.status_buffer(), _lib.stream())
        out = Fn.linear(lat, a.w_uv, groups=a.heads, tag="uv")
    if prompt:
        n_rows = sum(_up(start + n, PROMPT_ROWS) for start, n in meta.spans if n >= PROMPT_SPAN)
        rows = meta.gathered.get(cache.data_ptr())
        if rows is None:
            rows = torch.empty(n_rows, row, dtype=q.dtype, device=q.device)
            _lib.call("stk_latent_rows", *spans, PROMPT_SPAN, table, table.stride(0), cache, 1, row, rows, n_rows, _lib.stream())
            meta.gathered.clear()
            meta.gathered[cache.data_ptr()] = rows
        width = a.w_ukv.out_features // a.heads
        group = max(1, min(a.heads, EXPANDED_BYTES // (2 * n_rows * width)))
        for h0 in range(0, a.heads, group):
            nh = min(group, a.heads - h0)
            kv = Fn.linear(rows[:, :off], LinearWeight(a.w_ukv.w[h0 * width:(h0 + nh) * width]), tag="ukv")
            _lib.call("stk_latent_prompt", qc, qc.stride(0), qr, qr.stride(0), gate, gate.stride(0) if gate is not None else 0,
                      meta.query_start, meta.start_pos, meta.n_req, PROMPT_SPAN, rows, n_rows, row, off, kv, a.freq, a.heads, h0, nh,
                      a.dim, a.dp, a.rot_dim, a.vdim, a.vp, float(a.scale), out, out.stride(0), t, _lib.status_buffer(),
                      _lib.stream())
    return out


def prompt_ok(m) -> bool:
    """Whether long spans of a `LatentAttentionMixer` can run on the prompt kernel."""
    row, off = latent_row(m.kv_rank, m.rot_dim)
    return _lib.query("stk_latent_prompt_ok", m.dim, head_pads(m)[0], m.rot_dim, m.vdim, row, off) == 1
