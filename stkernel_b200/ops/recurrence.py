"""Linear recurrences S <- a S + k v^T, o = S^T q (state fp32).  With a scalar decay per head and token: retention (fixed decay, rotated
queries and keys) and Mamba-2 (decay and input weight from a step size, operands behind a short causal convolution).  With a decay
per key channel and a bonus for the current token: time mixing.

Short spans and float32 models run token by token (`*_scan`); longer spans of bf16 models in chunks on the tensor cores
(`stk_linear_chunks`, common to both).  What enters the recurrence in fp32 (rotated queries and keys, decays, weighted values, the
state) meets the tensor cores as bf16 pairs, high part and remainder.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from . import reference as R
from .functional import cpu_act_dtype
from .hybrid import HybridMeta, _is32, out_offset
from .scratch import scratch

BF16 = torch.bfloat16
F32 = torch.float32

# spans of at least this many tokens run in chunks (bf16 models)
CHUNK_SPAN = 24
CHUNK = 64


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def _chunked(t: torch.Tensor, meta: HybridMeta, dim: int) -> bool:
    return not _is32(t) and meta.max_span >= CHUNK_SPAN and dim <= 256


def _chunks(qk, v: torch.Tensor, v_off: int, heads_per_group: int, log_decay, per_token, skip, meta: HybridMeta, S: torch.Tensor,
            o: torch.Tensor) -> None:
    """qk: (q high, q remainder or None, k high, k remainder or None, row stride, head stride, columns), column views of one matrix.
    log_decay [H] fixed, or per_token = (log decay [H, T], input weight [H, T])."""
    qh, ql, kh, kl, ld, step, width = qk
    t, (_, h, d, vd) = v.shape[0], S.shape
    chunks = t // CHUNK + meta.n_req
    ws = scratch("scan.states", (chunks * h * _lib.query("stk_linear_state_slot", d, vd),), F32, v.device)
    g, w = per_token if per_token is not None else (None, None)
    _lib.call("stk_linear_chunks", qh, ql, kh, kl, ld, step, width, heads_per_group, v, v.stride(0), v_off, log_decay, g, w, skip,
              meta.query_start, meta.req_rows, meta.start_pos, meta.n_req, S, o, h, d, vd, CHUNK_SPAN, ws, chunks, t, _lib.stream())


# ----------------------------------------------------------------------------
# retention
# ----------------------------------------------------------------------------
@dataclass
class RetentionParams:
    heads: int
    dim: int
    vdim: int
    log_decay: torch.Tensor        # [heads] fp32
    decay: torch.Tensor            # [2, heads] fp32: the decays and what their rounding leaves over
    freq: torch.Tensor             # [2, pairs] (`latent.split_frequencies`): dimension i turns with i + pairs
    eps: float
    out_scale: float


def retention(p: torch.Tensor, q_off: int, k_off: int, v_off: int, g_off: int, a: RetentionParams, meta: HybridMeta,
              state: Tuple[torch.Tensor], out: torch.Tensor, left: int) -> None:
    """Runs the step's tokens through the recurrence (state updated) and writes norm(o) * silu(g) * out_scale into `out` from column
    col = out_offset(left) on, zeros into the columns left .. col and behind the output (another mixer owns the columns below
    `left`)."""
    t = p.shape[0]
    h, d, v, col = a.heads, a.dim, a.vdim, out_offset(left)
    S, = state
    scale = d ** -0.5
    if not p.is_cuda:
        seg = lambda o, w: p[:, o:o + h * w].reshape(t, h, w)
        q = R.rotate_half_split(seg(q_off, d), meta.positions, a.freq)
        k = R.rotate_half_split(seg(k_off, d), meta.positions, a.freq) * scale
        o = R.unit_rms(R.linear_scan(q, k, seg(v_off, v), a.log_decay.expand(t, -1), meta.tok_req, meta.positions, S), a.eps)
        g = p[:, g_off:g_off + h * v].to(F32)
        out[:, left:] = 0
        out[:, col:col + h * v] = (o.flatten(1) * torch.nn.functional.silu(g) * a.out_scale).to(out.dtype)
        return
    o = scratch("scan.out", (t, h * v), F32, p.device)
    pairs = a.freq.shape[1]
    chunked = _chunked(p, meta, d)
    if not chunked or meta.min_span < CHUNK_SPAN:
        _lib.call("stk_retention_scan", p, p.stride(0), q_off, k_off, v_off, a.freq, pairs, scale, a.decay, meta.query_start,
                  meta.req_rows, meta.start_pos, meta.n_req, S, o, h, d, v, _is32(p), 1, (CHUNK_SPAN - 1) if chunked else 1 << 30, t,
                  _lib.stream())
    if chunked:
        d8 = _up8(d)
        rot = scratch("scan.rotated", (t, 4, h * d8), BF16, p.device)
        _lib.call("stk_rotate_qk", p, p.stride(0), q_off, k_off, a.freq, pairs, scale, meta.positions, rot, h, d, d8, t, _lib.stream())
        _chunks((rot[:, 0], rot[:, 1], rot[:, 2], rot[:, 3], 4 * h * d8, d8, d8), p, v_off, 1, a.log_decay, None, None, meta, S, o)
    _lib.call("stk_retention_finish", o, float(a.eps), None, meta.tok_req, meta.positions, p, p.stride(0), g_off, float(a.out_scale), out,
              out.stride(0), left, col, out.shape[1], _is32(p), h, v, t, _lib.stream())


# ----------------------------------------------------------------------------
# time mixing
# ----------------------------------------------------------------------------
@dataclass
class TimeMixParams:
    heads: int
    dim: int
    np: int                        # columns of a projection (heads * dim, padded)
    w0: torch.Tensor               # [heads * dim] fp32: added to the decay's projection
    bonus: torch.Tensor            # [heads * dim] fp32
    norm: torch.Tensor             # [heads * dim] fp32
    eps: float


def tanh_pair(device) -> bool:
    """Whether a bf16 model on this device takes tanh as high part and remainder (the CPU path of a model with bf16 weights does so
    only when its activations are bf16 as well)."""
    return torch.device(device).type == "cuda" or cpu_act_dtype() == BF16


def tanh_rows(z: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """tanh(z [T, n] fp32): [T, n] in fp32 models; in bf16 models its high part and remainder side by side, [T, 2 n]."""
    t, n = z.shape
    pair = dtype == BF16
    if not z.is_cuda:
        y = torch.tanh(z)
        hi = y.to(dtype)
        return torch.cat([hi, (y - hi.to(F32)).to(dtype)], 1) if pair else y
    out = torch.empty(t, 2 * n if pair else n, dtype=dtype, device=z.device)
    _lib.call("stk_tanh_rows", z, z.stride(0), n, out, _is32(out), t, _lib.stream())
    return out


def time_mix(p: torch.Tensor, z: torch.Tensor, a: TimeMixParams, meta: HybridMeta, state: Tuple[torch.Tensor], out: torch.Tensor) -> None:
    """p [T, 4 * np]: r, k, v and the gate as projected; z [T, >= heads * dim] fp32: the decay's projection, log w = -exp(z + w0).
    Runs the step's tokens through the recurrence (state updated) and writes norm(o) * weight * silu(gate) into
    out[:, : heads * dim], zeros behind it."""
    t = p.shape[0]
    h, d, n = a.heads, a.dim, a.heads * a.dim
    S, = state
    if not p.is_cuda:
        r, k, v = (p[:, i * a.np:i * a.np + n].reshape(t, h, d) for i in range(3))
        log_decay = -torch.exp(z[:, :n] + a.w0).view(t, h, d)
        o = R.bonus_scan(r, k, v, log_decay, a.bonus.view(h, d), meta.tok_req, meta.positions, S)
        gate = torch.nn.functional.silu(p[:, 3 * a.np:3 * a.np + n].to(F32))
        out[:, n:] = 0
        out[:, :n] = (R.unit_rms(o, a.eps).flatten(1) * a.norm * gate).to(out.dtype)
        return
    o = scratch("scan.out", (t, n), F32, p.device)
    chunked = not _is32(p) and meta.max_span >= CHUNK_SPAN and _lib.query("stk_time_mix_chunks_ok", d) == 1
    if not chunked or meta.min_span < CHUNK_SPAN:
        _lib.call("stk_time_mix_scan", p, p.stride(0), a.np, z, z.stride(0), a.w0, a.bonus, meta.query_start, meta.req_rows, meta.start_pos,
                  meta.n_req, S, o, h, d, _is32(p), 1, (CHUNK_SPAN - 1) if chunked else 1 << 30, t, _lib.stream())
    if chunked:
        chunks = t // CHUNK + meta.n_req
        keys = scratch("scan.rotated", (t, 2, h * _up8(d)), BF16, p.device)
        channel = scratch("scan.channel", (chunks, h, d), F32, p.device)
        ws = scratch("scan.states", (chunks * h * _lib.query("stk_linear_state_slot", d, d),), F32, p.device)
        _lib.call("stk_time_mix_chunks", p, p.stride(0), a.np, z, z.stride(0), a.w0, a.bonus, meta.query_start, meta.req_rows, meta.start_pos,
                  meta.n_req, S, o, h, d, CHUNK_SPAN, keys, channel, ws, chunks, t, _lib.stream())
    _lib.call("stk_retention_finish", o, float(a.eps), a.norm, meta.tok_req, meta.positions, p, p.stride(0), 3 * a.np, 1.0, out, out.stride(0),
              0, 0, out.shape[1], _is32(p), h, d, t, _lib.stream())


# ----------------------------------------------------------------------------
# Mamba-2
# ----------------------------------------------------------------------------
@dataclass
class Mamba2Params:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: torch.Tensor             # [taps, channels] fp32, the current token's last
    conv_bias: torch.Tensor        # [channels] fp32
    dt_bias: torch.Tensor          # [heads] fp32
    neg_a: torch.Tensor            # [heads] fp32: -exp(A_log)
    skip: torch.Tensor             # [heads] fp32
    norm: torch.Tensor             # [heads * vdim] fp32
    eps: float


def mamba2(p: torch.Tensor, z_off: int, x_off: int, dt_off: int, a: Mamba2Params, meta: HybridMeta,
           state: Tuple[torch.Tensor, torch.Tensor], out: torch.Tensor) -> None:
    """p holds z at column z_off, (x | B | C) at x_off and dt at dt_off.  Runs the step's tokens (state and convolution inputs
    updated) and writes the gated, normed output into out[:, : heads * vdim], zeros behind it."""
    t = p.shape[0]
    h, v, n, g = a.heads, a.vdim, a.state, a.groups
    inner, cd, taps = h * v, h * v + 2 * g * n, a.taps.shape[0]
    S, ring = state
    if not p.is_cuda:
        raw = p[:, x_off:x_off + cd]
        c = R.causal_conv(raw, a.taps.t(), a.conv_bias, meta.tok_req, meta.positions, meta.first_pos, ring)
        c = torch.nn.functional.silu(c).to(p.dtype).to(F32)
        x, B, C = c[:, :inner].view(t, h, v), c[:, inner:inner + g * n].view(t, g, n), c[:, inner + g * n:].view(t, g, n)
        dt = torch.nn.functional.softplus(p[:, dt_off:dt_off + h].to(F32) + a.dt_bias, threshold=60.0)
        B, C = B.repeat_interleave(h // g, 1), C.repeat_interleave(h // g, 1)
        y = R.linear_scan(C, B * dt[..., None], x, dt * a.neg_a, meta.tok_req, meta.positions, S) + a.skip[:, None] * x
        y = y.flatten(1) * torch.nn.functional.silu(p[:, z_off:z_off + inner].to(F32))
        y = R.unit_rms(y.view(t, a.norm_groups, -1), a.eps).view(t, inner) * a.norm
        if taps > 1:
            R.keep_conv_inputs(raw, meta.tok_req, meta.positions, meta.last_pos, ring)
        out[:, inner:] = 0
        out[:, :inner] = y.to(out.dtype)
        return
    o = scratch("scan.out", (t, inner), F32, p.device)
    chunked = _chunked(p, meta, n)
    ld = _up8(cd)
    xbc = scratch("scan.xbc", (t, ld), p.dtype, p.device)
    step = scratch("scan.steps", (2, h, t), F32, p.device)
    _lib.call("stk_mamba2_conv", p, p.stride(0), x_off, dt_off, a.taps, a.conv_bias, taps, ring, a.dt_bias, a.neg_a, meta.positions,
              meta.tok_req, meta.first_pos, xbc, ld, step, h, cd, _is32(p), t, _lib.stream())
    if not chunked or meta.min_span < CHUNK_SPAN:
        _lib.call("stk_mamba2_scan", xbc, ld, step, a.skip, meta.query_start, meta.req_rows, meta.start_pos, meta.n_req, S, o, h, n, v, g,
                  _is32(p), 1, (CHUNK_SPAN - 1) if chunked else 1 << 30, t, _lib.stream())
    if chunked:
        _chunks((xbc[:, inner + g * n:], None, xbc[:, inner:], None, ld, n, n), xbc, 0, h // g, None, (step[0], step[1]), a.skip, meta,
                S, o)
    _lib.call("stk_mamba2_finish", o, p, p.stride(0), z_off, x_off, cd, a.norm, float(a.eps), a.norm_groups, meta.tok_req,
              meta.positions, meta.last_pos, ring, taps, out, out.stride(0), out.shape[1], _is32(p), inner, t, _lib.stream())
