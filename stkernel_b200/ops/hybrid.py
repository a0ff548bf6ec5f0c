"""Ops of the layer-by-layer decoders: scaled embedding, add + norm and norm + add on an fp32 residual, residual streams, paged windowed
attention whose values are the unrotated keys, mLSTM recurrence, and the parallel block's joined sublayer outputs.  (Latent attention:
`ops/latent.py`; grouped attention: `ops/grouped.py`; retention and Mamba-2: `ops/recurrence.py`; experts: `ops/moe.py`.)

Activations are bf16, or fp32 in a float32 model (every kernel here has both forms; the fp32 forms use no reduced-precision
products).  Residual, norms, scores and softmax, gates and recurrent state are fp32 in either.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple

import torch

from . import _lib
from . import reference as R
from .cache import PAGE
from .functional import cpu_act_dtype
from .scratch import scratch

BF16 = torch.bfloat16
F32 = torch.float32

# spans of at most this many tokens are attended token by token (the kernel of decode steps); longer ones in query tiles
ATTN_TOKEN_SPAN = 4
# spans of at least this many tokens take the tcgen05 kernel where its sizes allow
ATTN_TC_SPAN = 64
# spans of at least this many tokens run the recurrence in chunks on the tensor cores (bf16 models)
MLSTM_CHUNK_SPAN = 24
MLSTM_CHUNK = 64


def act_dtype(dtype: str, device) -> torch.dtype:
    if dtype == "float32":
        return F32
    return BF16 if torch.device(device).type == "cuda" else cpu_act_dtype()


def _is32(t: torch.Tensor) -> int:
    return 1 if t.dtype == F32 else 0


# ----------------------------------------------------------------------------
# residual
# ----------------------------------------------------------------------------
def embed_scaled(ids: torch.Tensor, embed: torch.Tensor, scale: float, h: Optional[torch.Tensor] = None,
                 streams: Optional[int] = None) -> torch.Tensor:
    """ids [T] -> fp32 residual [T, W] = embed[id] * scale.  h [T, width]: receives the rows in the compute type as well,
    zero-padded.  streams: that many equal copies, [T, streams, W]."""
    t, w = ids.shape[0], embed.shape[1]
    if not ids.is_cuda:
        ok = (ids >= 0) & (ids < embed.shape[0])
        x = torch.where(ok[:, None], embed[ids.clamp(0, embed.shape[0] - 1)].to(F32) * scale, torch.zeros(1))
        if h is not None:
            h.zero_()
            h[:, :w] = x.to(h.dtype)
        return x if streams is None else x[:, None].repeat(1, streams, 1)
    n = streams or 1
    x = torch.empty(t, n * w, dtype=F32, device=ids.device)
    _lib.call("stk_embed_scaled", ids, embed, _is32(embed), x, n * w, n, t, w, embed.shape[0], float(scale), h,
              h.stride(0) if h is not None else 0, h.shape[1] if h is not None else 0, _lib.status_buffer(), _lib.stream())
    return x if streams is None else x.view(t, n, w)


@dataclass
class StreamWeights:
    """How one sublayer reads and writes the residual streams (fp32): u = sum_s read[s] x_s before, x_t <- sum_s mix[s, t] x_s +
    write[t] y after it."""
    read: torch.Tensor             # [s]
    write: torch.Tensor            # [s]
    mix: torch.Tensor              # [s, s], [from, to]


def expert_sum(y, w_n: int) -> torch.Tensor:
    """CPU: fp32 rows [T, W] of a sublayer's output (`ExpertRows`: the weighted sum over each token's pairs)."""
    if isinstance(y, torch.Tensor):
        return y
    t, k = y.weights.shape
    at = y.pair_row.long() if y.pair_row is not None else torch.arange(t * k)
    return (y.y[at].to(F32).view(t, k, -1)[..., :w_n] * y.weights[..., None]).sum(1)


def stream_norm(x: torch.Tensor, y, after: Optional[StreamWeights], read: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float,
                width: int, dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Streams x [T, s, W] fp32: the previous sublayer's output y (fp32 rows or `ExpertRows`; None: nothing to add) goes into them as
    `after` says, in place, then the layer norm (weight w, bias b) of sum_s read[s] x_s in `dtype`, zero-padded to `width` columns.
    rows: only these rows are normed, and the streams are not written back."""
    t, s, w_n = x.shape
    if not x.is_cuda:
        if y is not None:
            y = expert_sum(y, w_n)[:, :w_n]
            new = R.stream_mix(x if rows is None else x[rows], y if rows is None else y[rows], after.mix, after.write)
            if rows is None:
                x.copy_(new)
        else:
            new = x if rows is None else x[rows]
        h = torch.zeros(new.shape[0], width, dtype=dtype)
        h[:, :w_n] = (R.layer_norm(torch.einsum("s,tsw->tw", read, new), w, eps) + b).to(dtype)
        return h
    n = t if rows is None else rows.shape[0]
    h = torch.empty(n, width, dtype=dtype, device=x.device)
    pairs = y if y is not None and not isinstance(y, torch.Tensor) else None
    plain = y if pairs is None else None
    _lib.call("stk_stream_norm", x, s, plain, plain.stride(0) if plain is not None else 0, pairs.y if pairs is not None else None,
              pairs.y.stride(0) if pairs is not None else 0, pairs.pair_row if pairs is not None else None,
              pairs.weights if pairs is not None else None, pairs.weights.shape[1] if pairs is not None else 0,
              after.mix if y is not None else None, after.write if y is not None else None, read, w, b, float(eps), h, h.stride(0), w_n,
              width, _is32(h), rows, n, _lib.stream())
    return h


def add_layer_norm(x: torch.Tensor, y: Optional[torch.Tensor], w: torch.Tensor, eps: float, width: int, dtype: torch.dtype,
                   rows: Optional[torch.Tensor] = None, center: bool = True) -> torch.Tensor:
    """x += y (fp32, in place; y None: nothing to add), then the layer norm of x in `dtype`, zero-padded to `width` columns.
    rows: only these rows are normed (and the addition is not written back).  center False: RMS norm."""
    w_n = x.shape[1]
    if not x.is_cuda:
        if rows is not None:
            x = x[rows]
            x = x + y[rows] if y is not None else x
        elif y is not None:
            x += y
        h = torch.zeros(x.shape[0], width, dtype=dtype)
        h[:, :w_n] = (R.layer_norm if center else R.rms_norm)(x, w, eps).to(dtype)
        return h
    t = x.shape[0] if rows is None else rows.shape[0]
    h = torch.empty(t, width, dtype=dtype, device=x.device)
    _lib.call("stk_add_layer_norm", x, x.stride(0), y, y.stride(0) if y is not None else 0, w, h, _is32(h), width, t, w_n, width,
              float(eps), rows, 1 if center else 0, _lib.stream())
    return h


def post_norm_add(x: torch.Tensor, y, w: torch.Tensor, eps: float, width: int, dtype: torch.dtype) -> torch.Tensor:
    """x += rms_norm(y) * w (fp32, in place) -> x in `dtype`, zero-padded to `width` columns.  y: fp32 [T, W], or `ExpertRows`
    whose weighted sum over each token's pairs is normed."""
    t, w_n = x.shape
    rows = None if isinstance(y, torch.Tensor) else y
    if not x.is_cuda:
        x += R.rms_norm(expert_sum(y, w_n), w, eps)
        h = torch.zeros(t, width, dtype=dtype)
        h[:, :w_n] = x.to(dtype)
        return h
    h = torch.empty(t, width, dtype=dtype, device=x.device)
    common = (w, float(eps), h, h.stride(0), w_n, width, _is32(h), t, _lib.stream())
    if rows is None:
        _lib.call("stk_post_norm_add", x, x.stride(0), y, y.stride(0), None, 0, None, None, 0, *common)
    else:
        _lib.call("stk_post_norm_add", x, x.stride(0), None, 0, rows.y, rows.y.stride(0), rows.pair_row, rows.weights,
                  rows.weights.shape[1], *common)
    return h


# ----------------------------------------------------------------------------
# step description
# ----------------------------------------------------------------------------
@dataclass
class HybridMeta:
    """Device-side description of one ragged step (decode rows and prompt portions alike)."""
    token_ids: torch.Tensor        # [T] int64
    tok_req: torch.Tensor          # [T] int32 request row, -1 padding
    positions: torch.Tensor        # [T] int64, -1 padding
    first_pos: torch.Tensor        # [T] int32 first position of the token's span in this step
    last_pos: torch.Tensor         # [T] int32
    query_start: torch.Tensor      # [n_req + 1] int32
    req_rows: torch.Tensor         # [n_req] int32
    start_pos: torch.Tensor        # [n_req] int32
    n_req: int
    max_span: int                  # longest span of the step (host knowledge: which kernels have work)
    pure_decode: bool = False      # every span is one token
    min_span: int = 1
    spans: Optional[Tuple[Tuple[int, int], ...]] = None      # (start, tokens) of every request, when the host knows them
    gathered: dict = field(default_factory=dict)             # cached rows that a layer copied out of their pages for this step
    max_context: int = 1 << 30     # no token of the step sees more keys (host knowledge: how far to split the key range)


# ----------------------------------------------------------------------------
# windowed attention
# ----------------------------------------------------------------------------
@dataclass
class AttentionParams:
    """Constants of one attention layer on the device."""
    heads: int
    kv_heads: int
    dim: int
    window: int
    scale: float
    softcap: float
    freq: torch.Tensor             # [rot_dims / 2] fp32 radians per position
    mag: float
    sink: Optional[torch.Tensor]   # [heads] fp32


def window_attention(proj: torch.Tensor, q_off: int, k_off: int, a: AttentionParams, meta: HybridMeta, table: torch.Tensor,
                     cache: torch.Tensor, out: torch.Tensor) -> None:
    """proj [T, *] holds q at column q_off and k at k_off.  Inserts the tokens' rows into the paged cache and writes the
    attention output of every token into out[:, : heads * dim] (a view of the joined sublayer buffer)."""
    t = proj.shape[0]
    h, g, d = a.heads, a.kv_heads, a.dim
    if not proj.is_cuda:
        q = proj[:, q_off:q_off + h * d].reshape(t, h, d)
        k = proj[:, k_off:k_off + g * d].reshape(t, g, d)
        R.window_kv_insert(k, meta.positions, meta.tok_req, table, cache, a.freq, a.mag)
        o = R.window_attention(q, meta.positions, meta.tok_req, table, cache, a.freq, a.mag, a.window, a.scale, a.softcap,
                               a.sink)
        out[:, :h * d] = o.flatten(1).to(out.dtype)
        return
    rd = 2 * a.freq.numel()
    common = (proj, proj.stride(0), q_off, k_off, meta.positions, meta.tok_req, table, table.stride(0), cache, cache.shape[3],
              a.freq, rd, float(a.mag), h, g, d)
    _lib.call("stk_window_kv_insert", *common, _is32(proj), t, _lib.stream())
    tail = (a.window, float(a.scale), float(a.softcap), a.sink, out, out.stride(0))
    rows = (rd, d, d, None, 0, 1.0)                      # scores from column rd, values as wide as keys, dense queries, no gate
    if _is32(proj) or d > 256 or cache.shape[3] % 8:
        _lib.call("stk_window_attention_simt", *common, *rows, *tail, _is32(proj), t, _lib.stream())
        return
    token_span = ATTN_TOKEN_SPAN if meta.max_span > ATTN_TOKEN_SPAN else meta.max_span
    if meta.min_span <= token_span:
        splits = _lib.query("stk_window_attention_splits", t, h, g, a.window, _lib.sm_count())
        part = scratch("wattn.part", (splits * t * h * (d + 2),), F32, proj.device) if splits > 1 else None
        _lib.call("stk_window_attention_tokens", *common, *rows, *tail, meta.first_pos, meta.last_pos, token_span, splits, part, t,
                  _lib.stream())
    spans = (meta.query_start, meta.req_rows, meta.start_pos, meta.n_req)
    tc = (meta.max_span >= ATTN_TC_SPAN and out.stride(0) % 8 == 0
          and _lib.query("stk_window_attention_tc_ok", h, g, d, rd, cache.shape[3]) == 1)
    if meta.max_span > token_span and not (tc and meta.min_span >= ATTN_TC_SPAN):
        _lib.call("stk_window_attention_tiles", *common, *rows, *tail, *spans, token_span + 1, ATTN_TC_SPAN - 1 if tc else 1 << 30, t,
                  _lib.stream())
    if tc:
        _lib.call("stk_window_attention_tc", *common, *tail, *spans, ATTN_TC_SPAN, cache.shape[0], t, _lib.status_buffer(),
                  _lib.stream())


# ----------------------------------------------------------------------------
# mLSTM
# ----------------------------------------------------------------------------
@dataclass
class MlstmParams:
    heads: int
    dim: int
    vdim: int
    cap: float
    gate_bias: torch.Tensor        # [2 * heads] fp32: input gates, forget gates
    norm: torch.Tensor             # [heads * vdim] fp32
    eps: float


def mlstm(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, g_off: int, gates: torch.Tensor, p: MlstmParams,
          meta: HybridMeta, state: Tuple[torch.Tensor, torch.Tensor, torch.Tensor], out: torch.Tensor,
          glu: Optional[Tuple[int, int, int]]) -> None:
    """Runs the step's tokens through the recurrence (state updated) and writes norm(o) * sigmoid(g) into
    out[:, : heads * vdim].  gates [T, 2 * heads] fp32 projections.  glu: see `join_glu` (done by the same launch)."""
    t = proj.shape[0]
    h, d, v = p.heads, p.dim, p.vdim
    S, n, m = state
    if not proj.is_cuda:
        seg = lambda o, w: proj[:, o:o + h * w].reshape(t, h, w)
        o = R.mlstm_scan(seg(q_off, d), seg(k_off, d), seg(v_off, v), gates, p.gate_bias, p.cap, meta.tok_req, meta.first_pos,
                         meta.positions, S, n, m)
        out[:, :h * v] = R.head_norm_gate(o, p.norm, proj[:, g_off:g_off + h * v], p.eps).to(out.dtype)
        join_glu(proj, out, h * v, glu)
        return
    dev = proj.device
    num = scratch("mlstm.num", (t, h * v), F32, dev)
    den = scratch("mlstm.den", (t, h), F32, dev)
    mt = scratch("mlstm.m", (t, h), F32, dev)
    chunked = not _is32(proj) and meta.max_span >= MLSTM_CHUNK_SPAN and d <= 256
    args = (proj, proj.stride(0), q_off, k_off, v_off, gates, p.gate_bias, float(p.cap), meta.query_start, meta.req_rows,
            meta.start_pos, meta.n_req, S, n, m, num, den, mt, h, d, v)
    if not chunked or meta.min_span < MLSTM_CHUNK_SPAN:
        _lib.call("stk_mlstm_scan", *args, _is32(proj), 1, (MLSTM_CHUNK_SPAN - 1) if chunked else 1 << 30, t, _lib.stream())
    if chunked:
        L = MLSTM_CHUNK
        chunks = t // L + meta.n_req
        a_ws = scratch("mlstm.gates", (chunks * h * _lib.query("stk_mlstm_gate_slot"),), F32, dev)
        u_ws = scratch("mlstm.states", (chunks * h * _lib.query("stk_mlstm_state_slot", d, v),), F32, dev)
        _lib.call("stk_mlstm_chunks", *args, MLSTM_CHUNK_SPAN, a_ws, u_ws, chunks, t, _lib.stream())
    go, uo, ff = glu if glu is not None else (0, 0, 0)
    _lib.call("stk_mlstm_finish", num, den, mt, m, p.norm, float(p.eps), meta.tok_req, meta.positions, meta.last_pos, proj,
              proj.stride(0), g_off, out, out.stride(0), _is32(proj), h, v, go, uo, ff, out_offset(h * v), out.shape[1], t,
              _lib.stream())


def out_offset(mixer_dim: int) -> int:
    """Column of the joined sublayer buffer where the feed-forward activation starts."""
    return (mixer_dim + 15) // 16 * 16


def xielu_rows(p: torch.Tensor, ff: int, act: Tuple[float, float], width: int) -> torch.Tensor:
    """xIELU of p[:, :ff] in p's type, zero-padded to `width` columns.  act: the factors of the positive and the negative side."""
    t = p.shape[0]
    if not p.is_cuda:
        return torch.nn.functional.pad(R.xielu(p[:, :ff], *act), (0, width - ff)).to(p.dtype)
    out = torch.empty(t, width, dtype=p.dtype, device=p.device)
    _lib.call("stk_xielu", p, p.stride(0), ff, float(act[0]), float(act[1]), out, out.stride(0), width, _is32(p), t, _lib.stream())
    return out


def join_glu(proj: torch.Tensor, out: torch.Tensor, mixer_dim: int, glu: Optional[Tuple[int, int, int]],
             act: str = "silu") -> None:
    """out[:, out_offset(mixer_dim):] = act(gate) * up with (gate, up) at columns glu[0], glu[1] of proj, glu[2] wide (None:
    no feed-forward); columns of `out` between and after the two parts become zero."""
    o0 = out_offset(mixer_dim)
    go, uo, ff = glu if glu is not None else (0, 0, 0)
    if not proj.is_cuda:
        out[:, mixer_dim:] = 0
        if ff:
            gate, up = proj[:, go:go + ff].to(F32), proj[:, uo:uo + ff].to(F32)
            gate = torch.relu(gate) if act == "relu" else torch.nn.functional.silu(gate)
            out[:, o0:o0 + ff] = (gate * up).to(out.dtype)
        return
    if out.shape[1] == mixer_dim:
        return
    _lib.call("stk_join_glu", proj, proj.stride(0), go, uo, ff, out, out.stride(0), _is32(proj), mixer_dim, o0, out.shape[1],
              1 if act == "relu" else 0, proj.shape[0], _lib.stream())
