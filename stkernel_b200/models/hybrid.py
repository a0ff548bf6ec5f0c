"""Decoder described layer by layer (`HybridConfig`): attention and recurrent mixers, in parallel, post-norm, streams or shifted blocks.

Parallel block: a layer is two matrix products.  Everything that reads the layer's norm (mixer projections, feed-forward gate and up) is one
weight `w_in`; everything that is added to the residual (mixer output and feed-forward down projection) is one weight `w_out`
over the joined activations, so the sum of both sublayers is formed inside that product, and the fp32 residual is touched
once per layer, by the kernel that also norms it for the next layer:

    h = norm(x += y_prev);  p = h W_in^T;  c = [mixer(p) | silu(p.gate) * p.up];  y = c W_out^T  (fp32)

Post-norm block: both sublayers read the residual itself (its copy h in the compute type) and one kernel per sublayer norms the
output, adds it to the fp32 residual and leaves the next copy; a mixture of experts' weighted sum is formed in that kernel too:

    h = x += norm1(mixer(h));  h = x += norm2(ff(h))

Streams block: several fp32 residual streams; one kernel per sublayer writes the previous sublayer's output into all of them (the
weighted sum over a token's experts on the way), forms the next sublayer's weighted sum of the new streams and norms it:

    x_t = sum_s mix[s, t] x_s + write[t] y;  h = norm(sum_s read[s] x_s);  y = sublayer(h)

Shifted block: one kernel per layer adds what the layer before left (both sides of its mixer, each normed, and its feed-forward) to the
fp32 residual, norms it, and forms the token-shifted input of the mixer and the blends that time mixing projects:

    h = norm(x += y_prev);  s = h + (h' - h) shift;  y = mixer(s) + ff(h)          (h': the previous token's h)

A parallel mixer (two mixers over the same input) is one product in and one product out, like the parallel block's sublayers.

Segments of both weights start on 16-column boundaries (zero-padded), whatever the configured sizes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..config import HybridConfig, HybridLayer, recurrent_part
from ..ops import attention as A
from ..ops import functional as Fn
from ..ops import grouped as GA
from ..ops import hybrid as HB
from ..ops import latent as LA
from ..ops import moe as MO
from ..ops import recurrence as RC
from ..ops import shifted as SH
from ..ops import talking as TK
from ..ops.functional import LinearWeight
from ..utils.spans import span
from .decoder import Decoder
from .sources import RANDOM_EXTENT, WeightSource

BF16 = torch.bfloat16
F32 = torch.float32
ALIGN = 16


def _pad(n: int) -> int:
    return (n + ALIGN - 1) // ALIGN * ALIGN


def weight_shapes(cfg: HybridConfig) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Checkpoint tensor name -> (shape, kind)."""
    W = cfg.hidden_size
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {"embed": ((cfg.vocab_size, W), "bf16")}
    for i, l in enumerate(cfg.layers):
        if l.weights_of is not None:
            continue
        m, p = l.mixer, f"l{i}"
        out[f"{p}.norm1"] = ((W,), "bf16")
        if cfg.block == "shifted":
            out[f"{p}.shift"] = ((W,), "bf16")
        if cfg.block == "streams":
            for q in (1, 2) if l.mlp is not None else (1,):
                out[f"{p}.norm{q}.b"] = ((W,), "bf16")
                out[f"{p}.hc{q}.in"] = ((cfg.streams,), "bf16")
                out[f"{p}.hc{q}.out"] = ((cfg.streams,), "bf16")
                out[f"{p}.hc{q}.mix"] = ((cfg.streams, cfg.streams), "bf16")
        if m.kind == "parallel":
            out.update(_parallel_shapes(f"{p}.mix", m, W))
        elif m.kind == "mamba2":
            out.update(_mamba2_shapes(f"{p}.mix", m, W))
        elif m.kind == "attention":
            out[f"{p}.mix.q"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.k"] = ((m.kv_heads * m.dim, W), "bf16")
            out[f"{p}.mix.sink"] = ((m.heads,), "bf16")
        elif m.kind == "latent_attention":
            out[f"{p}.mix.dq"] = ((m.q_rank, W), "bf16")
            out[f"{p}.mix.dq.norm"] = ((m.q_rank,), "bf16")
            out[f"{p}.mix.uq"] = ((m.heads * (m.dim + m.rot_dim), m.q_rank), "bf16")
            if m.kv_from is None:
                out[f"{p}.mix.dkv"] = ((m.kv_rank + m.rot_dim, W), "bf16")
                out[f"{p}.mix.dkv.norm"] = ((m.kv_rank,), "bf16")
            out[f"{p}.mix.uk"] = ((m.heads * m.dim, m.kv_rank), "bf16")
            out[f"{p}.mix.uv"] = ((m.heads * m.vdim, m.kv_rank), "bf16")
            out[f"{p}.mix.g"] = ((m.heads, W), "bf16")
        else:
            out[f"{p}.mix.q"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.k"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.v"] = ((m.heads * m.vdim, W), "bf16")
            out[f"{p}.mix.g"] = ((m.heads * m.vdim, W), "bf16")
            out[f"{p}.mix.norm"] = ((m.heads * m.vdim,), "bf16")
            for g in ("i", "f"):
                out[f"{p}.mix.{g}"] = ((m.heads, W), "bf16")
                out[f"{p}.mix.{g}.b"] = ((m.heads,), "bf16")
        if m.kind != "parallel":
            out[f"{p}.mix.o"] = ((W, m.out_dim), "bf16")
        if l.mlp is not None:
            if cfg.block not in ("parallel", "shifted"):
                out[f"{p}.norm2"] = ((W,), "bf16")
            if l.mlp.kind == "dense":
                if l.mlp.gated:
                    out[f"{p}.mlp.gate"] = ((l.mlp.ff, W), "bf16")
                else:
                    out[f"{p}.mlp.act"] = ((2,), "bf16")
                out[f"{p}.mlp.up"] = ((l.mlp.ff, W), "bf16")
                out[f"{p}.mlp.down"] = ((W, l.mlp.ff), "bf16")
            else:
                for e in range(l.mlp.experts):
                    if l.mlp.gated:
                        out[f"{p}.mlp.e{e}.gate"] = ((l.mlp.ff, W), "bf16")
                    out[f"{p}.mlp.e{e}.up"] = ((l.mlp.ff, W), "bf16")
                    out[f"{p}.mlp.e{e}.down"] = ((W, l.mlp.ff), "bf16")
                out[f"{p}.mlp.router"] = ((l.mlp.experts, W), "bf16")
                if l.mlp.router_bias:
                    out[f"{p}.mlp.router.b"] = ((l.mlp.experts,), "bf16")
                if l.mlp.scoring == "sigmoid":
                    out[f"{p}.mlp.correction"] = ((l.mlp.experts,), "bf16")
                if l.mlp.shared_ff:
                    out[f"{p}.mlp.shared.up"] = ((l.mlp.shared_ff, W), "bf16")
                    out[f"{p}.mlp.shared.down"] = ((W, l.mlp.shared_ff), "bf16")
    if cfg.bigram is not None:
        out["bigram"] = ((cfg.bigram.buckets + 1, W), "bf16")
    out["final.norm"] = ((W,), "bf16")
    if cfg.block == "streams":
        out["final.norm.b"] = ((W,), "bf16")
    if not cfg.tied_head:
        out["head"] = ((cfg.vocab_size, W), "bf16")
    return out


def _parallel_shapes(p: str, m, W: int) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    out = {}
    a, r = m.left, m.right
    for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
        out[f"{p}.left.{n}"] = ((rows, W), "bf16")
        if a.bias:
            out[f"{p}.left.{n}.b"] = ((rows,), "bf16")
    if a.gate:
        out[f"{p}.left.g"] = ((a.heads if a.kind == "talking_attention" else a.out_dim, W), "bf16")
    if a.kind == "talking_attention":
        if a.qk_norm:
            out[f"{p}.left.q.norm"] = out[f"{p}.left.k.norm"] = ((a.dim,), "bf16")
        out[f"{p}.left.talk"] = ((a.heads, a.heads), "bf16")
        if a.sink:
            out[f"{p}.left.sink"] = ((a.heads,), "bf16")
    if m.out_norm:
        out[f"{p}.left.out"] = out[f"{p}.right.out"] = ((W,), "bf16")
    if r.kind == "time_mix":
        N = r.out_dim
        for n in "rkvg":
            out[f"{p}.right.{n}"] = ((N, W), "bf16")
        for n in "rkvgw":
            out[f"{p}.right.mu.{n}"] = ((W,), "bf16")
        out[f"{p}.right.w1"] = ((r.rank, W), "bf16")
        out[f"{p}.right.w2"] = ((N, r.rank), "bf16")
        out[f"{p}.right.w0"] = out[f"{p}.right.norm"] = ((N,), "bf16")
        out[f"{p}.right.u"] = ((r.heads, r.dim), "bf16")
    else:
        for n, rows in (("q", r.heads * r.dim), ("k", r.heads * r.dim), ("v", r.out_dim), ("g", r.out_dim)):
            out[f"{p}.right.{n}"] = ((rows, W), "bf16")
    out[f"{p}.left.o"] = ((W, a.out_dim), "bf16")
    out[f"{p}.right.o"] = ((W, r.out_dim), "bf16")
    return out


def _mamba2_shapes(p: str, m, W: int) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    out = {f"{p}.in": ((m.out_dim + m.conv_dim + m.heads, W), "bf16"), f"{p}.conv": ((m.conv_dim, m.conv), "bf16"),
           f"{p}.conv.b": ((m.conv_dim,), "bf16"), f"{p}.norm": ((m.out_dim,), "bf16")}
    for n in ("dt_bias", "A_log", "D"):
        out[f"{p}.{n}"] = ((m.heads,), "bf16")
    return out


def init_random_weights(cfg: HybridConfig, seed: int = 0, std: Optional[float] = None) -> Dict[str, torch.Tensor]:
    """Random master weights: matrices ~N(0, std) (default: fan-in scaled), norms around 1, forget biases positive, residual streams
    that mostly stay themselves, step sizes around 0.1, blends between a token and its predecessor from 0 to 0.8, decays from fast to slow."""
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, torch.Tensor] = {}
    for name, (shape, _) in weight_shapes(cfg).items():
        shape = tuple(RANDOM_EXTENT if n is None else n for n in shape)
        r = torch.randn(shape, generator=g)
        if len(shape) == 1 and "norm" in name and not name.endswith(".b"):
            t = 1.0 + 0.2 * r
        elif ".hc" in name:
            t = 0.3 * r + (torch.eye(shape[0]) if len(shape) == 2 else 0.6)
        elif name.endswith(".dt_bias"):
            t = 0.7 * r - 2.0
        elif name.endswith(".f.b"):
            t = 3.0 + r
        elif name.endswith(".shift") or ".mu." in name:
            t = 0.4 + 0.4 * torch.tanh(r)
        elif name.endswith((".left.out", ".right.out")):
            t = 1.0 + 0.2 * r
        elif name.endswith(".w0"):
            t = -3.0 + 1.5 * r
        elif name.endswith(".talk"):
            t = torch.eye(shape[0]) + 0.3 * r
        elif name.endswith(".correction"):
            t = 0.3 * r - 1.0
        elif len(shape) == 1:
            t = 0.5 * r
        else:
            t = r * (std if std is not None else shape[-1] ** -0.5)
        w[name] = t
    return w


# ----------------------------------------------------------------------------
# weights in storage format
# ----------------------------------------------------------------------------
@dataclass
class BlockWeights:
    """Tensors of one layer (shared by every layer that names it in `weights_of`)."""
    norm: torch.Tensor                      # fp32 [W]
    w_in: LinearWeight                      # [segments, pad(W)]
    w_out: LinearWeight                     # [W, segments]
    seg: Dict[str, int]                     # first column of each segment of the w_in product
    attention: Optional[HB.AttentionParams] = None
    mlstm: Optional[HB.MlstmParams] = None
    latent: Optional[LA.LatentParams] = None
    grouped: Optional[GA.GroupedParams] = None
    retention: Optional[RC.RetentionParams] = None
    mamba2: Optional[RC.Mamba2Params] = None
    talking: Optional[TK.TalkingParams] = None
    time_mix: Optional[RC.TimeMixParams] = None
    # parallel mixers whose sides have products of their own
    w_mixes: Optional[LinearWeight] = None  # [4 * np, pad(W)]: r, k, v, gate of time mixing, each from its own blend
    w_decay: Tuple[LinearWeight, ...] = ()  # [pad(rank), pad(W)], [np, pad(rank) or twice that]
    w_sides: Tuple[LinearWeight, ...] = ()  # output projections, left and right
    out_norms: Tuple[torch.Tensor, ...] = ()            # fp32 [W] each
    # shifted blocks
    shift: Optional[torch.Tensor] = None    # fp32 [W]
    mu: Optional[torch.Tensor] = None       # fp32 [blends, W]
    w_gates: Optional[LinearWeight] = None  # [2 * heads, pad(W)]: input and forget gate of the recurrence (fp32 results)
    # streams blocks: norm biases and how the sublayers read and write the streams
    norm_b: Optional[torch.Tensor] = None
    norm2_b: Optional[torch.Tensor] = None
    streams: Tuple[HB.StreamWeights, ...] = ()          # mixer's, feed-forward's
    # post-norm and streams blocks: the feed-forward has weights of its own
    norm2: Optional[torch.Tensor] = None    # fp32 [W]
    w_gate_up: Optional[LinearWeight] = None            # gate and up, or up alone
    xielu: Tuple[float, float] = (0.0, 0.0)
    w_down: Optional[LinearWeight] = None
    router: Optional[LinearWeight] = None   # [experts, pad(W)]
    router_bias: Optional[torch.Tensor] = None          # fp32 [experts]
    experts: Optional[MO.PlainExperts] = None


@dataclass
class HybridWeights:
    embed: torch.Tensor                     # [V, W]
    head: LinearWeight                      # [V, pad(W)]
    norm: torch.Tensor                      # fp32 [W]
    layers: List[BlockWeights]              # one entry per layer; `weights_of` layers repeat an entry
    layer_offset: int = 0
    norm_b: Optional[torch.Tensor] = None   # fp32 [W]
    bigram: Optional[torch.Tensor] = None   # [buckets + 1, W]


def _stack(parts: List[Tuple[str, torch.Tensor]], width: int, dtype) -> Tuple[LinearWeight, Dict[str, int]]:
    """Row-stack [n_i, K] weights, every segment padded to whole alignment units and K to `width`."""
    seg: Dict[str, int] = {}
    n = 0
    for name, t in parts:
        seg[name] = n
        n += _pad(t.shape[0])
    w = torch.zeros(n, width, dtype=dtype, device=parts[0][1].device)
    for name, t in parts:
        w[seg[name]:seg[name] + t.shape[0], :t.shape[1]] = t.to(dtype)
    return LinearWeight(w), seg


def _spread(w: torch.Tensor, heads: int, rows: int, pad_rows: int, width: int, dtype) -> torch.Tensor:
    """[heads * rows, K] -> [heads * pad_rows, width]: zero rows after each head's, zero columns after K."""
    out = torch.zeros(heads, pad_rows, width, dtype=dtype, device=w.device)
    out[:, :rows, :w.shape[1]] = w.view(heads, rows, -1).to(dtype)
    return out.view(heads * pad_rows, width)


def build_latent(cfg: HybridConfig, get, m, dt, device) -> LA.LatentParams:
    H, D, R, C, Q = m.heads, m.dim, m.rot_dim, m.kv_rank, m.q_rank
    dp, cp, vp = LA.head_pads(m)
    f32 = lambda n: get(n).to(F32).contiguous()
    uq = get("mix.uq").view(H, D + R, Q)
    w_uq = torch.zeros(H * dp + _pad(H * R), _pad(Q), dtype=dt, device=device)
    w_uq[:H * dp] = _spread(uq[:, :D].reshape(H * D, Q), H, D, dp, _pad(Q), dt)
    if R:
        w_uq[H * dp:H * dp + H * R, :Q] = uq[:, D:].reshape(H * R, Q).to(dt)
    w_uk = _spread(get("mix.uk").view(H, D, C).transpose(1, 2).reshape(H * C, D), H, C, cp, dp, dt)
    w_uv = _spread(get("mix.uv"), H, m.vdim, vp, cp, dt)
    w_ukv = None
    if dt == BF16 and torch.device(device).type == "cuda" and LA.prompt_ok(m):
        # prompts expand keys and values from the latent columns of gathered rows
        v64, cols = (m.vdim + 63) // 64 * 64, LA.latent_row(C, R)[1]
        both = torch.zeros(H, dp + v64, cols, dtype=dt, device=device)
        both[:, :D, :C] = get("mix.uk").view(H, D, C).to(dt)
        both[:, dp:dp + m.vdim, :C] = get("mix.uv").view(H, m.vdim, C).to(dt)
        w_ukv = LinearWeight(both.view(H * (dp + v64), cols))
    freq = m.rotary.frequencies()[0] if m.rotary is not None else []
    return LA.LatentParams(H, D, R, m.vdim, Q, C, m.scale, cfg.norm_eps, dp, cp, vp, LA.split_frequencies(freq, device),
                           f32("mix.dq.norm"), f32("mix.dkv.norm") if m.kv_from is None else None, LinearWeight(w_uq),
                           LinearWeight(w_uk), LinearWeight(w_uv), w_ukv)


def _parallel_params(cfg: HybridConfig, m, f32, device) -> Tuple[GA.GroupedParams, RC.RetentionParams]:
    a, r = m.left, m.right
    bias = torch.cat([f32(f"mix.left.{n}.b") for n in ("q", "k", "v")]).contiguous() if a.bias else None
    temp = (a.q_temp.coef, a.q_temp.every) if a.q_temp is not None else (0.0, 1.0)
    sink = torch.zeros(a.heads, dtype=F32, device=device) if a.null_sink else None
    left = GA.GroupedParams(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, bias, cfg.norm_eps if a.qk_norm else None, temp, sink, a.gate,
                            m.left_scale)
    freq = r.rotary.frequencies()[0] if r.rotary is not None else []
    log_decay = torch.tensor(r.decay, dtype=torch.float64).log().to(F32).to(device)
    return left, RC.RetentionParams(r.heads, r.dim, r.vdim, log_decay, LA.split_frequencies(r.decay, device), LA.split_frequencies(freq, device), cfg.norm_eps, m.right_scale)


def _padded(w: torch.Tensor, rows: int, width: int, dtype) -> torch.Tensor:
    out = torch.zeros(rows, width, dtype=dtype, device=w.device)
    out[:w.shape[0], :w.shape[1]] = w.to(dtype)
    return out


def build_talking_time_mix(cfg: HybridConfig, b: BlockWeights, m, get, f32, dt, device) -> None:
    """Talking-heads attention beside time mixing."""
    a, r, W = m.left, m.right, cfg.hidden_size
    bias = torch.cat([f32(f"mix.left.{n}.b") for n in ("q", "k", "v")]).contiguous() if a.bias else None
    freq = a.rotary.frequencies()[0] if a.rotary is not None else []
    norms = [f32(f"mix.left.{n}.norm") for n in "qk"] if a.qk_norm else [None, None]
    b.talking = TK.TalkingParams(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk or 0, cfg.norm_eps, bias, *norms,
                                 LA.split_frequencies(freq, device), f32("mix.left.talk"), f32("mix.left.sink") if a.sink else None, a.gate)
    N, np = r.out_dim, (r.out_dim + 127) // 128 * 128       # whole tiles of a block-diagonal product
    b.w_mixes = LinearWeight(torch.cat([_padded(get(f"mix.right.{n}"), np, _pad(W), dt) for n in "rkvg"]))
    w1, w2 = get("mix.right.w1"), get("mix.right.w2")
    if w1.shape[0] != w2.shape[1]:
        raise ValueError(f"mix.right.w1 has {w1.shape[0]} rows, mix.right.w2 {w2.shape[1]} columns")
    rp = _pad(w1.shape[0])
    w2 = _padded(w2, np, rp, dt)
    # bf16: tanh comes as high part and remainder, both meet the same weights
    b.w_decay = (LinearWeight(_padded(w1, rp, _pad(W), dt)), LinearWeight(torch.cat([w2, w2], 1) if dt == BF16 and RC.tanh_pair(device) else w2))
    b.time_mix = RC.TimeMixParams(r.heads, r.dim, np, f32("mix.right.w0"), f32("mix.right.u").view(-1), f32("mix.right.norm"), cfg.norm_eps)
    b.w_sides = tuple(LinearWeight(_padded(get(f"mix.{s}.o"), W, _pad(p.out_dim), dt)) for s, p in (("left", a), ("right", r)))
    b.out_norms = (f32("mix.left.out"), f32("mix.right.out"))
    b.mu = torch.stack([f32(f"mix.right.mu.{n}") for n in "rkvgw"]).contiguous()


def _mamba2_params(cfg: HybridConfig, m, get, f32) -> RC.Mamba2Params:
    return RC.Mamba2Params(m.heads, m.vdim, m.state, m.groups, m.norm_groups, get("mix.conv").to(F32).t().contiguous(), f32("mix.conv.b"),
                           f32("mix.dt_bias"), (-torch.exp(get("mix.A_log").double())).to(F32).contiguous(), f32("mix.D"),
                           f32("mix.norm"), cfg.norm_eps)


def _stream_weights(f32, q: int) -> HB.StreamWeights:
    return HB.StreamWeights(f32(f"hc{q}.in"), f32(f"hc{q}.out"), f32(f"hc{q}.mix"))


def build_block(cfg: HybridConfig, src: WeightSource, i: int, device) -> BlockWeights:
    l: HybridLayer = cfg.layers[i]
    shapes = weight_shapes(cfg)
    get = lambda n: src.get(f"l{i}.{n}", shapes[f"l{i}.{n}"][0], device)
    f32 = lambda n: get(n).to(F32).contiguous()
    dt = F32 if cfg.dtype == "float32" else BF16
    m, W = l.mixer, cfg.hidden_size
    joined = l.mlp if cfg.block == "parallel" else None              # the feed-forward shares the mixer's two products
    if m.kind == "latent_attention":
        names = ["dq", "dkv", "g"] if m.kv_from is None else ["dq", "g"]
    elif m.kind == "parallel" and m.left.kind == "talking_attention":
        names = ["left.q", "left.k", "left.v"] + (["left.g"] if m.left.gate else [])
    elif m.kind == "parallel":
        names = ["left.q", "left.k", "left.v"] + (["left.g"] if m.left.gate else []) + [f"right.{n}" for n in "qkvg"]
    else:
        names = ["q", "k"] + (["v", "g"] if m.kind == "mlstm" else [])
    if m.kind == "mamba2":
        parts = list(zip(("z", "xbc", "dt"), get("mix.in").split([m.out_dim, m.conv_dim, m.heads])))
    else:
        parts = [(n, get(f"mix.{n}")) for n in names]
    if joined is not None:
        parts += [("gate", get("mlp.gate")), ("up", get("mlp.up"))]
    w_in, seg = _stack(parts, _pad(W), dt)
    if m.kind == "latent_attention":
        vp = LA.head_pads(m)[2]
        w_out = torch.zeros(W, m.heads, vp, dtype=dt, device=device)
        w_out[:, :, :m.vdim] = get("mix.o").view(W, m.heads, m.vdim).to(dt)
        w_out = w_out.view(W, m.heads * vp)
    elif m.kind == "parallel" and m.left.kind == "talking_attention":
        w_out = None                                       # each side has its own
    elif m.kind == "parallel":
        off = HB.out_offset(m.left.out_dim)
        w_out = torch.zeros(W, off + _pad(m.right.out_dim), dtype=dt, device=device)
        w_out[:, :m.left.out_dim] = get("mix.left.o").to(dt)
        w_out[:, off:off + m.right.out_dim] = get("mix.right.o").to(dt)
    else:
        off = HB.out_offset(m.out_dim)
        w_out = torch.zeros(W, off + (_pad(joined.ff) if joined is not None else 0), dtype=dt, device=device)
        w_out[:, :m.out_dim] = get("mix.o").to(dt)
        if joined is not None:
            w_out[:, off:off + joined.ff] = get("mlp.down").to(dt)
    b = BlockWeights(f32("norm1"), w_in, LinearWeight(w_out) if w_out is not None else None, seg)
    if m.kind == "attention":
        freq, mag = m.rotary.frequencies() if m.rotary is not None else ([], 1.0)
        b.attention = HB.AttentionParams(m.heads, m.kv_heads, m.dim, m.window, m.scale, m.softcap,
                                         torch.tensor(freq, dtype=torch.float64).to(F32).to(device), mag,
                                         f32("mix.sink") if m.sink else None)
    elif m.kind == "latent_attention":
        b.latent = build_latent(cfg, get, m, dt, device)
    elif m.kind == "parallel" and m.left.kind == "talking_attention":
        build_talking_time_mix(cfg, b, m, get, f32, dt, device)
    elif m.kind == "parallel":
        b.grouped, b.retention = _parallel_params(cfg, m, f32, device)
    elif m.kind == "mamba2":
        b.mamba2 = _mamba2_params(cfg, m, get, f32)
    else:
        b.w_gates, _ = _stack([("i", torch.cat([get("mix.i"), get("mix.f")], 0))], _pad(W), dt)
        b.w_gates = LinearWeight(b.w_gates.w[:2 * m.heads])
        b.mlstm = HB.MlstmParams(m.heads, m.dim, m.vdim, m.gate_cap, torch.cat([f32("mix.i.b"), f32("mix.f.b")]).contiguous(),
                                 f32("mix.norm"), cfg.norm_eps)
    if cfg.block == "streams":
        b.norm_b = f32("norm1.b")
        b.streams = (_stream_weights(f32, 1),)
        if l.mlp is not None:
            b.norm2_b = f32("norm2.b")
            b.streams += (_stream_weights(f32, 2),)
    if cfg.block == "shifted":
        b.shift = f32("shift")
    if l.mlp is not None and joined is None:
        if cfg.block != "shifted":
            b.norm2 = f32("norm2")
        build_feed_forward(b, l.mlp, get, W, dt, device)
    return b


def build_feed_forward(b: BlockWeights, mlp, get, W: int, dt, device) -> None:
    ff = _pad(mlp.ff)
    if mlp.kind == "dense":
        b.w_gate_up, seg = _stack(([("gate", get("mlp.gate"))] if mlp.gated else []) + [("up", get("mlp.up"))], _pad(W), dt)
        if mlp.act == "xielu":
            sp = torch.nn.functional.softplus(get("mlp.act").double().cpu()).tolist()
            b.xielu = (sp[0], sp[1] + 0.5)
        b.seg.update(seg)
        down = torch.zeros(W, ff, dtype=dt, device=device)
        down[:, :mlp.ff] = get("mlp.down").to(dt)
        b.w_down = LinearWeight(down)
        return
    # the shared expert's columns in equal parts, each an expert that every token takes
    ff, n = _pad(mlp.expert_width), mlp.experts + mlp.shared_parts
    up = torch.zeros(n, (2 if mlp.gated else 1) * ff, _pad(W), dtype=dt, device=device)
    down = torch.zeros(n, _pad(W), ff, dtype=dt, device=device)
    for e in range(mlp.experts):
        if mlp.gated:
            up[e, 0:2 * mlp.ff:2, :W] = get(f"mlp.e{e}.gate").to(dt)
            up[e, 1:2 * mlp.ff:2, :W] = get(f"mlp.e{e}.up").to(dt)
        else:
            up[e, :mlp.ff, :W] = get(f"mlp.e{e}.up").to(dt)
        down[e, :W, :mlp.ff] = get(f"mlp.e{e}.down").to(dt)
    if mlp.shared_parts:
        wide = mlp.expert_width
        rows, cols = get("mlp.shared.up").split(wide), get("mlp.shared.down").split(wide, 1)
        for j, (r, c) in enumerate(zip(rows, cols)):
            up[mlp.experts + j, :r.shape[0], :W] = r.to(dt)
            down[mlp.experts + j, :W, :c.shape[1]] = c.to(dt)
    b.experts = MO.PlainExperts(up, down, mlp.act)
    router, _ = _stack([("router", get("mlp.router"))], _pad(W), dt)
    b.router = LinearWeight(router.w[:mlp.experts])
    bias = "mlp.correction" if mlp.scoring == "sigmoid" else "mlp.router.b" if mlp.router_bias else None
    b.router_bias = get(bias).to(F32).contiguous() if bias is not None else None


def build_hybrid_weights(cfg: HybridConfig, src: WeightSource, device) -> HybridWeights:
    dt = F32 if cfg.dtype == "float32" else BF16
    V, W = cfg.vocab_size, cfg.hidden_size
    blocks: Dict[int, BlockWeights] = {}
    for i in range(len(cfg.layers)):
        j = cfg.weight_layer(i)
        if j not in blocks:
            blocks[j] = build_block(cfg, src, j, device)
    embed = src.get("embed", (V, W), device).to(dt).contiguous()
    if cfg.tied_head and _pad(W) == W:
        head = LinearWeight(embed)
    else:
        table = embed if cfg.tied_head else src.get("head", (V, W), device)
        head = LinearWeight(_stack([("head", table)], _pad(W), dt)[0].w[:V])
    # a factor on the logits is one on the norm in front of the head
    norm = lambda n: (src.get(n, (W,), device).to(F32) * cfg.logit_scale).contiguous()
    return HybridWeights(embed, head, norm("final.norm"), [blocks[cfg.weight_layer(i)] for i in range(len(cfg.layers))],
                         norm_b=norm("final.norm.b") if cfg.block == "streams" else None,
                         bigram=src.get("bigram", (cfg.bigram.buckets + 1, W), device).to(dt).contiguous() if cfg.bigram is not None else None)


# ----------------------------------------------------------------------------
# model
# ----------------------------------------------------------------------------
class HybridModel(Decoder):
    def __init__(self, cfg: HybridConfig, weights: HybridWeights, kv):
        super().__init__(weights.embed.device)
        self.cfg = cfg
        self.w = weights
        self.kv = kv
        self.act = HB.act_dtype(cfg.dtype, self.device)
        self.width = _pad(cfg.hidden_size)
        self.recurrent = cfg.block == "shifted" or any(recurrent_part(l.mixer) is not None for l in cfg.layers)
        self.on_layer = None                # optional hook (layer index, residual [T, W] fp32; streams: their sum) after each layer
        self.read_sum = torch.ones(cfg.streams, dtype=F32, device=self.device)

    def build_meta(self, buf, t_pad: int, n_req: int, max_comp_rows: int, pure_decode: bool = False,
                   spans: Tuple = (1, 1)) -> HB.HybridMeta:
        tok_req, positions, first, last = A.token_maps(buf.d_qstart, buf.d_rows, buf.d_start, n_req, t_pad)
        return HB.HybridMeta(buf.d_tokens[:t_pad], tok_req, positions, first, last, buf.d_qstart, buf.d_rows, buf.d_start, n_req,
                             spans[1], pure_decode, spans[0], spans[2] if len(spans) > 2 else None, max_context=4 * max_comp_rows + 4)

    def decode_bucket(self, max_comp_rows: int) -> int:
        # full-context attention splits the key range by the longest context a graph serves: one graph per power of two
        if self.kv.full is None:
            return 0
        bucket = 256
        while bucket < max_comp_rows + 1:
            bucket *= 2
        return bucket

    def layer(self, li: int, x: torch.Tensor, y: Optional[torch.Tensor], meta: HB.HybridMeta) -> torch.Tensor:
        """Parallel block: adds the previous layer's output y to the residual x (in place) and returns this layer's output
        [T, W] fp32."""
        cfg, b = self.cfg, self.w.layers[li]
        m, mlp = cfg.layers[li].mixer, cfg.layers[li].mlp
        h = HB.add_layer_norm(x, y, b.norm, cfg.norm_eps, self.width, self.act)
        glu = (b.seg["gate"], b.seg["up"], mlp.ff) if mlp is not None else None
        c = self.mix(li, h, meta, glu, mlp.act if mlp is not None else "silu")
        return Fn.linear(c, b.w_out, out_dtype=F32, tag="out")

    def mix(self, li: int, h: torch.Tensor, meta: HB.HybridMeta, glu: Optional[Tuple[int, int, int]] = None,
            act: str = "silu") -> torch.Tensor:
        """Mixer output of layer li (before its output projection), joined with the feed-forward activation where the block
        shares its products (glu)."""
        b, m = self.w.layers[li], self.cfg.layers[li].mixer
        t = h.shape[0]
        if m.kind == "latent_attention":
            p = Fn.linear(h, b.w_in, out_dtype=F32, tag="in")
            src = self.cfg.cache_layer(li)
            table, cache = self.kv.group_of(src).table_dev, self.kv.kv_cache[src]
            cq = LA.latent_prep(p, b.seg["dq"], b.seg.get("dkv", -1), b.latent, meta, table, cache, self.act)
            q = Fn.linear(cq, b.latent.w_uq, tag="uq")
            with span("latent_attention", t):
                return LA.latent_attention(q, p[:, b.seg["g"]:b.seg["g"] + m.heads], b.latent, meta, table, cache)
        p = Fn.linear(h, b.w_in, tag="in")
        c = torch.empty(t, b.w_out.in_features, dtype=self.act, device=h.device)
        if m.kind == "parallel":
            with span("parallel_mixer", t):
                s, table, cache = b.seg, self.kv.group_of(li).table_dev, self.kv.kv_cache[li]
                q = GA.grouped_prep(p, s["left.q"], s["left.k"], s["left.v"], b.grouped, meta, table, cache)
                GA.grouped_attention(p, q, s.get("left.g", 0), b.grouped, meta, table, cache, c)
                RC.retention(p, s["right.q"], s["right.k"], s["right.v"], s["right.g"], b.retention, meta, self.kv.state[li], c,
                             m.left.out_dim)
        elif m.kind == "mamba2":
            with span("mamba2", t):
                RC.mamba2(p, b.seg["z"], b.seg["xbc"], b.seg["dt"], b.mamba2, meta, self.kv.state[li], c)
        elif m.kind == "attention":
            with span("window_attention", t):
                HB.window_attention(p, b.seg["q"], b.seg["k"], b.attention, meta, self.kv.group_of(li).table_dev,
                                    self.kv.kv_cache[li], c)
                HB.join_glu(p, c, m.out_dim, glu, act)
        else:
            with span("mlstm", t):
                gates = Fn.linear(h, b.w_gates, out_dtype=F32, tag="gates")
                HB.mlstm(p, b.seg["q"], b.seg["k"], b.seg["v"], b.seg["g"], gates, b.mlstm, meta, self.kv.state[li], c, glu)
        return c

    def feed_forward(self, li: int, h: torch.Tensor):
        """Feed-forward output of a post-norm or streams layer: fp32 rows, or expert rows whose sum the next kernel forms."""
        b, mlp = self.w.layers[li], self.cfg.layers[li].mlp
        if mlp.kind == "dense":
            p = Fn.linear(h, b.w_gate_up, tag="gate_up")
            if not mlp.gated:
                return Fn.linear(HB.xielu_rows(p, mlp.ff, b.xielu, b.w_down.in_features), b.w_down, out_dtype=F32, tag="down")
            c = torch.empty(h.shape[0], b.w_down.in_features, dtype=self.act, device=h.device)
            HB.join_glu(p, c, 0, (b.seg["gate"], b.seg["up"], mlp.ff), mlp.act)
            return Fn.linear(c, b.w_down, out_dtype=F32, tag="down")
        with span("experts", h.shape[0]):
            how = (b.router_bias, mlp.top, mlp.scoring, True, mlp.scale)
            kw = dict(always=mlp.shared_parts, groups=mlp.groups, keep=mlp.keep)
            routed = Fn.gate_route(h, b.router, *how, **kw) if h.is_cuda else None
            if routed is None:
                routed = MO.router(Fn.linear(h, b.router, out_dtype=F32, tag="router"), *how, **kw)
            return MO.plain_experts(h, *routed, b.experts)

    def post_norm_layer(self, li: int, x: torch.Tensor, h: torch.Tensor, meta: HB.HybridMeta) -> torch.Tensor:
        """Adds both sublayers to the residual x (in place); h is x in the compute type, as is the result."""
        cfg, b = self.cfg, self.w.layers[li]
        y = Fn.linear(self.mix(li, h, meta), b.w_out, out_dtype=F32, tag="out")
        h = HB.post_norm_add(x, y, b.norm, cfg.norm_eps, self.width, self.act)
        if cfg.layers[li].mlp is not None:
            h = HB.post_norm_add(x, self.feed_forward(li, h), b.norm2, cfg.norm_eps, self.width, self.act)
        return h

    def sides(self, li: int, s: torch.Tensor, blends: Optional[torch.Tensor], meta: HB.HybridMeta) -> SH.Pending:
        """Outputs of layer li's mixer on the shifted rows s (and their blends, for time mixing), as the next norm adds them."""
        b, m = self.w.layers[li], self.cfg.layers[li].mixer
        if m.kind != "parallel":
            return SH.Pending([(Fn.linear(self.mix(li, s, meta), b.w_out, out_dtype=F32, tag="out"), None, 1.0)])
        t, width, sg = s.shape[0], self.width, b.seg
        p = Fn.linear(s, b.w_in, tag="in")
        table, cache = self.kv.group_of(li).table_dev, self.kv.kv_cache[li]
        with span("talking_attention", t):
            q, gate = TK.talking_prep(p, sg["left.q"], sg["left.k"], sg["left.v"], sg.get("left.g", 0), b.talking, meta, table, cache)
            c = torch.empty(t, b.w_sides[0].in_features, dtype=self.act, device=s.device)
            TK.talking_attention(q, gate, b.talking, meta, table, cache, c)
        left = Fn.linear(c, b.w_sides[0], out_dtype=F32, tag="out")
        with span("time_mix", t):
            p = Fn.linear_blocks(blends[:, :4 * width], b.w_mixes, 4, tag="mixes")
            z = RC.tanh_rows(Fn.linear(blends[:, 4 * width:], b.w_decay[0], out_dtype=F32, tag="decay1"), self.act)
            z = Fn.linear(z, b.w_decay[1], out_dtype=F32, tag="decay2")
            c = torch.empty(t, b.w_sides[1].in_features, dtype=self.act, device=s.device)
            RC.time_mix(p, z, b.time_mix, meta, self.kv.state[li], c)
        right = Fn.linear(c, b.w_sides[1], out_dtype=F32, tag="out")
        return SH.Pending([(left, b.out_norms[0], m.left_scale), (right, b.out_norms[1], m.right_scale)])

    def shifted_hidden(self, meta: HB.HybridMeta):
        """-> (residual before the last layer's outputs, those outputs)."""
        cfg, st = self.cfg, self.kv.shift
        x = SH.embed_bigram(meta, self.w.embed, cfg.embedding_scale, self.w.bigram, cfg.bigram, st)
        pending = None
        for li, b in enumerate(self.w.layers):
            x, h, s, blends = SH.shifted_norm(x, pending, b.norm, cfg.norm_eps, self.width, self.act, b.shift, b.mu, st, li, meta)
            if self.on_layer is not None and li:
                self.on_layer(li - 1, x.clone())
            pending = self.sides(li, s, blends, meta)
            if cfg.layers[li].mlp is not None:
                pending.ff = self.feed_forward(li, h)
        if self.on_layer is not None:
            self.on_layer(len(self.w.layers) - 1, SH.shifted_norm(x, pending, self.w.norm, cfg.norm_eps, self.width, self.act)[0])
        SH.commit(st, meta)
        return x, pending

    def streams_hidden(self, meta: HB.HybridMeta):
        """-> (streams before the last sublayer's output, (that output, how it enters them))."""
        cfg = self.cfg
        x = HB.embed_scaled(meta.token_ids, self.w.embed, cfg.embedding_scale, streams=cfg.streams)
        y, after = None, None
        for li, b in enumerate(self.w.layers):
            h = HB.stream_norm(x, y, after, b.streams[0].read, b.norm, b.norm_b, cfg.norm_eps, self.width, self.act)
            y, after = Fn.linear(self.mix(li, h, meta), b.w_out, out_dtype=F32, tag="out"), b.streams[0]
            if cfg.layers[li].mlp is not None:
                h = HB.stream_norm(x, y, after, b.streams[1].read, b.norm2, b.norm2_b, cfg.norm_eps, self.width, self.act)
                y, after = self.feed_forward(li, h), b.streams[1]
            if self.on_layer is not None:
                rows = HB.expert_sum(y, cfg.hidden_size)[:, :cfg.hidden_size]
                self.on_layer(li, (torch.einsum("sr,tsw->tw", after.mix, x) + after.write.sum() * rows))
        return x, (y, after)

    def forward_hidden(self, meta: HB.HybridMeta):
        """-> (residual before the last layer's output, that output), both [T, W] fp32: the sum is formed where it is normed.
        Post-norm blocks: (residual, None); streams and shifted blocks: see `streams_hidden`, `shifted_hidden`."""
        cfg = self.cfg
        if cfg.block == "streams":
            return self.streams_hidden(meta)
        if cfg.block == "shifted":
            return self.shifted_hidden(meta)
        if cfg.block == "post_norm":
            h = torch.empty(meta.token_ids.shape[0], self.width, dtype=self.act, device=self.device)
            x = HB.embed_scaled(meta.token_ids, self.w.embed, cfg.embedding_scale, h)
            for li in range(len(self.w.layers)):
                h = self.post_norm_layer(li, x, h, meta)
                if self.on_layer is not None:
                    self.on_layer(li, x.clone())
            return x, None
        x = HB.embed_scaled(meta.token_ids, self.w.embed, cfg.embedding_scale)
        y = None
        for li in range(len(self.w.layers)):
            y = self.layer(li, x, y, meta)
            if self.on_layer is not None:
                self.on_layer(li, x + y)
        return x, y

    def head_hidden(self, X, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        x, y = X
        if self.cfg.block == "streams":
            return HB.stream_norm(x, *y, self.read_sum, self.w.norm, self.w.norm_b, self.cfg.norm_eps, self.width, self.act, rows=rows)
        if self.cfg.block == "shifted":
            if rows is None:
                rows = torch.arange(x.shape[0], device=x.device)
            return SH.shifted_norm(x, y, self.w.norm, self.cfg.norm_eps, self.width, self.act, rows=rows)[1]
        return HB.add_layer_norm(x, y, self.w.norm, self.cfg.norm_eps, self.width, self.act, rows=rows,
                                 center=self.cfg.block == "parallel")

    def compute_logits(self, h: torch.Tensor) -> torch.Tensor:
        return Fn.linear(h, self.w.head, out_dtype=F32, tag="head")
