"""Decoder described layer by layer (`HybridConfig`): attention and recurrent mixers in parallel blocks.

A layer is two matrix products.  Everything that reads the layer's norm (mixer projections, feed-forward gate and up) is one
weight `w_in`; everything that is added to the residual (mixer output and feed-forward down projection) is one weight `w_out`
over the joined activations, so the sum of both sublayers is formed inside that product, and the fp32 residual is touched
once per layer, by the kernel that also norms it for the next layer:

    h = norm(x += y_prev);  p = h W_in^T;  c = [mixer(p) | silu(p.gate) * p.up];  y = c W_out^T  (fp32)

Segments of both weights start on 16-column boundaries (zero-padded), whatever the configured sizes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..config import HybridConfig, HybridLayer
from ..ops import attention as A
from ..ops import functional as Fn
from ..ops import hybrid as HB
from ..ops.functional import LinearWeight
from ..utils.spans import span
from .decoder import Decoder
from .sources import WeightSource

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
        if m.kind == "attention":
            out[f"{p}.mix.q"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.k"] = ((m.kv_heads * m.dim, W), "bf16")
            out[f"{p}.mix.sink"] = ((m.heads,), "bf16")
        else:
            out[f"{p}.mix.q"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.k"] = ((m.heads * m.dim, W), "bf16")
            out[f"{p}.mix.v"] = ((m.heads * m.vdim, W), "bf16")
            out[f"{p}.mix.g"] = ((m.heads * m.vdim, W), "bf16")
            out[f"{p}.mix.norm"] = ((m.heads * m.vdim,), "bf16")
            for g in ("i", "f"):
                out[f"{p}.mix.{g}"] = ((m.heads, W), "bf16")
                out[f"{p}.mix.{g}.b"] = ((m.heads,), "bf16")
        out[f"{p}.mix.o"] = ((W, m.out_dim), "bf16")
        if l.mlp is not None:
            out[f"{p}.mlp.gate"] = ((l.mlp.ff, W), "bf16")
            out[f"{p}.mlp.up"] = ((l.mlp.ff, W), "bf16")
            out[f"{p}.mlp.down"] = ((W, l.mlp.ff), "bf16")
    out["final.norm"] = ((W,), "bf16")
    out["head"] = ((cfg.vocab_size, W), "bf16")
    return out


def init_random_weights(cfg: HybridConfig, seed: int = 0, std: Optional[float] = None) -> Dict[str, torch.Tensor]:
    """Random master weights: matrices ~N(0, std) (default: fan-in scaled), norms around 1, forget biases positive."""
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, torch.Tensor] = {}
    for name, (shape, _) in weight_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if len(shape) == 1 and "norm" in name:
            t = 1.0 + 0.2 * r
        elif name.endswith(".f.b"):
            t = 3.0 + r
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
    w_gates: Optional[LinearWeight] = None  # [2 * heads, pad(W)]: input and forget gate of the recurrence (fp32 results)


@dataclass
class HybridWeights:
    embed: torch.Tensor                     # [V, W]
    head: LinearWeight                      # [V, pad(W)]
    norm: torch.Tensor                      # fp32 [W]
    layers: List[BlockWeights]              # one entry per layer; `weights_of` layers repeat an entry
    layer_offset: int = 0


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


def build_block(cfg: HybridConfig, src: WeightSource, i: int, device) -> BlockWeights:
    l: HybridLayer = cfg.layers[i]
    shapes = weight_shapes(cfg)
    get = lambda n: src.get(f"l{i}.{n}", shapes[f"l{i}.{n}"][0], device)
    f32 = lambda n: get(n).to(F32).contiguous()
    dt = F32 if cfg.dtype == "float32" else BF16
    m, W = l.mixer, cfg.hidden_size
    names = ["q", "k"] + (["v", "g"] if m.kind == "mlstm" else [])
    parts = [(n, get(f"mix.{n}")) for n in names]
    if l.mlp is not None:
        parts += [("gate", get("mlp.gate")), ("up", get("mlp.up"))]
    w_in, seg = _stack(parts, _pad(W), dt)
    off = HB.out_offset(m.out_dim)
    w_out = torch.zeros(W, off + (_pad(l.mlp.ff) if l.mlp is not None else 0), dtype=dt, device=device)
    w_out[:, :m.out_dim] = get("mix.o").to(dt)
    if l.mlp is not None:
        w_out[:, off:off + l.mlp.ff] = get("mlp.down").to(dt)
    b = BlockWeights(f32("norm1"), w_in, LinearWeight(w_out), seg)
    if m.kind == "attention":
        freq, mag = m.rotary.frequencies() if m.rotary is not None else ([], 1.0)
        b.attention = HB.AttentionParams(m.heads, m.kv_heads, m.dim, m.window, m.scale, m.softcap,
                                         torch.tensor(freq, dtype=torch.float64).to(F32).to(device), mag,
                                         f32("mix.sink") if m.sink else None)
    else:
        b.w_gates, _ = _stack([("i", torch.cat([get("mix.i"), get("mix.f")], 0))], _pad(W), dt)
        b.w_gates = LinearWeight(b.w_gates.w[:2 * m.heads])
        b.mlstm = HB.MlstmParams(m.heads, m.dim, m.vdim, m.gate_cap, torch.cat([f32("mix.i.b"), f32("mix.f.b")]).contiguous(),
                                 f32("mix.norm"), cfg.norm_eps)
    return b


def build_hybrid_weights(cfg: HybridConfig, src: WeightSource, device) -> HybridWeights:
    dt = F32 if cfg.dtype == "float32" else BF16
    V, W = cfg.vocab_size, cfg.hidden_size
    blocks: Dict[int, BlockWeights] = {}
    for i in range(len(cfg.layers)):
        j = cfg.weight_layer(i)
        if j not in blocks:
            blocks[j] = build_block(cfg, src, j, device)
    head, _ = _stack([("head", src.get("head", (V, W), device))], _pad(W), dt)
    return HybridWeights(src.get("embed", (V, W), device).to(dt).contiguous(), LinearWeight(head.w[:V]),
                         src.get("final.norm", (W,), device).to(F32).contiguous(),
                         [blocks[cfg.weight_layer(i)] for i in range(len(cfg.layers))])


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
        self.recurrent = any(l.mixer.kind == "mlstm" for l in cfg.layers)
        self.on_layer = None                # optional hook (layer index, residual [T, W] fp32) after each layer

    def build_meta(self, buf, t_pad: int, n_req: int, max_comp_rows: int, pure_decode: bool = False,
                   spans: Tuple[int, int] = (1, 1)) -> HB.HybridMeta:
        tok_req, positions, first, last = A.token_maps(buf.d_qstart, buf.d_rows, buf.d_start, n_req, t_pad)
        return HB.HybridMeta(buf.d_tokens[:t_pad], tok_req, positions, first, last, buf.d_qstart, buf.d_rows, buf.d_start, n_req,
                             spans[1], pure_decode, spans[0])

    def layer(self, li: int, x: torch.Tensor, y: Optional[torch.Tensor], meta: HB.HybridMeta) -> torch.Tensor:
        """Adds the previous layer's output y to the residual x (in place) and returns this layer's output [T, W] fp32."""
        cfg, b = self.cfg, self.w.layers[li]
        m, mlp = cfg.layers[li].mixer, cfg.layers[li].mlp
        t = x.shape[0]
        h = HB.add_layer_norm(x, y, b.norm, cfg.norm_eps, self.width, self.act)
        p = Fn.linear(h, b.w_in, tag="in")
        c = torch.empty(t, b.w_out.in_features, dtype=self.act, device=x.device)
        glu = (b.seg["gate"], b.seg["up"], mlp.ff) if mlp is not None else None
        if m.kind == "attention":
            with span("window_attention", t):
                HB.window_attention(p, b.seg["q"], b.seg["k"], b.attention, meta, self.kv.group_of(li).table_dev,
                                    self.kv.kv_cache[li], c)
                HB.join_glu(p, c, m.out_dim, glu)
        else:
            with span("mlstm", t):
                gates = Fn.linear(h, b.w_gates, out_dtype=F32, tag="gates")
                HB.mlstm(p, b.seg["q"], b.seg["k"], b.seg["v"], b.seg["g"], gates, b.mlstm, meta, self.kv.state[li], c, glu)
        return Fn.linear(c, b.w_out, out_dtype=F32, tag="out")

    def forward_hidden(self, meta: HB.HybridMeta):
        """-> (residual before the last layer's output, that output), both [T, W] fp32: the sum is formed where it is normed."""
        x = HB.embed_scaled(meta.token_ids, self.w.embed, self.cfg.embedding_scale)
        y = None
        for li in range(len(self.w.layers)):
            y = self.layer(li, x, y, meta)
            if self.on_layer is not None:
                self.on_layer(li, x + y)
        return x, y

    def head_hidden(self, X, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        x, y = X
        return HB.add_layer_norm(x, y, self.w.norm, self.cfg.norm_eps, self.width, self.act, rows=rows)

    def compute_logits(self, h: torch.Tensor) -> torch.Tensor:
        return Fn.linear(h, self.w.head, out_dtype=F32, tag="head")
