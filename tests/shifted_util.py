"""Configurations and weights shared by the tests of the shifted decoder (Fogizen)."""
import dataclasses

import torch

import fogizen_oracle as O
from hybrid_util import error, feed, make_engine, tokens  # noqa: F401  (one import for the tests)
from streams_util import LIMITS, close  # noqa: F401
from stkernel_b200.config import (BigramTable, DenseMlp, HybridConfig, HybridLayer, LinearScaling, MoeMlp, ParallelMixer, RotaryConfig,
                                  TalkingAttentionMixer, TimeMixMixer, fogizen_config_to_json)
from stkernel_b200.models.hybrid import init_random_weights


def att(heads=4, kv_heads=2, dim=20, vdim=28, scale=None, chunk=24, rot=12, base=700.0, factor=3.0):
    return TalkingAttentionMixer(heads, kv_heads, dim, vdim, scale or 1.6 * dim ** -0.5, chunk,
                                 RotaryConfig(base, rot, LinearScaling(factor), interleaved=True))


def tm(heads=3, dim=20, rank=None):
    return TimeMixMixer(heads, dim, rank)


def both(left=None, right=None):
    return ParallelMixer(left or att(), right or tm(), 0.5, 0.5, True)


def dense(ff=72):
    return DenseMlp(ff, "xielu")


def moe(experts=6, top=2, ff=40, groups=3, keep=2, scale=1.3):
    return MoeMlp(experts, top, ff, "silu", False, scoring="sigmoid", groups=groups, keep=keep, scale=scale)


def config(*layers, vocab=211, width=88, dtype="float32", eps=1e-5, bigram=(97, 13, 5)):
    """layers: mixers (with a dense feed-forward), or (mixer, feed-forward)."""
    out = tuple(HybridLayer(*l) if isinstance(l, tuple) else HybridLayer(l, dense()) for l in layers)
    cfg = HybridConfig(vocab, width, out, eps, 1.0, dtype, architecture="Fogizen", block="shifted", bigram=BigramTable(*bigram))
    cfg.validate()
    return cfg


def plain(dtype, **kw):
    """Experts that every token takes all of: no close decisions."""
    return config(both(), (both(att(3, 1, 16, 16, chunk=40, rot=16), tm(2, 12, 5)), moe(3, 3, 24, 1, 1)), (both(att(2, 2, 24, 8, chunk=7)), None),
                  dtype=dtype, **kw)


def mixed(dtype, **kw):
    """Routers that choose."""
    return config((both(), moe()), both(att(6, 2, 16, 24, chunk=33)), (both(), moe(8, 3, 24, 2, 1, 0.7)), dtype=dtype, **kw)


def weights(cfg, seed=0):
    """Random weights with routers that decide clearly.  Rounded to bf16 so that every compute type runs the same model."""
    w = init_random_weights(cfg, seed)
    for k in w:
        if k.endswith(".router"):
            w[k] = w[k] * 3.0
        w[k] = w[k].to(torch.bfloat16).float()
    return w


def oracle(cfg, w, toks):
    return O.logits(fogizen_config_to_json(cfg), w, toks)


def clear_routing(cfg, w, toks, margin):
    """Tokens of the sequence up to the first one that some router decides by less than `margin` (a compute type with rounding may
    take another expert there, and what follows sees it)."""
    seen = []
    keep = O.route

    def watch(z, correction, r):
        s = O.sigmoid(z) + correction
        n, k = len(z) // r["groups"]["count"], r["groups"]["keep"]
        score = torch.stack([s[g * n:(g + 1) * n].topk(min(2, n)).values.sum() for g in range(r["groups"]["count"])])
        order = score.sort(descending=True)
        gap = 9.0 if k == len(score) else float(order.values[k - 1] - order.values[k])
        open_ = torch.cat([s[g * n:(g + 1) * n] for g in order.indices[:k].tolist()]).sort(descending=True).values
        if r["top"] < len(open_):
            gap = min(gap, float(open_[r["top"] - 1] - open_[r["top"]]))
        seen.append(gap)
        return keep(z, correction, r)

    O.route = watch
    try:
        O.hidden_states(fogizen_config_to_json(cfg), w, toks)
    finally:
        O.route = keep
    if not seen:
        return len(toks)
    narrow = (torch.tensor(seen).view(-1, len(toks)).min(0).values < margin).nonzero().flatten()
    return int(narrow[0]) if len(narrow) else len(toks)


def needle(cfg, at, n, q_token=1, k_token=2, seed=3):
    """A one-layer model whose last token (q_token) gives nearly all its attention to token k_token at place `at` if it sees it (None: the
    sequence has no such token), and in which nothing but that attention carries anything from one token to another."""
    m, W = cfg.layers[0].mixer.left, cfg.hidden_size
    assert len(cfg.layers) == 1 and m.rotary.dims < m.dim
    w = weights(cfg, seed)
    e = w["embed"]
    e[:, :2] = 0
    e[k_token, 0] = 6.0
    e[q_token, 1] = 6.0
    w["bigram"] = torch.zeros_like(w["bigram"])
    w["l0.shift"] = torch.zeros(W)
    w["l0.norm1"] = torch.ones(W)
    w["l0.mix.right.out"] = torch.zeros(W)
    d = m.dim - 1                                             # a dimension that does not turn
    for name, axis, heads in (("q", 1, m.heads), ("k", 0, m.kv_heads)):
        x = w[f"l0.mix.left.{name}"].view(heads, m.dim, W) * 0.3
        x[:, d] = 0
        x[:, d, axis] = 12.0                                  # this dimension is all there is to the norm of the two tokens
        w[f"l0.mix.left.{name}"] = x.view(-1, W)
        w[f"l0.mix.left.{name}.b"] = torch.zeros(heads * m.dim)
        w[f"l0.mix.left.{name}.norm"] = torch.ones(m.dim)
    w["l0.mix.left.talk"] = torch.eye(m.heads) * 0.7 + 0.3 / m.heads
    w["l0.mix.left.out"] = 4.0 * torch.ones(W)
    for k in w:
        w[k] = w[k].to(torch.bfloat16).float()
    toks = [3 + x % (cfg.vocab_size - 3) for x in tokens(cfg, n, seed + 1)]
    toks[-1] = q_token
    if at is not None:
        toks[at] = k_token
    return w, toks


def with_layer(cfg, i, **kw):
    layers = list(cfg.layers)
    layers[i] = dataclasses.replace(layers[i], **kw)
    return dataclasses.replace(cfg, layers=tuple(layers))
