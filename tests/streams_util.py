"""Configurations and weights shared by the tests of the streams decoder (Fanulix)."""
import dataclasses

import torch

import fanulix_oracle as O
from hybrid_util import error, feed, make_engine, tokens  # noqa: F401  (one import for the tests)
from stkernel_b200.config import (GroupedAttentionMixer, HybridConfig, HybridLayer, Mamba2Mixer, MoeMlp, ParallelMixer, QueryTemperature,
                                  RetentionMixer, RotaryConfig, fanulix_config_to_json)
from stkernel_b200.models.hybrid import init_random_weights


def att(heads=4, kv_heads=2, dim=20, vdim=28, scale=None, coef=0.4, every=11):
    return GroupedAttentionMixer(heads, kv_heads, dim, vdim, scale or 1.6 * dim ** -0.5, QueryTemperature(coef, every))


def ret(heads=3, dim=16, vdim=20, rot=12, base=700.0, decay=None):
    decay = decay or tuple(1.0 - 2.0 ** (-2.0 - 3.0 * i) for i in range(heads))
    return RetentionMixer(heads, dim, vdim, tuple(decay), RotaryConfig(base, rot))


def both(left=None, right=None, ls=0.8, rs=0.55):
    return ParallelMixer(left or att(), right or ret(), ls, rs)


def ssm(heads=4, vdim=24, state=20, groups=2, conv=4, norm_groups=2):
    return Mamba2Mixer(heads, vdim, state, groups, conv, norm_groups)


def moe(experts=6, top=2, ff=40, shared=72):
    return MoeMlp(experts, top, ff, "gelu", False, shared)


def config(*layers, vocab=211, width=88, streams=2, dtype="float32", eps=1e-5, logit_scale=0.7):
    """layers: mixers (with a mixture of experts that takes them all: no close decisions), or (mixer, feed-forward)."""
    out = tuple(HybridLayer(*l) if isinstance(l, tuple) else HybridLayer(l, moe(3, 3)) for l in layers)
    cfg = HybridConfig(vocab, width, out, eps, 1.0, dtype, architecture="Fanulix", block="streams", streams=streams, tied_head=True,
                       logit_scale=logit_scale)
    cfg.validate()
    return cfg


def plain(dtype, **kw):
    return config(both(), ssm(), (both(att(3, 1, 16, 16), ret(2, 12, 24, 8)), None), (ssm(3, 16, 12, 1, 3, 1), moe(2, 2, 24, 30)),
                  dtype=dtype, **kw)


def mixed(dtype, **kw):
    """Routers that choose."""
    return config((both(), moe()), (ssm(), moe(5, 3, 24, 24)), (ssm(2, 16, 12, 2, 2, 1), None), dtype=dtype, **kw)


def weights(cfg, seed=0):
    """Random weights with routers that decide clearly.  Rounded to bf16 so that every compute type runs the same model."""
    w = init_random_weights(cfg, seed)
    for k in w:
        if k.endswith(".router"):
            w[k] = w[k] * 3.0
        w[k] = w[k].to(torch.bfloat16).float()
    return w


def oracle(cfg, w, toks):
    return O.logits(fanulix_config_to_json(cfg), w, toks)


# compute type -> (limit of a position, median position).  A few positions in a hundred are ill-conditioned (a retention head whose
# read-out nearly cancels before its norm): bf16 rounding alone costs the reference path up to 0.17 there and 0.03 elsewhere.
LIMITS = {"float32": (1e-4, 2e-5), "bfloat16": (0.12, 0.03)}


def close(got, ref, dtype, factor=1.0):
    """Root mean square over the vocabulary of the centred difference, relative to the logits' spread, at every position.  With
    rounding, one position in forty may be up to three times over the limit."""
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    e = (d ** 2).mean(-1).sqrt() / ref.std()
    limit, median = LIMITS[dtype]
    over = int((e > limit * factor).sum())
    assert over <= (len(e) // 40 if dtype == "bfloat16" else 0) and e.max() < 3 * limit * factor, (e.max(), e.argmax(), over)
    assert e.median() < median * factor, e.median()


def clear_routing(cfg, w, toks, margin):
    """Tokens of the sequence up to the first one that some router decides by less than `margin` (a compute type with rounding
    may take another expert there, and what follows sees it)."""
    seen = []
    keep = O.mixture

    def watch(h, ws, p, mlp):
        z = h @ ws[p + "router"].T
        top = z.topk(min(mlp["router"]["top"] + 1, z.shape[1]), -1).values
        seen.append(top[:, -2] - top[:, -1] if top.shape[1] > mlp["router"]["top"] else torch.full((len(h),), 9.0))
        return keep(h, ws, p, mlp)

    O.mixture = watch
    try:
        O.hidden_states(fanulix_config_to_json(cfg), w, toks)
    finally:
        O.mixture = keep
    if not seen:
        return len(toks)
    narrow = (torch.stack(seen).min(0).values < margin).nonzero().flatten()
    return int(narrow[0]) if len(narrow) else len(toks)


def needle(cfg, at, n, q_token=1, k_token=2, seed=3):
    """A model whose first layer is a parallel mixer, and a sequence whose last token (q_token) gives nearly all its attention there to
    token k_token at place `at` (None: the sequence has no such token)."""
    m, W = cfg.layers[0].mixer.left, cfg.hidden_size
    w = weights(cfg, seed)
    ax = torch.zeros(2, W)                                    # directions that the removal of the mean leaves alone
    ax[0, 0], ax[0, 1], ax[1, 2], ax[1, 3] = 0.7, -0.7, 0.7, -0.7
    e = w["embed"]
    e[:, :4] = 0
    e[k_token] = e[k_token] + 4.0 * ax[0]
    e[q_token] = e[q_token] + 4.0 * ax[1]
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(W), torch.zeros(W)
    for name, a, heads in (("q", ax[1], m.heads), ("k", ax[0], m.kv_heads)):
        x = w[f"l0.mix.left.{name}"].view(heads, m.dim, W) * 0.3
        x[:, 0] = 12.0 * a                                    # this dimension is all there is to the norm of the two tokens
        w[f"l0.mix.left.{name}"] = x.view(-1, W)
        w[f"l0.mix.left.{name}.b"] = torch.zeros(heads * m.dim)
    w["l0.mix.left.o"] = 4.0 * w["l0.mix.left.o"]
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
