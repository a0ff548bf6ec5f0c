"""Configurations and weights shared by the tests of the latent-attention decoder."""
import torch

import domilix_oracle as O
from hybrid_util import error, feed, make_engine, tokens  # noqa: F401  (one import for the tests)
from stkernel_b200.config import DenseMlp, HybridConfig, HybridLayer, LatentAttentionMixer, MoeMlp, RotaryConfig, domilix_config_to_json
from stkernel_b200.models.hybrid import init_random_weights


def lat(heads=3, dim=20, rot=8, vdim=28, q_rank=44, kv_rank=36, kv_from=None, base=700.0, scale=None):
    return LatentAttentionMixer(heads, dim, rot, vdim, q_rank, kv_rank, scale or 1.2 * (dim + rot) ** -0.5,
                                RotaryConfig(base, rot, interleaved=True) if rot else None, kv_from)


def dense(ff=72):
    return DenseMlp(ff, "relu")


def moe(experts=6, top=2, ff=40):
    return MoeMlp(experts, top, ff)


def config(*layers, vocab=211, width=88, dtype="float32", eps=1e-5, scale=0.7):
    """layers: mixers (with a dense feed-forward), or (mixer, feed-forward)."""
    out = tuple(HybridLayer(*l) if isinstance(l, tuple) else HybridLayer(l, dense()) for l in layers)
    cfg = HybridConfig(vocab, width, out, eps, scale, dtype, architecture="Domilix", block="post_norm")
    cfg.validate()
    return cfg


def weights(cfg, seed=0, sharp=1.5):
    """Random weights whose attention singles keys out (scaled query and key expansions) and whose routers decide clearly.
    Rounded to bf16 so that every compute type runs the same model."""
    w = init_random_weights(cfg, seed)
    for k in w:
        if k.endswith((".mix.uq", ".mix.uk")):
            w[k] = w[k] * sharp
        if k.endswith(".router"):
            w[k] = w[k] * 4.0
        w[k] = w[k].to(torch.bfloat16).float()
    return w


def oracle(cfg, w, toks):
    return O.logits(domilix_config_to_json(cfg), w, toks)


# compute type -> (worst position, median position): with these weights bf16 rounding alone costs the reference path 0.09 at its
# worst position
LIMITS = {"float32": (1e-4, 2e-5), "bfloat16": (0.12, 0.03)}


def close(got, ref, dtype, factor=1.0):
    """Root mean square over the vocabulary of the centred difference, relative to the logits' spread, at every position."""
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    e = (d ** 2).mean(-1).sqrt() / ref.std()
    worst, median = LIMITS[dtype]
    assert e.max() < worst * factor and e.median() < median * factor, (e.max(), e.median())


def clear_routing(cfg, w, toks, margin):
    """Tokens of the sequence up to the first one that some router decides by less than `margin` (a compute type with rounding
    may take another expert there, and what follows sees it)."""
    seen = []
    keep = O.mixture

    def watch(h, ws, p, mlp):
        z = h @ ws[p + "router"].T + ws[p + "router.b"]
        top = z.topk(min(mlp["router"]["top"] + 1, z.shape[1]), -1).values
        seen.append(top[:, -2] - top[:, -1] if top.shape[1] > mlp["router"]["top"] else torch.full((len(h),), 9.0))
        return keep(h, ws, p, mlp)

    O.mixture = watch
    try:
        O.hidden_states(domilix_config_to_json(cfg), w, toks)
    finally:
        O.mixture = keep
    if not seen:
        return len(toks)
    narrow = (torch.stack(seen).min(0).values < margin).nonzero().flatten()
    return int(narrow[0]) if len(narrow) else len(toks)


def needle(cfg, at, n, q_token=1, k_token=2, seed=3):
    """A sequence whose last token (q_token) gives nearly all its weight in layer 0 to token k_token at place `at` (None: the
    sequence has no such token)."""
    m, W = cfg.layers[0].mixer, cfg.hidden_size
    w = weights(cfg, seed, sharp=0.2)
    e = w["embed"]
    ax = torch.eye(W)[:2]                                   # key direction, query direction
    e[:, :2] = 0
    e[k_token, 0] = e[q_token, 1] = 2.0
    for name, a in (("dkv", 0), ("dq", 1)):
        w[f"l0.mix.{name}"][:, :2] = 0
        w[f"l0.mix.{name}"][0] = 8.0 * ax[a]
    uk, uq = w["l0.mix.uk"].view(m.heads, m.dim, -1), w["l0.mix.uq"].view(m.heads, m.dim + m.rot_dim, -1)
    uk[:, 0], uq[:, 0] = 0, 0
    uk[:, 0, 0] = uq[:, 0, 0] = 3.0
    w["l0.mix.uv"][:, 0] = 0                                # what tells the key apart is not what it says
    for k in w:
        w[k] = w[k].to(torch.bfloat16).float()
    toks = [3 + x % (cfg.vocab_size - 3) for x in tokens(cfg, n, seed + 1)]
    toks[-1] = q_token
    if at is not None:
        toks[at] = k_token
    return w, toks
