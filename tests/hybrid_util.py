"""Configurations, weights and drivers shared by the CPU and GPU tests of the hybrid decoder."""
import torch

import timalorn_oracle as O
from stkernel_b200.config import (AttentionMixer, CacheConfig, DenseMlp, EngineConfig, HybridConfig, HybridLayer, MlstmMixer,
                                  RotaryConfig, SchedulerConfig, YarnScaling, timalorn_config_to_json)
from stkernel_b200.models.hybrid import build_hybrid_weights, init_random_weights
from stkernel_b200.models.sources import DictSource
from stkernel_b200.runtime.engine import Engine

YARN = YarnScaling(4.0, 96, 6.0, 0.75)


def attn(heads=4, kv_heads=2, dim=24, window=20, rot=8, scale=None, cap=12.0, base=3000.0, yarn=YARN):
    return AttentionMixer(heads, kv_heads, dim, window, scale or 1.3 * dim ** -0.5,
                          RotaryConfig(base, rot, yarn) if rot else None, cap)


def rec(heads=3, dim=16, vdim=24, cap=8.0):
    return MlstmMixer(heads, dim, vdim, cap)


def config(*layers, vocab=211, width=88, dtype="float32", eps=1e-5, scale=6.0):
    """layers: mixers, or (mixer, ff) / (mixer, ff, weights_of)."""
    out = []
    for l in layers:
        m, ff, of = (l + (None,) * (3 - len(l))) if isinstance(l, tuple) else (l, 72, None)
        out.append(HybridLayer(m, DenseMlp(ff) if ff else None, of))
    cfg = HybridConfig(vocab, width, tuple(out), eps, scale, dtype)
    cfg.validate()
    return cfg


def weights(cfg, seed=0, sharp=1.6, sink=1.0):
    """Random weights whose attention singles keys out (scaled q and k) and whose sinks matter.  Rounded to bf16 so that every
    compute type runs the same model."""
    w = init_random_weights(cfg, seed)
    for k in w:
        if k.endswith((".mix.q", ".mix.k")):
            w[k] = w[k] * sharp
        if k.endswith(".sink"):
            w[k] = torch.randn(w[k].shape, generator=torch.Generator().manual_seed(seed + 5)) * sink
        w[k] = w[k].to(torch.bfloat16).float()
    return w


def make_engine(cfg, w, device="cpu", ctx=640, seqs=6, chunk=640, graph_cap=0, **sched):
    ec = EngineConfig(model=cfg, sched=SchedulerConfig(max_model_len=ctx, max_num_seqs=seqs, max_num_batched_tokens=chunk,
                                                       graph_cap=graph_cap, **sched), cache=CacheConfig()).validate()
    return Engine(ec, build_hybrid_weights(cfg, DictSource(w), device), device, max_context=ctx)


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(eng, toks, cuts=None, close=True):
    """Logits of every position of one sequence, its tokens cut into portions (the last size repeats)."""
    r = eng.open_sequence()
    out, at, i = [], 0, 0
    cuts = cuts or [len(toks)]
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(eng.feed([(r, toks[at:at + n], list(range(n)))]).double().cpu())
        at, i = at + n, i + 1
    if close:
        eng.close_sequence(r)
    return torch.cat(out)


def oracle(cfg, w, toks):
    return O.logits(timalorn_config_to_json(cfg), w, toks)


def error(got, ref):
    """Root mean square over the vocabulary of the centred difference, relative to the logits' spread: worst position."""
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return float(((d ** 2).mean(-1).sqrt() / ref.std()).max())


def needle(cfg, at, n, layer=0, q_token=1, k_token=2, gain=1.4, seed=3):
    """A one-attention-layer model and a sequence in which token `q_token` (last place) looks for token `k_token` (place
    `at`): their embeddings share a direction that the query and key projections pick out, all other tokens lack it."""
    m = cfg.layers[layer].mixer
    w = weights(cfg, seed, sharp=0.3, sink=0.3)
    W = cfg.hidden_size
    e = w["embed"] - w["embed"].mean(0)
    ax = torch.zeros(W)
    ax[0], ax[1] = 1.0, -1.0                              # a direction that the mean removal of the norm leaves alone
    ax = ax / ax.norm()
    e = e - (e @ ax)[:, None] * ax
    e[k_token] = e[k_token] + ax
    e[q_token] = e[q_token] + ax
    w["embed"] = e.to(torch.bfloat16).float()
    w[f"l{layer}.norm1"] = torch.ones(W)
    d = m.dim - 1                                         # an unrotated dimension
    assert d >= m.rot_dims
    q = w[f"l{layer}.mix.q"].view(m.heads, m.dim, W)
    k = w[f"l{layer}.mix.k"].view(m.kv_heads, m.dim, W)
    q[:, d] = gain * ax
    k[:, d] = gain * ax
    # the shared dimension is the same for both keys: the read-out ignores it and weighs the rest
    o = 12.0 * w[f"l{layer}.mix.o"].view(W, m.heads, m.dim)
    o[:, :, d] = 0
    w[f"l{layer}.mix.o"] = o.reshape(W, -1)
    for nme in ("q", "k", "o"):
        w[f"l{layer}.mix.{nme}"] = w[f"l{layer}.mix.{nme}"].to(torch.bfloat16).float()
    toks = [3 + x % (cfg.vocab_size - 3) for x in tokens(cfg, n, seed + 1)]
    toks[-1] = q_token
    if at is not None:
        toks[at] = k_token
    return w, toks


