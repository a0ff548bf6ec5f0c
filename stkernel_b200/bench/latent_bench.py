"""Prefill and decode of the latent-attention decoder (Domilix: latent attention, ungated bf16 experts, post-norm blocks) at sizes like
a real model's layers, beside the DeepSeek-V4-style decoder of the same width, depth and expert counts, with every kernel's distance
from its roofline.

    python bench.py --latent [--latent-sizes 2048,4096]

Measured as `hybrid_bench` measures (same functions, same prompt lengths and chunks).
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from ..config import HybridConfig, latent_stack
from ..ops import _lib
from ..ops.latent import PROMPT_SPAN, latent_row
from . import hybrid_bench as HBench

GROUPS = [("latent attention, prompt", ("latent_prompt_tc",)), ("latent attention, tokens", ("latent_tokens_tc", "latent_attn_simt")),
          ("latent attention, merge", ("latent_merge",)), ("cached rows gather", ("latent_rows",)), ("latent norms + insert", ("latent_prep",)),
          ("post norm + add", ("post_norm_add",)), ("experts", ("experts_wide", "experts_slim", "expert_rows")),
          ("expert sort + gather", ("moe_align", "expert_gather")), ("router", ("router_kernel", "gate_route")),
          ("feed-forward join", ("join_glu",)), ("embedding", ("embed_scaled",)), ("final norm", ("add_layer_norm",)),
          ("projections", ("gemm", "skinny"))]


def latent_config(width: int, layers: int, vocab: int) -> HybridConfig:
    """128-wide heads, 64 rotated dimensions, latents of 512; the experts of `hybrid_bench.dsv4_config`; the last layer shares the
    latents of the one before it."""
    return latent_stack(layers, width, heads=width // 128, dim=128, rot_dim=64, vdim=128, q_rank=width * 3 // 8, kv_rank=512,
                        ff=width * 11 // 4, experts=64, top=6, expert_ff=width // 2, vocab=vocab, share_from=layers - 2)


def latent_work(cfg: HybridConfig, spans: List[Tuple[int, int]]) -> Dict[str, HBench.Work]:
    """Algorithmic work of one step over spans (start, tokens); every operand once."""
    out: Dict[str, List[float]] = {}

    def add(g: str, flops: float, byts: float) -> None:
        w = out.setdefault(g, [0.0, 0.0, 0.0])
        w[0] += flops
        w[1] += byts

    def product(t: float, n: float, k: float, out_bytes: float = 2.0, blocks: int = 1) -> None:
        """t rows through an [n, k] weight (blocks > 1: block-diagonal, k per block)."""
        add("projections", 2.0 * t * n * k, 2.0 * n * k + 2.0 * t * k * blocks + out_bytes * t * n)

    T, W = sum(n for _, n in spans), cfg.hidden_size
    product(len(spans), cfg.vocab_size, W, 4.0)
    prompt = min(n for _, n in spans) >= PROMPT_SPAN
    rows = sum(s + n for s, n in spans)
    pairs = sum(HBench._keys(n, s, 1 << 40) for s, n in spans)
    for li, l in enumerate(cfg.layers):
        m = l.mixer
        H, D, R, V, C, Q = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank
        row = latent_row(C, R)[0] * 2.0
        n_in = Q + H + (C + R if m.kv_from is None else 0)
        product(T, n_in, W, 4.0)
        product(T, H * (D + R), Q)
        product(T, W, H * V, 4.0)
        add("latent norms + insert", 0, T * (4.0 * n_in + 2.0 * Q + (row if m.kv_from is None else 0)))
        if prompt:
            product(rows, H * (D + V), C)
            if li == 0 or cfg.cache_layer(li) != cfg.cache_layer(li - 1):
                add("cached rows gather", 0, 2 * rows * row)
            add("latent attention, prompt", 2.0 * pairs * H * (D + R + V), rows * (2.0 * H * (D + V) + 2.0 * R) + 2.0 * T * H * (D + R + V))
        else:
            product(T, H * C, D, blocks=H)
            product(T, H * V, C, blocks=H)
            add("latent attention, tokens", 2.0 * pairs * H * (2 * C + R), rows * row + 2.0 * T * H * (C + R) + 4.0 * T * H * C)
            add("latent attention, merge", 0, 6.0 * T * H * C)
        add("post norm + add", 0, T * W * (4 + 4 + 4 + 2.0))
        if l.mlp is None:
            continue
        if l.mlp.kind == "dense":
            product(T, 2 * l.mlp.ff, W)
            product(T, W, l.mlp.ff, 4.0)
            add("feed-forward join", 0, 6.0 * T * l.mlp.ff)
            add("post norm + add", 0, T * W * (4 + 4 + 4 + 2.0))
        else:
            E, top, F = l.mlp.experts, l.mlp.top, l.mlp.ff
            product(T, E, W, 4.0)
            used = E * (1.0 - (1.0 - top / E) ** T)
            add("experts", 4.0 * T * top * W * F, used * 4.0 * W * F + T * top * (4.0 * W + 4.0 * F))
            add("expert sort + gather", 0, 4.0 * T * top * W)
            add("post norm + add", 0, T * W * (2.0 * top + 4 + 4 + 2.0))
    add("embedding", 0, T * W * 8.0)
    return {g: tuple(v) for g, v in out.items()}


def dsv4_work(cfg, spans) -> Dict[str, HBench.Work]:
    """The like kernels of the other family, experts included (NVFP4 weights: 4.5 bits each)."""
    w = HBench.dsv4_work(cfg, spans)
    T, H, I = sum(n for _, n in spans), cfg.hidden_size, cfg.moe_intermediate_size
    E, top, L = cfg.n_routed_experts, cfg.num_experts_per_tok, cfg.num_hidden_layers
    used = E * (1.0 - (1.0 - top / E) ** T)
    w["experts"] = (L * 6.0 * T * top * H * I, L * (used * 3.0 * H * I * 4.5 / 8 + T * top * (4.0 * H + 4.0 * I)), 0.0)
    return w


def run(widths: List[int], layers: int = 4, vocab: int = 32768, ctx: int = 4096, batches=(1, 8, 64), profile: bool = True,
        beside: bool = True) -> Dict:
    pdl = _lib.query("stk_pdl_enabled")
    res: Dict = {"peaks": HBench.peaks(), "layers": layers, "vocab": vocab, "prefill_tokens": 4 * HBench.CHUNK, "decode_context": ctx}
    for width in widths:
        models = [("domilix", latent_config(width, layers, vocab), GROUPS, latent_work)]
        if beside:
            models.append(("deepseek-v4-style", HBench.dsv4_config(width, layers, vocab), HBench.DSV4_GROUPS, dsv4_work))
        for name, cfg, groups, work in models:
            r: Dict = {"prefill_tok_s": round(HBench.time_prefill(cfg, 4 * HBench.CHUNK)), "decode": {}}
            for b in batches:
                r["decode"][str(b)] = HBench.time_decode(cfg, b, ctx)
            if profile:
                _lib.call("stk_set_pdl", 0)
                try:
                    r["prefill_kernels"] = HBench.profile_prefill(cfg, groups, lambda s: work(cfg, s))
                    r["decode_kernels"] = {str(b): HBench.profile_decode(cfg, groups, lambda s: work(cfg, s), b, ctx)
                                           for b in (batches[0], batches[-1])}
                finally:
                    _lib.call("stk_set_pdl_mask", pdl)
            res[f"{name} width {width}"] = r
    return res


def main() -> None:
    """One op of a layer on its own (profilers): `python -m stkernel_b200.bench.latent_bench --op prompt|tokens|experts`."""
    import argparse
    from ..models.hybrid import build_latent
    from ..models.sources import RandomSource
    from ..ops import hybrid as HB
    from ..ops import latent as LA
    from ..ops import moe as MO
    ap = argparse.ArgumentParser()
    ap.add_argument("--op", choices=("prompt", "tokens", "experts"), required=True)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--tokens", type=int, default=4096, help="prompt tokens, decode rows, or tokens through the experts")
    ap.add_argument("--context", type=int, default=8192)
    ap.add_argument("--repeat", type=int, default=3)
    a = ap.parse_args()
    dev, n, ctx = torch.device("cuda:0"), a.tokens, a.context
    cfg = latent_config(a.width, 3, 1024)
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev).to(torch.bfloat16)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    if a.op == "experts":
        e = cfg.layers[1].mlp
        ex = MO.PlainExperts(rnd(e.experts, e.ff, a.width) * 0.02, rnd(e.experts, a.width, e.ff) * 0.02)
        ids = torch.rand(n, e.experts, generator=g, device=dev).topk(e.top).indices.to(torch.int32)
        x, wts = rnd(n, a.width), torch.full((n, e.top), 1.0 / e.top, device=dev)
        run_op = lambda: MO.plain_experts(x, ids, wts, ex)
    else:
        m = cfg.layers[0].mixer
        src, shapes = RandomSource(0), {"mix.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank), "mix.uk": (m.heads * m.dim, m.kv_rank),
                                        "mix.uv": (m.heads * m.vdim, m.kv_rank), "mix.dq.norm": (m.q_rank,), "mix.dkv.norm": (m.kv_rank,)}
        p = build_latent(cfg, lambda k: src.get(k, shapes[k], dev), m, torch.bfloat16, dev)
        prompt = a.op == "prompt"
        spans = [(ctx, n)] if prompt else [(ctx, 1)] * n
        pages = (ctx + (n if prompt else 1)) // 64 + 1
        pos = torch.arange(ctx, ctx + n, device=dev) if prompt else torch.full((n,), ctx, dtype=torch.int64, device=dev)
        last = i32([ctx + n - 1] * n) if prompt else i32([ctx] * n)
        tok = i32([0] * n) if prompt else torch.arange(n, dtype=torch.int32, device=dev)
        meta = HB.HybridMeta(pos, tok, pos, i32([ctx] * n), last, i32([0, n] if prompt else list(range(n + 1))),
                             i32(list(range(len(spans)))), i32([ctx] * len(spans)), len(spans), max(k for _, k in spans), not prompt,
                             min(k for _, k in spans), tuple(spans), max_context=ctx + n)
        cache = rnd(pages * len(spans), 64, LA.latent_row(m.kv_rank, m.rot_dim)[0])
        table = torch.arange(pages * len(spans), dtype=torch.int32, device=dev).view(len(spans), pages)
        q, gate = rnd(n, p.w_uq.out_features), torch.zeros(n, m.heads, device=dev)

        def run_op():
            meta.gathered.clear()
            LA.latent_attention(q, gate, p, meta, table, cache)
    e0, e1 = (torch.cuda.Event(enable_timing=True) for _ in range(2))
    for _ in range(a.repeat):
        e0.record()
        run_op()
        e1.record()
        torch.cuda.synchronize()
    _lib.check_status()
    print(f"{a.op} width {a.width} tokens {n} context {ctx}: {e0.elapsed_time(e1) * 1e3:.1f} us")


if __name__ == "__main__":
    main()
