"""Prefill and decode of the shifted decoder (Fogizen: talking-heads attention in chunks beside time mixing, gated experts chosen in groups, bigram
embedding) at sizes like a real model's layers, beside the closest decoders of the same width and depth: Fanulix (attention beside
retention, Mamba-2, gelu experts) and Domilix (latent attention, ungated experts), with every kernel's distance from its
roofline.

    python bench.py --shifted [--shifted-sizes 2048,4096] [--shifted-alone]

Measured as `hybrid_bench` measures (same functions, same prompt lengths and chunks).
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from ..config import HybridConfig, shifted_stack
from ..ops import _lib
from ..ops.latent import PROMPT_SPAN
from ..ops.recurrence import CHUNK, CHUNK_SPAN
from ..ops.talking import talking_row
from . import hybrid_bench as HBench
from . import latent_bench as LBench
from . import streams_bench as SBench

GROUPS = [("attention, prompt", ("talking_prompt_tc",)), ("attention, tokens", ("talking_tokens_tc", "talking_simt")),
          ("attention, merge", ("talking_merge",)), ("cached rows gather", ("talking_rows",)), ("attention prep + insert", ("talking_prep",)),
          ("time mixing scan", ("TimeMixFront",)), ("time mixing chunk keys", ("time_mix_keys",)),
          ("time mixing chunk states", ("linear_chunk_state_kernel",)), ("time mixing chunk outputs", ("time_mix_out",)),
          ("time mixing finish", ("retention_finish",)), ("decay tanh", ("tanh_rows",)), ("shifted norm", ("shifted_norm", "sum_norm", "shift_blend")),
          ("state commit", ("shift_commit",)), ("experts", ("experts_wide", "experts_slim", "expert_rows")),
          ("expert sort + gather", ("moe_align", "expert_gather")), ("router", ("router_kernel", "gate_route")), ("xielu", ("xielu",)),
          ("embedding", ("embed_bigram",)), ("projections", ("gemm", "skinny"))]


def shifted_config(width: int, layers: int, vocab: int) -> HybridConfig:
    """128-wide attention heads over four key/value heads, chunks of 8192, 64 x 64 time-mixing states with decays of rank width / 32, gated
    experts half as wide as the model (64 in 8 groups, 6 of the best 4 groups)."""
    return shifted_stack(layers, width, heads=width // 128, kv_heads=4, dim=128, vdim=128, chunk=8192, mix_heads=width // 64, mix_dim=64,
                         rank=width // 32, ff=width * 11 // 4, experts=64, top=6, groups=8, keep=4, expert_ff=width // 2, vocab=vocab)


def shifted_work(cfg: HybridConfig, spans: List[Tuple[int, int]]) -> Dict[str, HBench.Work]:
    """Algorithmic work of one step over spans (start, tokens); every operand once."""
    out: Dict[str, List[float]] = {}

    def add(g: str, flops: float, byts: float) -> None:
        w = out.setdefault(g, [0.0, 0.0, 0.0])
        w[0] += flops
        w[1] += byts

    def product(t: float, n: float, k: float, out_bytes: float = 2.0, blocks: int = 1) -> None:
        add("projections", 2.0 * t * n * k, 2.0 * n * k + 2.0 * t * k * blocks + out_bytes * t * n)

    T, W = sum(n for _, n in spans), cfg.hidden_size
    product(len(spans), cfg.vocab_size, W, 4.0)
    prompt = min(n for _, n in spans) >= PROMPT_SPAN
    for li, l in enumerate(cfg.layers):
        a, r = l.mixer.left, l.mixer.right
        H, G, D, V = a.heads, a.kv_heads, a.dim, a.vdim
        C = a.chunk or 1 << 40
        pairs = sum(p % C + 1 for s, n in spans for p in range(s, s + n))
        rows = sum(s + n - s // C * C for s, n in spans)
        row = talking_row(G, D, V)[0] * 2.0
        q_row = 2.0 * H * talking_row(G, D, V)[2] * G
        product(T, H * D + G * (D + V) + H, W)
        product(T, W, a.out_dim, 4.0)
        add("attention prep + insert", 2.0 * T * H * H * D, T * (2.0 * H * D + 2.0 * G * (D + V) + row + q_row))
        # scores of H heads, their mixture, values; the mixed queries are given
        add("attention, prompt" if prompt else "attention, tokens", 2.0 * pairs * H * (D + V + H), rows * row + T * (q_row + 2.0 * H * V))
        if prompt:
            add("cached rows gather", 0, 2 * rows * row)
        N, state = r.out_dim, r.heads * r.dim * r.dim * 4.0
        product(T, 4 * N, W, blocks=4)
        product(T, r.rank, W, 4.0)
        product(T, N, r.rank, 4.0)
        product(T, W, N, 4.0)
        add("decay tanh", 0, T * r.rank * 8.0)
        if min(n for _, n in spans) < CHUNK_SPAN:
            add("time mixing scan", 6.0 * T * N * r.dim, 2 * state * len(spans) + T * N * (6.0 + 4.0 + 4.0))
        else:
            chunks = sum(-(-n // CHUNK) for _, n in spans)
            add("time mixing chunk keys", 0, T * N * (2.0 + 4.0 + 4.0))
            add("time mixing chunk states", 2.0 * T * N * r.dim, T * N * (4.0 + 2.0) + chunks * state + 2 * state * len(spans))
            add("time mixing chunk outputs", 2.0 * T * N * r.dim + 2.0 * T * N * CHUNK, T * N * (6.0 + 4.0 + 4.0) + chunks * state)
        add("time mixing finish", 0, T * N * (4.0 + 2 + 2))
        # residual, both outputs and the feed-forward's rows in (from the second layer on), residual, norm, shifted row and blends out
        before = cfg.layers[li - 1].mlp if li else None
        tail = 0.0 if before is None else 4.0 if before.kind == "dense" else 2.0 * before.top
        add("shifted norm", 0, T * W * (4.0 + (4.0 + 8.0 + tail if li else 0.0) + 2.0 * 7))
        if l.mlp is None:
            continue
        if l.mlp.kind == "dense":
            product(T, l.mlp.ff, W)
            product(T, W, l.mlp.ff, 4.0)
            add("xielu", 0, 4.0 * T * l.mlp.ff)
            continue
        E, top, F = l.mlp.experts, l.mlp.top, l.mlp.ff
        product(T, E, W, 4.0)
        used = E * (1.0 - (1.0 - top / E) ** T)
        add("experts", 6.0 * T * top * W * F, used * 6.0 * W * F + T * top * (4.0 * W + 4.0 * F))
        add("expert sort + gather", 0, 4.0 * T * top * W)
    add("shifted norm", 0, len(spans) * W * (4.0 + 8.0 + 12.0 + 2.0))
    add("state commit", 0, len(spans) * len(cfg.layers) * 16.0 * W)
    add("embedding", 0, T * W * 8.0)
    return {g: tuple(v) for g, v in out.items()}


def run(widths: List[int], layers: int = 4, vocab: int = 32768, ctx: int = 4096, batches=(1, 8, 64), profile: bool = True,
        beside: bool = True) -> Dict:
    pdl = _lib.query("stk_pdl_enabled")
    res: Dict = {"peaks": HBench.peaks(), "layers": layers, "vocab": vocab, "prefill_tokens": 4 * HBench.CHUNK, "decode_context": ctx}
    for width in widths:
        models = [("fogizen", shifted_config(width, layers, vocab), GROUPS, shifted_work)]
        if beside:
            models.append(("fanulix", SBench.streams_config(width, layers, vocab), SBench.GROUPS, SBench.streams_work))
            models.append(("domilix", LBench.latent_config(width, layers, vocab), LBench.GROUPS, LBench.latent_work))
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
    """One op of a layer on its own (profilers): `python -m stkernel_b200.bench.shifted_bench --op attention|time_mix|norm`."""
    import argparse
    from ..models.hybrid import build_block
    from ..models.sources import RandomSource
    from ..ops import hybrid as HB
    from ..ops import recurrence as RC
    from ..ops import shifted as SH
    from ..ops import talking as TK
    ap = argparse.ArgumentParser()
    ap.add_argument("--op", choices=("attention", "time_mix", "norm"), required=True)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--tokens", type=int, default=4096, help="prompt tokens, or with --decode decode rows")
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--decode", action="store_true")
    ap.add_argument("--repeat", type=int, default=3)
    a = ap.parse_args()
    dev, n, ctx = torch.device("cuda:0"), a.tokens, a.context
    cfg = shifted_config(a.width, 1, 1024)
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    spans = [(ctx, 1)] * n if a.decode else [(ctx, n)]
    pos = torch.full((n,), ctx, dtype=torch.int64, device=dev) if a.decode else torch.arange(ctx, ctx + n, device=dev)
    tok = torch.arange(n, dtype=torch.int32, device=dev) if a.decode else i32([0] * n)
    meta = HB.HybridMeta(pos, tok, pos, i32([ctx] * n), pos.to(torch.int32) if a.decode else i32([ctx + n - 1] * n),
                         i32(list(range(n + 1)) if a.decode else [0, n]), i32(list(range(len(spans)))), i32([ctx] * len(spans)), len(spans),
                         max(k for _, k in spans), a.decode, min(k for _, k in spans), tuple(spans), max_context=ctx + n)
    blk, m, W = build_block(cfg, RandomSource(0), 0, dev), cfg.layers[0].mixer, cfg.hidden_size
    if a.op == "norm":
        st = SH.shift_state(1, len(spans), W, dev)
        x, y0, y1, f = (rnd(n, W) for _ in range(4))
        pend = SH.Pending([(y0, blk.out_norms[0], 0.5), (y1, blk.out_norms[1], 0.5)], f)
        run_op = lambda: SH.shifted_norm(x, pend, blk.norm, 1e-5, W, torch.bfloat16, blk.shift, blk.mu, st, 0, meta)
    elif a.op == "time_mix":
        p, z = rnd(n, blk.w_mixes.out_features).to(torch.bfloat16), rnd(n, blk.time_mix.np)
        c = torch.empty(n, blk.w_sides[1].in_features, dtype=torch.bfloat16, device=dev)
        st = (rnd(len(spans), m.right.heads, m.right.dim, m.right.dim),)
        run_op = lambda: RC.time_mix(p, z, blk.time_mix, meta, st, c)
    else:
        l, sg = m.left, blk.seg
        p = rnd(n, blk.w_in.out_features).to(torch.bfloat16)
        c = torch.empty(n, blk.w_sides[0].in_features, dtype=torch.bfloat16, device=dev)
        pages = (ctx + (1 if a.decode else n)) // 64 + 1
        cache = rnd(pages * len(spans), 64, talking_row(l.kv_heads, l.dim, l.vdim)[0]).to(torch.bfloat16)
        table = torch.arange(pages * len(spans), dtype=torch.int32, device=dev).view(len(spans), pages)

        def run_op():
            q, gate = TK.talking_prep(p, sg["left.q"], sg["left.k"], sg["left.v"], sg["left.g"], blk.talking, meta, table, cache)
            TK.talking_attention(q, gate, blk.talking, meta, table, cache, c)
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
