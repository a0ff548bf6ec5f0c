"""Prefill and decode of the streams decoder (Fanulix: residual streams over Mamba-2 and attention beside retention, gelu experts with a
shared one) at sizes like a real model's layers, beside the closest decoders of the same width and depth: Timalorn (attention and
a matrix-memory recurrence) and Domilix (full-context attention and ungated experts), with every kernel's distance from its roofline.

    python bench.py --streams [--streams-sizes 2048,4096] [--streams-alone]

Measured as `hybrid_bench` measures (same functions, same prompt lengths and chunks).
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from ..config import HybridConfig, streams_stack
from ..ops import _lib
from ..ops.grouped import grouped_row
from ..ops.latent import PROMPT_SPAN
from ..ops.recurrence import CHUNK, CHUNK_SPAN
from . import hybrid_bench as HBench
from . import latent_bench as LBench

GROUPS = [("attention, prompt", ("latent_prompt_tc",)), ("attention, tokens", ("window_attn_tokens", "window_attn_tiles")),
          ("attention, merge", ("window_attn_combine",)), ("cached rows gather", ("latent_rows",)), ("attention prep + insert", ("grouped_prep",)),
          ("retention scan", ("RetentionFront",)), ("mamba2 scan", ("Mamba2Front",)), ("retention rotation", ("rotate_qk",)),
          ("retention chunk states", ("linear_chunk_state_kernel<true",)), ("retention chunk outputs", ("linear_chunk_out_kernel<true",)),
          ("mamba2 chunk states", ("linear_chunk_state_kernel<false",)), ("mamba2 chunk outputs", ("linear_chunk_out_kernel<false",)),
          ("retention finish", ("retention_finish",)), ("mamba2 convolution", ("mamba2_conv",)), ("mamba2 finish", ("mamba2_finish",)),
          ("stream mix + norm", ("stream_norm",)), ("experts", ("experts_wide", "experts_slim", "expert_rows")),
          ("expert sort + gather", ("moe_align", "expert_gather")), ("router", ("router_kernel", "gate_route")),
          ("embedding", ("embed_scaled",)), ("projections", ("gemm", "skinny"))]


def streams_config(width: int, layers: int, vocab: int) -> HybridConfig:
    """128-wide attention heads in groups of four, 128 x 256 retention states, Mamba-2 of twice the width with 64 x 128 states, the
    experts of `hybrid_bench.dsv4_config` and a shared one twice their size, four streams."""
    return streams_stack(layers, width, 4, heads=width // 128, kv_heads=width // 512, dim=128, vdim=128, ret_heads=width // 256,
                         ret_dim=128, ret_vdim=256, ssm_heads=width // 32, ssm_vdim=64, ssm_state=128, ssm_groups=8, experts=64, top=6,
                         expert_ff=width // 2, shared_ff=width, vocab=vocab)


def streams_work(cfg: HybridConfig, spans: List[Tuple[int, int]]) -> Dict[str, HBench.Work]:
    """Algorithmic work of one step over spans (start, tokens); every operand once."""
    out: Dict[str, List[float]] = {}

    def add(g: str, flops: float, byts: float) -> None:
        w = out.setdefault(g, [0.0, 0.0, 0.0])
        w[0] += flops
        w[1] += byts

    def product(t: float, n: float, k: float, out_bytes: float = 2.0) -> None:
        add("projections", 2.0 * t * n * k, 2.0 * n * k + 2.0 * t * k + out_bytes * t * n)

    def recurrence(name: str, H: int, D: int, V: int, qk: float, v: float) -> None:
        """qk, v: bytes of a token's queries and keys, and values."""
        state = H * D * V * 4.0
        if min(n for _, n in spans) < CHUNK_SPAN:
            add(f"{name} scan", 4.0 * T * H * D * V, 2 * state * len(spans) + T * (qk + v + 4.0 * H * V))
            return
        chunks = sum(-(-n // CHUNK) for _, n in spans)
        add(f"{name} chunk states", 2.0 * T * H * D * V, T * (qk / 2 + v) + chunks * state + 2 * state * len(spans))
        add(f"{name} chunk outputs", 2.0 * T * H * D * V + T * H * CHUNK * (D + V), T * (qk + v + 4.0 * H * V) + chunks * state)

    T, W, s = sum(n for _, n in spans), cfg.hidden_size, cfg.streams
    product(len(spans), cfg.vocab_size, W, 4.0)
    prompt = min(n for _, n in spans) >= PROMPT_SPAN
    rows = sum(a + n for a, n in spans)
    pairs = sum(HBench._keys(n, a, 1 << 40) for a, n in spans)
    for li, l in enumerate(cfg.layers):
        m = l.mixer
        if m.kind == "parallel":
            a, r = m.left, m.right
            H, G, D, V = a.heads, a.kv_heads, a.dim, a.vdim
            product(T, H * D + G * (D + V) + H * V + r.heads * 2 * (r.dim + r.vdim), W)
            product(T, W, m.out_dim, 4.0)
            row = grouped_row(D, V)[0] * 2.0 * G
            add("attention prep + insert", 0, T * (4.0 * H * D + 2.0 * G * (D + V) + row))
            g = "attention, prompt" if prompt else "attention, tokens"
            add(g, 2.0 * pairs * H * (D + V), rows * row + 2.0 * T * H * (D + 2 * V))
            if prompt:
                add("cached rows gather", 0, 2 * rows * row)
                add("retention rotation", 0, T * r.heads * r.dim * 2 * (2.0 + 4.0))
            recurrence("retention", r.heads, r.dim, r.vdim, r.heads * r.dim * (8.0 if prompt else 4.0), 2.0 * r.out_dim)
            add("retention finish", 0, T * r.out_dim * (4.0 + 2 + 2))
        else:
            H, V, N, G = m.heads, m.vdim, m.state, m.groups
            product(T, m.out_dim + m.conv_dim + H, W)
            product(T, W, m.out_dim, 4.0)
            if prompt:
                add("mamba2 convolution", 0, T * (4.0 * m.conv_dim + 10.0 * H))
            recurrence("mamba2", H, N, V, 4.0 * G * N, 2.0 * H * V)
            add("mamba2 finish", 0, T * m.out_dim * (4.0 + 2 + 2))
        first = 0.0 if li == 0 else 4.0 + 4.0 * s                                # output of the sublayer before, streams written back
        add("stream mix + norm", 0, T * W * (4.0 * s + first + 2))
        if l.mlp is None:
            continue
        E, top, F, n = l.mlp.experts, l.mlp.top, l.mlp.expert_width, l.mlp.shared_parts
        product(T, E, W, 4.0)
        used = E * (1.0 - (1.0 - top / E) ** T) + n
        add("experts", 4.0 * T * (top + n) * W * F, used * 4.0 * W * F + T * (top + n) * (4.0 * W + 4.0 * F))
        add("expert sort + gather", 0, 4.0 * T * (top + n) * W)
        add("stream mix + norm", 0, T * W * (4.0 * s + 4 + 4.0 * s + 2))
        # the experts' rows are summed where the next norm is formed
        add("stream mix + norm", 0, T * W * (2.0 * (top + n) - 4.0))
    add("stream mix + norm", 0, len(spans) * W * (4.0 * s + 2))
    add("embedding", 0, T * W * (2.0 + 4.0 * s))
    return {g: tuple(v) for g, v in out.items()}


def run(widths: List[int], layers: int = 4, vocab: int = 32768, ctx: int = 4096, batches=(1, 8, 64), profile: bool = True,
        beside: bool = True) -> Dict:
    pdl = _lib.query("stk_pdl_enabled")
    res: Dict = {"peaks": HBench.peaks(), "layers": layers, "vocab": vocab, "prefill_tokens": 4 * HBench.CHUNK, "decode_context": ctx}
    for width in widths:
        models = [("fanulix", streams_config(width, layers, vocab), GROUPS, streams_work, streams_work)]
        if beside:
            t = HBench.hybrid_config(width, layers, vocab)
            models.append(("timalorn", t, HBench.HYBRID_GROUPS, lambda c, s: HBench.hybrid_work(c, s, False),
                           lambda c, s: HBench.hybrid_work(c, s, True)))
            models.append(("domilix", LBench.latent_config(width, layers, vocab), LBench.GROUPS, LBench.latent_work, LBench.latent_work))
        for name, cfg, groups, work, decode_work in models:
            r: Dict = {"prefill_tok_s": round(HBench.time_prefill(cfg, 4 * HBench.CHUNK)), "decode": {}}
            for b in batches:
                r["decode"][str(b)] = HBench.time_decode(cfg, b, ctx)
            if profile:
                _lib.call("stk_set_pdl", 0)
                try:
                    r["prefill_kernels"] = HBench.profile_prefill(cfg, groups, lambda s: work(cfg, s))
                    r["decode_kernels"] = {str(b): HBench.profile_decode(cfg, groups, lambda s: decode_work(cfg, s), b, ctx)
                                           for b in (batches[0], batches[-1])}
                finally:
                    _lib.call("stk_set_pdl_mask", pdl)
            res[f"{name} width {width}"] = r
    return res


def main() -> None:
    """One op of a layer on its own (profilers): `python -m stkernel_b200.bench.streams_bench --op retention|mamba2|attention|norm`."""
    import argparse
    from ..models.hybrid import build_block
    from ..models.registry import family_of
    from ..models.sources import RandomSource
    from ..ops import grouped as GA
    from ..ops import hybrid as HB
    from ..ops import recurrence as RC
    ap = argparse.ArgumentParser()
    ap.add_argument("--op", choices=("retention", "mamba2", "attention", "norm"), required=True)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--tokens", type=int, default=4096, help="prompt tokens, or with --decode decode rows")
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--decode", action="store_true")
    ap.add_argument("--repeat", type=int, default=3)
    a = ap.parse_args()
    dev, n, ctx = torch.device("cuda:0"), a.tokens, a.context
    cfg = streams_config(a.width, 2, 1024)
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    spans = [(ctx, 1)] * n if a.decode else [(ctx, n)]
    pos = torch.full((n,), ctx, dtype=torch.int64, device=dev) if a.decode else torch.arange(ctx, ctx + n, device=dev)
    tok = torch.arange(n, dtype=torch.int32, device=dev) if a.decode else i32([0] * n)
    meta = HB.HybridMeta(pos, tok, pos, i32([ctx] * n), pos.to(torch.int32) if a.decode else i32([ctx + n - 1] * n),
                         i32(list(range(n + 1)) if a.decode else [0, n]), i32(list(range(len(spans)))), i32([ctx] * len(spans)), len(spans),
                         max(k for _, k in spans), a.decode, min(k for _, k in spans), tuple(spans), max_context=ctx + n)
    if a.op == "norm":
        s, W = cfg.streams, cfg.hidden_size
        sw = HB.StreamWeights(rnd(s), rnd(s), rnd(s, s))
        x, y, w, b = rnd(n, s, W), rnd(n, W), rnd(W), rnd(W)
        run_op = lambda: HB.stream_norm(x, y, sw, sw.read, w, b, 1e-6, W, torch.bfloat16)
    else:
        li = 0 if a.op == "mamba2" else 1
        assert family_of(cfg).name == "hybrid"
        blk, m = build_block(cfg, RandomSource(0), li, dev), cfg.layers[li].mixer
        p = rnd(n, blk.w_in.out_features).to(torch.bfloat16)
        c = torch.empty(n, blk.w_out.in_features, dtype=torch.bfloat16, device=dev)
        sg = blk.seg
        if a.op == "mamba2":
            st = (rnd(len(spans), m.heads, m.state, m.vdim), rnd(len(spans), m.conv - 1, m.conv_dim).to(torch.bfloat16))
            run_op = lambda: RC.mamba2(p, sg["z"], sg["xbc"], sg["dt"], blk.mamba2, meta, st, c)
        elif a.op == "retention":
            r = m.right
            st = (rnd(len(spans), r.heads, r.dim, r.vdim),)
            run_op = lambda: RC.retention(p, sg["right.q"], sg["right.k"], sg["right.v"], sg["right.g"], blk.retention, meta, st, c, m.left.out_dim)
        else:
            l = m.left
            pages = (ctx + (1 if a.decode else n)) // 64 + 1
            cache = rnd(pages * len(spans), l.kv_heads, 64, grouped_row(l.dim, l.vdim)[0]).to(torch.bfloat16)
            table = torch.arange(pages * len(spans), dtype=torch.int32, device=dev).view(len(spans), pages)

            def run_op():
                q = GA.grouped_prep(p, sg["left.q"], sg["left.k"], sg["left.v"], blk.grouped, meta, table, cache)
                GA.grouped_attention(p, q, sg["left.g"], blk.grouped, meta, table, cache, c)
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
