"""Prefill and decode of the hybrid decoder (Timalorn: windowed attention + mLSTM) at sizes like a real model's layers, beside the
DeepSeek-V4-style decoder of the same width and depth, with every kernel's distance from its roofline.

    python bench.py --hybrid [--hybrid-sizes 2048,4096]

Random weights and tokens.  Throughput: CUDA events around whole engine steps (decode steps replay captured graphs, tokens
forced, no host read-back).  Kernel times: torch profiler over eager steps with programmatic dependent launch off, so that a
kernel's time is its own.  Roofline of a kernel: the larger of its operations over the measured bf16 rate and its bytes over
the measured copy bandwidth; for the attention kernels with capped scores also the exponentials and reciprocals over the
special-function rate, given separately as `sfu_us`.
"""
from __future__ import annotations

import json
import os
import tempfile
from typing import Dict, List, Optional, Tuple

import torch

from ..config import EngineConfig, HybridConfig, SchedulerConfig, YarnScaling, flash_config, hybrid_stack
from ..models.registry import family_of
from ..models.sources import RandomSource
from ..ops import _lib
from ..runtime.engine import Engine, SamplingParams
from .decode_bench import timed_steps

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
CHUNK = 4096


def peaks() -> Dict[str, float]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return {"hbm_gbs": p["hbm_gbs"], "bf16_tflops": p["bf16_tflops"], "source": "measured"}
    except (OSError, KeyError, ValueError):
        return {**FALLBACK_PEAKS, "source": "fallback"}


def hybrid_config(width: int, layers: int, vocab: int) -> HybridConfig:
    """Layer shapes in proportion to the width: 128-wide attention heads in groups of four, 256 x 512 matrix memories."""
    return hybrid_stack(layers, width, heads=width // 128, kv_heads=width // 512, dim=128, window=width, ff=width * 11 // 4,
                        vocab=vocab, mlstm_heads=width // 512, mlstm_dim=256, mlstm_vdim=512,
                        yarn=YarnScaling(4.0, 4096, 32.0, 1.0))


def dsv4_config(width: int, layers: int, vocab: int):
    return flash_config(layers, hidden_size=width, vocab_size=vocab, n_routed_experts=64, moe_intermediate_size=width // 2)


def make_engine(cfg, ctx: int, seqs: int, graphs: bool) -> Engine:
    ec = EngineConfig(model=cfg, sched=SchedulerConfig(max_model_len=ctx, max_num_seqs=seqs, max_num_batched_tokens=CHUNK,
                                                       graph_cap=seqs if graphs else 0)).validate()
    fam = family_of(cfg)
    dev = torch.device("cuda:0")
    if not hasattr(make_engine, "weights"):
        make_engine.weights = {}
    key = id(cfg)
    if key not in make_engine.weights:
        make_engine.weights.clear()
        torch.cuda.empty_cache()
        make_engine.weights[key] = fam.build_weights(cfg, RandomSource(0), dev)
    return Engine(ec, make_engine.weights[key], dev, max_context=ctx)


def prompts(cfg, n: int, length: int, seed: int) -> List[List[int]]:
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg.vocab_size, (length,), generator=g).tolist() for _ in range(n)]


def time_prefill(cfg, length: int) -> float:
    """Tokens per second over one prompt, second pass (kernels warm)."""
    eng = make_engine(cfg, length + 64, 2, False)
    ms = []
    for rep in range(3):
        rid = eng.add_request(prompts(cfg, 1, length, rep)[0], SamplingParams(max_tokens=1))
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        while not eng.requests[rid].finished:
            eng.step()
        e1.record()
        torch.cuda.synchronize()
        ms.append(e0.elapsed_time(e1))
    _lib.check_status()
    return length / min(ms[1:]) * 1e3


def start_decode(cfg, batch: int, ctx: int, graphs: bool) -> Engine:
    """An engine with `batch` requests whose prompts of ctx tokens are computed (real prefill)."""
    eng = make_engine(cfg, ctx + 600, max(batch, 2), graphs)
    for p in prompts(cfg, batch, ctx, 7):
        eng.add_request(p, SamplingParams(max_tokens=500, ignore_eos=True))
    while eng.sched.waiting or any(r.in_prefill for r in eng.sched.running):
        eng.step()
    return eng


def time_decode(cfg, batch: int, ctx: int, steps: int = 48) -> Dict[str, float]:
    eng = start_decode(cfg, batch, ctx, True)
    timed_steps(eng, 6, 1, cfg.vocab_size, batch, False)
    runs = sorted(timed_steps(eng, steps, 1, cfg.vocab_size, batch, False)[0] for _ in range(3))
    _lib.check_status()
    return {"ms_per_step": round(runs[1], 4), "tok_s": round(batch * 1e3 / runs[1], 1)}


def kernel_times(step, steps: int) -> Dict[str, List[float]]:
    from .kernel_table import summarise_trace
    step()
    torch.cuda.synchronize()
    with torch.profiler.profile(activities=[torch.profiler.ProfilerActivity.CUDA]) as prof:
        for _ in range(steps):
            step()
        torch.cuda.synchronize()
    path = os.path.join(tempfile.gettempdir(), f"stk_hybrid_trace_{os.getpid()}.json")
    prof.export_chrome_trace(path)
    s = summarise_trace(path, steps)
    os.unlink(path)
    return s["kernels"]


# ---- rooflines ------------------------------------------------------------------------------------------
# group -> (pattern in the kernel name); work per step below uses the same group names
HYBRID_GROUPS = [("projections", ("gemm", "skinny")), ("window_attention", ("window_attn_tc", "window_attn_tiles", "window_attn_tokens")),
                 ("window_attention combine", ("window_attn_combine",)), ("kv insert", ("window_kv_insert",)),
                 ("add + layer norm", ("add_layer_norm",)), ("feed-forward join", ("join_glu",)),
                 ("mlstm scan", ("mlstm_scan_kernel",)), ("mlstm chunk states", ("mlstm_chunk_state",)),
                 ("mlstm chunk gates", ("mlstm_chunk_gates",)), ("mlstm chunk outputs", ("mlstm_chunk_out",)),
                 ("mlstm finish", ("mlstm_finish",)), ("embedding", ("embed_scaled",))]
DSV4_GROUPS = [("projections", ("gemm_", "skinny")), ("sparse attention", ("sparse_mla", "mla_decode")),
               ("sparse attention merge", ("mla_merge", "mla_combine")),
               ("kv insert", ("rope_kv_insert",)), ("rms norm", ("rmsnorm",)), ("stream mix", ("mhc_",)),
               ("experts", ("moe_grouped", "moe_fc", "expert")), ("feed-forward join", ("swiglu",))]

Work = Tuple[float, float, float]          # flops, bytes, special-function operations


def _keys(n_tok: int, start: int, window: int) -> int:
    """(query, key) pairs of n_tok tokens from position `start` on."""
    return sum(min(p + 1, window) for p in range(start, start + n_tok))


def hybrid_work(cfg: HybridConfig, spans: List[Tuple[int, int]], decode: bool) -> Dict[str, Work]:
    """Algorithmic work of one step over spans (start, tokens); every operand once."""
    out: Dict[str, List[float]] = {}

    def add(g: str, flops: float, byts: float, sfu: float = 0.0) -> None:
        w = out.setdefault(g, [0.0, 0.0, 0.0])
        w[0] += flops
        w[1] += byts
        w[2] += sfu

    T, W = sum(n for _, n in spans), cfg.hidden_size
    heads_rows = len(spans)                                           # logits are taken at the last token of each span
    add("projections", 2.0 * heads_rows * cfg.vocab_size * W, 2.0 * cfg.vocab_size * W)
    for l in cfg.layers:
        m, ff = l.mixer, l.mlp.ff if l.mlp else 0
        n_in = 2 * ff + (m.heads + m.kv_heads) * m.dim if m.kind == "attention" else \
            2 * ff + 2 * m.heads * (m.dim + m.vdim) + 2 * m.heads
        k_out = m.out_dim + ff
        add("projections", 2.0 * T * W * (n_in + k_out),
            2.0 * W * (n_in + k_out) + 2.0 * T * (W + n_in + k_out) + 4.0 * T * W)
        add("add + layer norm", 0, T * W * (4 + 4 + 4 + 2.0))
        if m.kind == "attention":
            pairs = sum(_keys(n, s, m.window) for s, n in spans)
            row = (m.dim + m.rot_dims) * 2.0
            kept = sum(min(s + n, m.window + n - 1) for s, n in spans) * m.kv_heads * row
            add("window_attention", 4.0 * pairs * m.heads * m.dim, kept + 4.0 * T * m.heads * m.dim,
                3.0 * pairs * m.heads)
            add("kv insert", 0, T * m.kv_heads * (2.0 * m.dim + row))
            add("feed-forward join", 0, 6.0 * T * ff)
        else:
            D, V, H = m.dim, m.vdim, m.heads
            state = H * D * (V + 1) * 4.0
            if decode:
                add("mlstm scan", 4.0 * T * H * D * V, 2 * state * len(spans) + T * H * (4.0 * D + 6.0 * V))
            else:
                chunks = sum(-(-n // 64) for _, n in spans)
                add("mlstm chunk gates", 0, T * H * (8.0 + 12.0))
                add("mlstm chunk states", 2.0 * T * H * D * V, T * H * 2.0 * (D + V) + chunks * state + 2 * state * len(spans))
                add("mlstm chunk outputs", 2.0 * T * H * D * V + T * H * 64.0 * (D + V), T * H * (4.0 * D + 6.0 * V) + chunks * state)
            add("mlstm finish", 0, T * (H * V * (4.0 + 2 + 2) + 6.0 * ff))
    add("embedding", 0, T * W * 6.0)
    return {g: tuple(v) for g, v in out.items()}


def dsv4_work(cfg, spans: List[Tuple[int, int]]) -> Dict[str, Work]:
    """The like kernels of the other family: projections, attention over the selected rows, inserts, norms, stream mixing."""
    T, H = sum(n for _, n in spans), cfg.hidden_size
    D, nh, hc = cfg.head_dim, cfg.num_attention_heads, cfg.hc_mult
    pf = pb = af = ab = nb = mb = kb = 0.0
    for li in range(cfg.num_hidden_layers):
        kind = cfg.layer_kind(li)
        I = cfg.moe_intermediate_size * cfg.n_shared_experts
        mats = [(cfg.q_lora_rank + D, H), (nh * D, cfg.q_lora_rank), (cfg.o_groups * cfg.o_lora_rank, nh // cfg.o_groups * D),
                (H, cfg.o_groups * cfg.o_lora_rank), (2 * I, H), (H, I)]
        for n, k in mats:
            pf += 2.0 * T * n * k
            pb += n * k + T * (k + 2.0 * n)
        keys = 0
        rows = 0
        for s, n in spans:
            for p in range(s, s + n):
                keys += min(p + 1, cfg.sliding_window) + (min((p + 1) // 4, cfg.index_topk) if kind == "c4a" else 0)
            rows += min(s + n, cfg.sliding_window + n) + ((s + n) // 4 if kind == "c4a" else 0)
        af += 4.0 * keys * nh * D
        ab += rows * cfg.kv_row_bytes + 4.0 * T * nh * D
        kb += T * (cfg.kv_row_bytes + 2.0 * D + 4.0 * nh * D)
        nb += T * 4.0 * (cfg.q_lora_rank + D)
        mb += 2 * T * H * 2.0 * (2 * hc + 2)
    return {"projections": (pf, pb, 0.0), "sparse attention": (af, ab, 0.0), "kv insert": (0.0, kb, 0.0), "rms norm": (0.0, nb, 0.0),
            "stream mix": (0.0, mb, 0.0)}


def table(times: Dict[str, List[float]], groups, work: Dict[str, Work], steps: int, sm_mhz: float = 1900.0) -> List[Dict]:
    """Per group: device microseconds per step, launches, roofline microseconds and their ratio."""
    pk = peaks()
    rows: List[Dict] = []
    rest, rest_n = 0.0, 0
    got: Dict[str, List[float]] = {}
    for name, durs in times.items():
        for g, pats in groups:
            if any(p in name for p in pats):
                got.setdefault(g, []).extend(durs)
                break
        else:
            rest += sum(durs)
            rest_n += len(durs)
    for g, durs in sorted(got.items(), key=lambda x: -sum(x[1])):
        us = sum(durs) / steps
        row = {"group": g, "us": round(us, 1), "launches": round(len(durs) / steps, 2)}
        if g in work:
            f, b, s = work[g]
            t = max(f / pk["bf16_tflops"] * 1e-6, b / pk["hbm_gbs"] * 1e-3)
            row.update(roofline_us=round(t, 1), fraction=round(t / us, 3), tflops=round(f / us * 1e-6, 1), gbs=round(b / us * 1e-3, 1))
            if s:
                # 16 special-function results a clock and SM
                row["sfu_us"] = round(s / (16.0 * _lib.sm_count() * sm_mhz), 1)
        rows.append(row)
    rows.append({"group": "other", "us": round(rest / steps, 1), "launches": round(rest_n / steps, 2)})
    return rows


def profile_prefill(cfg, groups, work_fn, chunk: int = CHUNK) -> List[Dict]:
    eng = make_engine(cfg, 4 * chunk + 64, 2, False)
    rid = eng.add_request(prompts(cfg, 1, 4 * chunk, 3)[0], SamplingParams(max_tokens=1))
    eng.step()                                                            # positions 0 .. chunk: a partly filled window
    times = kernel_times(eng.step, 1)                                     # one step inside kernel_times warms, one is recorded
    assert eng.requests[rid].num_computed == 3 * chunk
    return table(times, groups, work_fn([(2 * chunk, chunk)]), 1)


def profile_decode(cfg, groups, work_fn, batch: int, ctx: int, steps: int = 6) -> List[Dict]:
    eng = start_decode(cfg, batch, ctx, False)
    eng.step()
    times = kernel_times(lambda: eng.step([1] * batch), steps)
    return table(times, groups, work_fn([(ctx + 4, 1)] * batch), steps)


def run(widths: List[int], layers: int = 4, vocab: int = 32768, ctx: int = 4096, batches=(1, 8, 64), profile: bool = True) -> Dict:
    pdl = _lib.query("stk_pdl_enabled")
    res: Dict = {"peaks": peaks(), "layers": layers, "vocab": vocab, "prefill_tokens": 4 * CHUNK, "decode_context": ctx}
    for width in widths:
        for name, cfg, groups, work in (
                ("timalorn", hybrid_config(width, layers, vocab), HYBRID_GROUPS, None),
                ("deepseek-v4-style", dsv4_config(width, layers, vocab), DSV4_GROUPS, None)):
            hybrid = name == "timalorn"
            r: Dict = {"prefill_tok_s": round(time_prefill(cfg, 4 * CHUNK)), "decode": {}}
            for b in batches:
                r["decode"][str(b)] = time_decode(cfg, b, ctx)
            if profile:
                _lib.call("stk_set_pdl", 0)
                try:
                    w = (lambda s: hybrid_work(cfg, s, False)) if hybrid else (lambda s: dsv4_work(cfg, s))
                    wd = (lambda s: hybrid_work(cfg, s, True)) if hybrid else (lambda s: dsv4_work(cfg, s))
                    r["prefill_kernels"] = profile_prefill(cfg, groups, w)
                    r["decode_kernels"] = {str(b): profile_decode(cfg, groups, wd, b, ctx) for b in (batches[0], batches[-1])}
                finally:
                    _lib.call("stk_set_pdl_mask", pdl)
            res[f"{name} width {width}"] = r
    return res


def render(res: Dict) -> str:
    lines = [f"{res['layers']} layers, vocabulary {res['vocab']}, prefill of {res['prefill_tokens']} tokens in chunks of {CHUNK}, "
             f"decode at context {res['decode_context']}; peaks {res['peaks']}"]
    for k, r in res.items():
        if " width " not in k:
            continue
        lines.append(f"\n{k}: prefill {r['prefill_tok_s']} tok/s; decode "
                     + ", ".join(f"batch {b} {d['ms_per_step']} ms ({d['tok_s']} tok/s)" for b, d in r["decode"].items()))
        tabs = [("prefill chunk", r.get("prefill_kernels"))] + [(f"decode batch {b}", t) for b, t in r.get("decode_kernels", {}).items()]
        for title, rows in tabs:
            if rows:
                lines.append(f"  {title}")
                for x in rows:
                    extra = ""
                    if "roofline_us" in x:
                        extra = (f"  roofline {x['roofline_us']:8.1f} us  fraction {x['fraction']:.3f}  {x['tflops']:7.1f} TFLOP/s "
                                 f"{x['gbs']:7.1f} GB/s" + (f"  special functions {x['sfu_us']} us" if "sfu_us" in x else ""))
                    lines.append(f"    {x['us']:9.1f} us {x['launches']:6.1f}x  {x['group']:26s}{extra}")
    return "\n".join(lines)


def main() -> None:
    """One op of a layer on its own (profilers): `python -m stkernel_b200.bench.hybrid_bench --op attention|mlstm`."""
    import argparse
    from ..ops import hybrid as HB
    ap = argparse.ArgumentParser()
    ap.add_argument("--op", choices=("attention", "mlstm"), required=True)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--tokens", type=int, default=4096)
    ap.add_argument("--context", type=int, default=8192)
    ap.add_argument("--repeat", type=int, default=3)
    a = ap.parse_args()
    dev = torch.device("cuda:0")
    cfg = hybrid_config(a.width, 2, 1024)
    g = torch.Generator(device=dev).manual_seed(0)
    n, ctx = a.tokens, a.context
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    meta = HB.HybridMeta(torch.zeros(n, dtype=torch.int64, device=dev), torch.zeros(n, dtype=torch.int32, device=dev),
                         torch.arange(ctx, ctx + n, device=dev), i32([ctx] * n), i32([ctx + n - 1] * n), i32([0, n]), i32([0]),
                         i32([ctx]), 1, n, False, n)
    m = next(l.mixer for l in cfg.layers if l.mixer.kind == a.op)
    pages = (ctx + n) // 64 + 1
    e0, e1 = (torch.cuda.Event(enable_timing=True) for _ in range(2))
    if a.op == "attention":
        proj = torch.randn(n, (m.heads + m.kv_heads) * m.dim, generator=g, device=dev).to(torch.bfloat16)
        cache = torch.randn(pages, m.kv_heads, 64, m.dim + m.rot_dims, generator=g, device=dev).to(torch.bfloat16)
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1)
        freq, mag = m.rotary.frequencies()
        p = HB.AttentionParams(m.heads, m.kv_heads, m.dim, m.window, m.scale, m.softcap, torch.tensor(freq, device=dev), mag,
                               torch.zeros(m.heads, device=dev))
        out = torch.empty(n, m.out_dim, dtype=torch.bfloat16, device=dev)
        run_op = lambda: HB.window_attention(proj, 0, m.heads * m.dim, p, meta, table, cache, out)
    else:
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        proj = torch.randn(n, 2 * qk + 2 * vv, generator=g, device=dev).to(torch.bfloat16)
        gates = torch.randn(n, 2 * m.heads, generator=g, device=dev)
        p = HB.MlstmParams(m.heads, m.dim, m.vdim, m.gate_cap, torch.zeros(2 * m.heads, device=dev), torch.ones(vv, device=dev), 1e-6)
        st = tuple(torch.zeros(1, m.heads, *s, device=dev) for s in ((m.dim, m.vdim), (m.dim,), ()))
        out = torch.empty(n, vv, dtype=torch.bfloat16, device=dev)
        run_op = lambda: HB.mlstm(proj, 0, qk, 2 * qk, 2 * qk + vv, gates, p, meta, st, out, None)
    for _ in range(a.repeat):
        e0.record()
        run_op()
        e1.record()
        torch.cuda.synchronize()
    _lib.check_status()
    print(f"{a.op} width {a.width} tokens {n} context {ctx}: {e0.elapsed_time(e1) * 1e3:.1f} us")


if __name__ == "__main__":
    main()
