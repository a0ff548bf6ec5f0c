"""Replay of a token trace: given tokens go through the engine step by step, logits come out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive as lines of JSON on standard input:

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [812, 44], "want": [1]}], "end": ["chat-0"]}

An entry feeds a request its next tokens and names the places among them whose logits are to be written; `end` lists requests
that are over once the step has run, so their pages and rows become free.  OUT/<step>.f32 receives the logits (little-endian
fp32, one vocabulary-long row per place, in the order of the entries and their places); `done <step>` on standard output says
that the step is complete.

The model, its step function, caches and kernels are the engine's own (`Engine.feed`); nothing is sampled.  In bfloat16 they
are what serving uses, in float32 every operand is fp32.  Exit code 3: the architecture has no float32 form.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional, Sequence, Tuple

MAX_STEP = 8192              # tokens of one engine step; longer portions are fed in pieces
MAX_SEQUENCES = 64           # live requests


def build_engine(model: str, dtype: str, max_tokens: int):
    """The engine as the server builds it, sized for `max_tokens` live tokens."""
    from ..config import CacheConfig, ConfigError, EngineConfig, SchedulerConfig
    from ..models.loader import CheckpointSource
    from ..models.registry import family_of, load_model_config, use_native
    import torch
    try:
        cfg = load_model_config(model, dtype)
    except ConfigError as e:
        if dtype == "float32" and "float32" in str(e):
            print(f"trace_run: {e}", file=sys.stderr)
            raise SystemExit(3)
        raise
    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a CUDA device")
    family = family_of(cfg)
    use_native(cfg)
    device = torch.device("cuda:0")
    torch.cuda.set_device(device)
    context = max(64, max_tokens)
    step = min(MAX_STEP, context)
    seqs = min(MAX_SEQUENCES, context)
    # the live tokens all together, and the page every sequence leaves partly filled
    ecfg = EngineConfig(model=cfg, sched=SchedulerConfig(max_model_len=context, max_num_seqs=seqs, max_num_batched_tokens=step),
                        cache=CacheConfig(kv_pool_tokens=context + 64 * seqs)).validate()
    weights = family.build_weights(cfg, CheckpointSource(model), device)
    from ..runtime.engine import Engine
    return Engine(ecfg, weights, device, max_context=context)


def pieces(entries: Sequence[Tuple[object, List[int], List[int]]], limit: int):
    """Cut a step's entries into engine steps of at most `limit` tokens."""
    cur: List[Tuple[object, List[int], List[int]]] = []
    room = limit
    for req, tokens, want in entries:
        at = 0
        while at < len(tokens):
            if room == 0:
                yield cur
                cur, room = [], limit
            n = min(room, len(tokens) - at)
            cur.append((req, tokens[at:at + n], [w - at for w in want if at <= w < at + n]))
            at += n
            room -= n
            if at < len(tokens):
                yield cur
                cur, room = [], limit
    if cur:
        yield cur


def run(engine, lines, out_dir: str, done) -> None:
    import torch
    live: Dict[str, object] = {}
    limit = engine.cfg.sched.max_num_batched_tokens
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_sequence()
            want = [int(w) for w in e.get("want", [])]
            if any(not 0 <= w < len(e["tokens"]) for w in want):
                raise ValueError(f"step {step['step']}: a wanted place is outside the tokens of {e['id']}")
            entries.append((live[e["id"]], [int(t) for t in e["tokens"]], want))
        # pieces return logits in ascending places; the file keeps the order that was asked for
        rows: Dict[Tuple[int, int], torch.Tensor] = {}
        fed = {id(r): 0 for r, _, _ in entries}
        for part in pieces(entries, limit):
            order = [(id(r), fed[id(r)] + w) for r, _, ws in part for w in ws]
            logits = engine.feed(part)
            for r, toks, _ in part:
                fed[id(r)] += len(toks)
            if logits is not None:
                for key, row in zip(order, logits.cpu()):
                    rows[key] = row
        wanted = [rows[(id(r), w)] for r, _, ws in entries for w in ws]
        if wanted:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path, "wb") as f:
                f.write(torch.stack(wanted).to(torch.float32).contiguous().numpy().astype("<f4").tobytes())
        for rid in step.get("end", []):
            if rid in live:
                engine.close_sequence(live.pop(rid))
        done(step["step"])


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=8192, help="bound on the tokens of all open requests together (sizes the cache)")
    a = ap.parse_args(argv)
    engine = build_engine(a.model, a.dtype, a.max_tokens)
    run(engine, sys.stdin, a.out, lambda n: print(f"done {n}", flush=True))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
