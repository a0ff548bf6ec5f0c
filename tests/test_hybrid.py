"""The hybrid decoder (windowed attention + mLSTM in parallel blocks) against the plain oracle: whole prompts, portions, decoding,
batches, reused pages and rows, window edges, generation through the scheduler.  Runs on the CPU reference ops and, marked
`gpu`, on the kernels in both compute types."""
import dataclasses
import json
import os

import pytest
import torch

import hybrid_util as U
import timalorn_oracle as O
from hybrid_util import attn, config, error, feed, make_engine, oracle, rec, tokens, weights
from stkernel_b200.config import timalorn_config_to_json
from stkernel_b200.runtime.engine import SamplingParams

CPU = pytest.param(("cpu", "float32"), id="cpu")
G32 = pytest.param(("cuda:0", "float32"), id="gpu-f32", marks=pytest.mark.gpu)
G16 = pytest.param(("cuda:0", "bfloat16"), id="gpu-bf16", marks=pytest.mark.gpu)
ALL = pytest.mark.parametrize("where", [CPU, G32, G16])
EXACT = pytest.mark.parametrize("where", [CPU, G32])
TOL = {"float32": 3e-4, "bfloat16": 6e-2}


def close(got, ref, where, factor=1.0):
    e = error(got, ref)
    assert e < TOL[where[1]] * factor, e


def mixed(where, **kw):
    return config(rec(), attn(), (attn(), 72, 1), (rec(2, 24, 40), None), dtype=where[1], **kw)


# ---- whole models ---------------------------------------------------------------------------------------
SHAPES = {
    "mixed": lambda d: config(rec(), attn(), (attn(), 72, 1), (rec(2, 24, 40), None), dtype=d),
    "one_kv_head": lambda d: config(attn(heads=6, kv_heads=1, dim=32, window=33, rot=16), rec(1, 8, 8), dtype=d, width=64),
    "every_head_its_own": lambda d: config(attn(heads=3, kv_heads=3, dim=40, window=64, rot=40), dtype=d, width=72),
    "odd_sizes": lambda d: config((attn(heads=2, kv_heads=1, dim=23, window=65, rot=6), 53), (rec(5, 9, 13), 31), dtype=d,
                                  width=77, vocab=101),
    "many_heads_per_group": lambda d: config(attn(heads=72, kv_heads=1, dim=16, window=40, rot=4), dtype=d, width=96),
    "twenty_heads_per_group": lambda d: config(attn(heads=40, kv_heads=2, dim=16, window=70, rot=8), dtype=d, width=96),
    "wide_head": lambda d: config(attn(heads=2, kv_heads=1, dim=136, window=50, rot=24), (rec(1, 136, 72), 40), dtype=d),
    "widest_tensor_core_head": lambda d: config(attn(heads=2, kv_heads=1, dim=256, window=70, rot=64), (rec(1, 256, 80), None),
                                                dtype=d),
    "beyond_the_tensor_core_sizes": lambda d: config(attn(heads=2, kv_heads=1, dim=264, window=50, rot=32), (rec(1, 272, 20), 8),
                                                     dtype=d),
    "window_of_one": lambda d: config(attn(window=1), rec(), dtype=d),
    "window_past_the_context": lambda d: config(attn(window=100000), dtype=d),
    "plain_rotary": lambda d: config(attn(yarn=None, rot=24), dtype=d),
    "no_rotation": lambda d: config(attn(rot=0), dtype=d),
    "no_cap": lambda d: config(attn(cap=0.0), dtype=d),
    "two_windows": lambda d: config(attn(window=9), rec(), attn(window=90), dtype=d),
    "weights_of_a_recurrence": lambda d: config(rec(), (rec(), 72, 0), (rec(), 72, 1), attn(), dtype=d),
    "aligned": lambda d: config(rec(4, 64, 128), attn(heads=8, kv_heads=2, dim=64, window=96, rot=32), dtype=d, width=256),
}


@ALL
@pytest.mark.parametrize("shape", list(SHAPES))
def test_prompt_then_decoding(where, shape):
    cfg = SHAPES[shape](where[1])
    w = weights(cfg, 1)
    toks = tokens(cfg, 140, 2)
    ref = oracle(cfg, w, toks)
    eng = make_engine(cfg, w, where[0])
    close(feed(eng, toks), ref, where)
    close(feed(eng, toks, [121, 1]), ref, where)
    close(feed(eng, toks, [63, 2, 66, 3, 2, 1]), ref, where)


def test_bf16_activations_on_the_reference_path():
    cfg = config(rec(), attn(), dtype="bfloat16")
    w, toks = weights(cfg, 1), tokens(cfg, 50, 2)
    assert error(feed(make_engine(cfg, w), toks), oracle(cfg, w, toks)) < TOL["bfloat16"]


@ALL
def test_residual_stream_after_every_layer(where):
    cfg = mixed(where)
    w, toks = weights(cfg, 4), tokens(cfg, 45, 5)
    ref = O.hidden_states(timalorn_config_to_json(cfg), w, toks)
    eng = make_engine(cfg, w, where[0])
    got = []
    eng.model.on_layer = lambda i, x: got.append(x.double().cpu())
    feed(eng, toks)
    assert len(got) == len(ref) == 4
    for a, b in zip(got, ref):
        assert a.dtype == torch.float64 and ((a - b).norm() / b.norm()).item() < {"float32": 1e-5, "bfloat16": 2e-2}[where[1]]


@ALL
@pytest.mark.parametrize("cuts", [[2], [3, 5], [7, 64, 1, 1, 30], [64], [65, 2], [128, 24, 23, 25], [1]])
def test_portions(where, cuts):
    cfg = mixed(where)
    w, toks = weights(cfg, 6), tokens(cfg, 150, 7)
    close(feed(make_engine(cfg, w, where[0]), toks, cuts), oracle(cfg, w, toks), where)


@ALL
def test_long_decoding(where):
    cfg = config(rec(2, 16, 16), attn(heads=2, kv_heads=1, dim=16, window=70, rot=8), dtype=where[1], width=48, vocab=97)
    w, toks = weights(cfg, 8), tokens(cfg, 420, 9)
    close(feed(make_engine(cfg, w, where[0]), toks, [9, 1]), oracle(cfg, w, toks), where)


# ---- batches ----------------------------------------------------------------------------------------------
@ALL
def test_unequal_requests_in_one_step(where):
    """Prompt portions and decode rows of several requests share steps; each sees only its own tokens."""
    cfg = mixed(where)
    w = weights(cfg, 10)
    eng = make_engine(cfg, w, where[0], seqs=5)
    lens = [1, 150, 37, 90, 64]
    seqs = [tokens(cfg, n, 20 + i) for i, n in enumerate(lens)]
    plans = [[1], [64, 3, 60, 1], [35, 1], [2, 1, 1, 80, 1], [64]]
    reqs = [eng.open_sequence() for _ in lens]
    got, at, turn = [[] for _ in lens], [0] * 5, [0] * 5
    while any(a < n for a, n in zip(at, lens)):
        spans = []
        for i in range(5):
            if at[i] < lens[i]:
                n = min(plans[i][min(turn[i], len(plans[i]) - 1)], lens[i] - at[i])
                spans.append((i, n))
        rows = eng.feed([(reqs[i], seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in spans]).double().cpu()
        for i, n in spans:
            got[i].append(rows[:n])
            rows, at[i], turn[i] = rows[n:], at[i] + n, turn[i] + 1
    for i in range(5):
        close(torch.cat(got[i]), oracle(cfg, w, seqs[i]), where)


@ALL
def test_pages_and_rows_are_reused(where):
    """Later requests run in pages and state rows that earlier ones filled; a diverged predecessor leaves nothing behind."""
    cfg = mixed(where)
    w = weights(cfg, 11)
    eng = make_engine(cfg, w, where[0], ctx=256, seqs=1, chunk=256)
    toks = tokens(cfg, 150, 12)
    ref = oracle(cfg, w, toks)
    group = next(iter(eng.kv.by_window.values()))
    pages = group.num_pages
    for i in range(4):
        feed(eng, tokens(cfg, 200 - 31 * i, 30 + i), [50, 1, 20])
    for cache in eng.kv.kv_cache.values():
        cache.fill_(float("nan"))                       # whatever is left in freed pages must not be read
        cache[..., cfg.layers[1].mixer.dim + cfg.layers[1].mixer.rot_dims:] = 0
    for st in eng.kv.state.values():
        for t in st:
            t.fill_(float("nan"))
    close(feed(eng, toks, [100, 7, 1]), ref, where)
    assert len(group.free) == pages and len(eng.kv.free_rows) == 1


@EXACT
def test_pages_leave_with_the_window(where):
    cfg = config(attn(window=70), rec(), attn(window=200), dtype=where[1])
    w = weights(cfg, 13)
    eng = make_engine(cfg, w, where[0])
    r = eng.open_sequence()
    for i in range(0, 600, 50):
        eng.feed([(r, tokens(cfg, 50, i), [])])
        held = {win: g.pages_in_use for win, g in eng.kv.by_window.items()}
        assert held[70] <= 4 and held[200] <= 6
    eng.close_sequence(r)
    assert all(g.pages_in_use == 0 for g in eng.kv.by_window.values())


# ---- what a position sees -----------------------------------------------------------------------------------
@ALL
@pytest.mark.parametrize("window", [5, 64, 70])
@pytest.mark.parametrize("cuts", [None, [133, 1], [60, 64, 2, 1]])
def test_window_edge(where, window, cuts):
    """A key that stands out counts at distance window - 1 and not at distance window."""
    cfg = config((attn(heads=2, kv_heads=1, dim=32, window=window, rot=16, cap=60.0), None), dtype=where[1])
    n = 150
    eng = None
    seen = {}
    for dist in (window - 1, window):
        w, toks = U.needle(cfg, n - 1 - dist, n)
        eng = eng or make_engine(cfg, w, where[0])
        got, ref = feed(eng, toks, cuts), oracle(cfg, w, toks)
        close(got, ref, where, 2.0)
        _, plain = U.needle(cfg, None, n)
        seen[dist] = error(got[-1:], feed(eng, plain, cuts)[-1:])
    assert seen[window - 1] > 0.1 and seen[window] < 1e-6


@ALL
def test_far_key_on_both_sides_of_page_borders(where):
    cfg = config((attn(heads=2, kv_heads=1, dim=32, window=400, rot=16, cap=60.0), None), dtype=where[1])
    eng = None
    for at in (0, 1, 63, 64, 127, 128, 191, 192):
        w, toks = U.needle(cfg, at, 195)
        eng = eng or make_engine(cfg, w, where[0])
        _, plain = U.needle(cfg, None, 195)
        ref = oracle(cfg, w, toks)
        for cuts in (None, [194, 1]):
            got = feed(eng, toks, cuts)
            close(got[-1:], ref[-1:], where, 2.0)
            assert error(got[-1:], feed(eng, plain, cuts)[-1:]) > 0.1


@ALL
def test_first_tokens_and_sink(where):
    """At the first positions the sink competes with one or two keys: leaving it out, or counting it twice, shows."""
    cfg = config((attn(), None), dtype=where[1])
    w = weights(cfg, 14, sink=3.0)
    toks = tokens(cfg, 6, 15)
    eng = make_engine(cfg, w, where[0])
    for cuts in (None, [1], [2]):
        close(feed(eng, toks, cuts), oracle(cfg, w, toks), where)
    for name, change in (("out", -100.0), ("twice", 0.6931)):
        other = dict(w)
        other["l0.mix.sink"] = w["l0.mix.sink"] + change
        assert error(feed(eng, toks), oracle(cfg, other, toks)) > 1.5 * TOL[where[1]], name


@ALL
def test_recurrence_over_chunk_borders_with_closed_and_open_gates(where):
    """Forget gates near zero and near one, input gates at their cap: sums of log gates reach the hundreds inside a chunk."""
    cfg = config((rec(4, 32, 40, cap=12.0), None), dtype=where[1])
    w = weights(cfg, 16)
    # queries close to the keys: the normaliser stays away from zero, where its sign would hang on rounding
    w["l0.mix.q"] = (w["l0.mix.k"] + 0.25 * w["l0.mix.q"]).to(torch.bfloat16).float()
    for f_bias in (-9.0, 0.0, 9.0):
        w["l0.mix.f.b"] = torch.full((4,), f_bias) + torch.tensor([-2.0, -1.0, 1.0, 2.0])
        w["l0.mix.i.b"] = torch.tensor([9.0, 0.0, -9.0, 3.0])
        toks = tokens(cfg, 200, 17)
        ref = oracle(cfg, w, toks)
        eng = make_engine(cfg, w, where[0])
        for cuts in (None, [63, 65, 2, 70], [190, 1]):
            close(feed(eng, toks, cuts), ref, where)


# ---- generation -----------------------------------------------------------------------------------------------
@EXACT
@pytest.mark.parametrize("sched", [dict(), dict(chunk=24), dict(seqs=2), dict(async_scheduling=True)])
def test_greedy_generation_equals_the_oracle(where, sched):
    cfg = mixed(where)
    w = weights(cfg, 18)
    prompts = [tokens(cfg, n, 40 + n) for n in (5, 1, 61, 26)]
    eng = make_engine(cfg, w, where[0], graph_cap=4, **sched)
    got = eng.generate(prompts, SamplingParams(max_tokens=9))
    for p, g in zip(prompts, got):
        assert g == O.greedy(timalorn_config_to_json(cfg), w, p, 9)
    assert all(g.pages_in_use == 0 for g in eng.kv.by_window.values())
    assert len(eng.kv.free_rows) == eng.cfg.sched.max_num_seqs


@ALL
def test_batch_and_alone_sample_the_same_text(where):
    cfg = config(rec(), attn(), dtype=where[1])
    w = weights(cfg, 19)
    prompts = [tokens(cfg, n, 60 + n) for n in (30, 4, 77)]
    par = SamplingParams(temperature=0.7, seed=5, max_tokens=12, top_k=20)
    alone = [make_engine(cfg, w, where[0], graph_cap=4).generate([p], par)[0] for p in prompts]
    together = make_engine(cfg, w, where[0], graph_cap=4, chunk=40).generate(prompts, par)
    if where[1] == "float32":
        assert together == alone
    else:                       # rounding may flip a sampled token; the first ones agree
        assert all(a[:2] == b[:2] for a, b in zip(alone, together))


@EXACT
def test_logprobs_and_abort(where):
    cfg = config(rec(), attn(), dtype=where[1])
    w = weights(cfg, 20)
    eng = make_engine(cfg, w, where[0])
    p = tokens(cfg, 12, 3)
    rid = eng.add_request(p, SamplingParams(max_tokens=3, logprobs=2))
    gone = eng.add_request(tokens(cfg, 40, 4), SamplingParams(max_tokens=30))
    eng.step()
    assert eng.abort(gone)
    while eng.has_work():
        eng.step()
    r = eng.requests[rid]
    lp = torch.log_softmax(oracle(cfg, w, p + r.output), -1)
    for i, (v, alts) in enumerate(r.logprobs):
        assert abs(v - lp[len(p) - 1 + i, r.output[i]].item()) < 1e-3 and len(alts) == 2
    assert all(g.pages_in_use == 0 for g in eng.kv.by_window.values())


# ---- product interfaces -----------------------------------------------------------------------------------------
def save_model(path, cfg, w):
    from stkernel_b200.models.loader import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}, {})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(timalorn_config_to_json(cfg), f)


@ALL
def test_trace_replay(where, tmp_path):
    """Logits of a replayed trace are the engine's; requests come and go, portions longer than a step are cut."""
    import numpy as np
    from stkernel_b200.models.loader import CheckpointSource
    from stkernel_b200.models.registry import family_of, load_model_config
    from stkernel_b200.runtime.engine import Engine
    from stkernel_b200.serve.trace_run import run
    cfg = config(rec(), attn(), dtype=where[1])
    w = weights(cfg, 21)
    save_model(tmp_path / "m", cfg, w)
    loaded = load_model_config(str(tmp_path / "m"), where[1])
    assert loaded == cfg
    src = CheckpointSource(str(tmp_path / "m"))
    assert not src.missing(loaded) and not src.unexpected(loaded)
    ec = make_engine(cfg, w, "cpu", chunk=40, seqs=2).cfg
    eng = Engine(ec, family_of(loaded).build_weights(loaded, src, where[0]), where[0], max_context=640)
    a, b = tokens(cfg, 100, 1), tokens(cfg, 30, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:90], "want": [89, 0, 41]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:20], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[90:], "want": [3]}, {"id": "b", "tokens": b[20:], "want": [9]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": b, "want": [5]}], "end": ["a"]}]
    done = []
    run(eng, [json.dumps(s) for s in steps], str(tmp_path), done.append)
    assert done == [0, 1, 2, 3] and not (tmp_path / "1.f32").exists()
    ra, rb = oracle(cfg, w, a), oracle(cfg, w, b)
    for n, ref in ((0, ra[[89, 0, 41]]), (2, torch.stack([ra[93], rb[29]])), (3, rb[[5]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").copy()).view(-1, cfg.vocab_size).double()
        close(got, ref, where)
    assert len(eng.kv.free_rows) == 2
    with pytest.raises(ValueError):
        run(eng, [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": [1], "want": [1]}], "end": []})], str(tmp_path),
            done.append)
