"""The latent-attention decoder (Domilix) against the plain oracle: whole prompts, portions, decoding, batches, reused pages and rows,
shared latents, far keys, generation through the scheduler.  Runs on the CPU reference ops and, marked `gpu`, on the kernels in
both compute types."""
import dataclasses
import json
import os

import pytest
import torch

import domilix_oracle as O
import latent_util as U
from latent_util import config, dense, error, feed, lat, make_engine, moe, oracle, tokens, weights
from stkernel_b200.config import CacheConfig, EngineConfig, SchedulerConfig, domilix_config_to_json
from stkernel_b200.runtime.engine import SamplingParams

CPU = pytest.param(("cpu", "float32"), id="cpu")
G32 = pytest.param(("cuda:0", "float32"), id="gpu-f32", marks=pytest.mark.gpu)
G16 = pytest.param(("cuda:0", "bfloat16"), id="gpu-bf16", marks=pytest.mark.gpu)
ALL = pytest.mark.parametrize("where", [CPU, G32, G16])
EXACT = pytest.mark.parametrize("where", [CPU, G32])
TOL = {k: v[0] for k, v in U.LIMITS.items()}


def close(got, ref, where, factor=1.0):
    U.close(got, ref, where[1], factor)


def mixed(where, **kw):
    """Own and shared latents, both feed-forwards and none."""
    return config(lat(), (lat(heads=2, vdim=16), moe()), (lat(kv_from=1, heads=4, dim=12), moe(5, 3, 24)),
                  (lat(kv_from=0, vdim=40, q_rank=20), None), dtype=where[1], **kw)


def plain(where, **kw):
    """No close routing decisions: every expert is chosen, the router only weighs."""
    return config(lat(), (lat(heads=2, vdim=16), moe(3, 3, 40)), (lat(kv_from=1, heads=4, dim=12), dense()),
                  (lat(kv_from=0, q_rank=20), None), dtype=where[1], **kw)


def checked(cfg, w, toks, where):
    """How much of a sequence a compute type with rounding must reproduce."""
    return len(toks) if where[1] == "float32" else U.clear_routing(cfg, w, toks, 0.12)


SHAPES = {
    "mixed": lambda d: mixed((None, d)),
    "dense_only": lambda d: config(lat(), lat(kv_from=0), dtype=d),
    "one_head": lambda d: config((lat(heads=1, dim=16, rot=16, vdim=16, q_rank=16, kv_rank=16), moe(4, 1, 16)), dtype=d, width=48),
    "odd_sizes": lambda d: config((lat(heads=3, dim=23, rot=6, vdim=21, q_rank=37, kv_rank=35), dense(53)),
                                  (lat(heads=5, dim=7, rot=6, vdim=9, q_rank=11, kv_rank=35, kv_from=0), moe(7, 4, 19)), dtype=d,
                                  width=77, vocab=101),
    "all_experts_chosen": lambda d: config((lat(), moe(3, 3, 24)), dtype=d),
    "one_expert": lambda d: config((lat(), moe(1, 1, 24)), dtype=d),
    "many_heads": lambda d: config((lat(heads=40, dim=8, rot=4, vdim=8), dense()), dtype=d),
    "no_rotation": lambda d: config(lat(rot=0), (lat(rot=0, kv_from=0), moe()), dtype=d),
    "aligned": lambda d: config((lat(heads=8, dim=64, rot=32, vdim=64, q_rank=128, kv_rank=128), dense(256)),
                                (lat(heads=4, dim=64, rot=32, vdim=64, q_rank=96, kv_rank=128, kv_from=0), moe(16, 4, 64)), dtype=d,
                                width=256),
    "large_latent": lambda d: config((lat(heads=2, dim=128, rot=64, vdim=128, q_rank=160, kv_rank=512), moe(4, 2, 128)), dtype=d,
                                     width=128),
    "wide_values": lambda d: config((lat(heads=2, dim=40, rot=72, vdim=136, q_rank=40, kv_rank=72), dense()), dtype=d),
}


@ALL
@pytest.mark.parametrize("shape", list(SHAPES))
def test_prompt_then_decoding(where, shape):
    cfg = SHAPES[shape](where[1])
    w = weights(cfg, 1)
    toks = tokens(cfg, 180, 2)
    n = checked(cfg, w, toks, where)
    toks = toks[:max(n, 1)]
    ref = oracle(cfg, w, toks)[:n]
    eng = make_engine(cfg, w, where[0])
    for cuts in (None, [161, 1], [63, 2, 66, 3, 2, 1]):
        if n:
            close(feed(eng, toks, cuts)[:n], ref, where)


def test_bf16_activations_on_the_reference_path():
    cfg = config(lat(), lat(kv_from=0), dtype="bfloat16")
    w, toks = weights(cfg, 1), tokens(cfg, 50, 2)
    U.close(feed(make_engine(cfg, w), toks), oracle(cfg, w, toks), "bfloat16")


@ALL
def test_residual_stream_after_every_layer(where):
    cfg = config(lat(), (lat(kv_from=0, heads=2), moe(3, 3, 40)), (lat(), None), dtype=where[1])
    w, toks = weights(cfg, 4), tokens(cfg, 45, 5)
    ref = O.hidden_states(domilix_config_to_json(cfg), w, toks)
    eng = make_engine(cfg, w, where[0])
    got = []
    eng.model.on_layer = lambda i, x: got.append(x.double().cpu())
    feed(eng, toks)
    assert len(got) == len(ref) == 3
    for a, b in zip(got, ref):
        assert ((a - b).norm() / b.norm()).item() < {"float32": 1e-5, "bfloat16": 2e-2}[where[1]]


@ALL
@pytest.mark.parametrize("cuts", [[2], [3, 5], [7, 64, 1, 1, 30], [64], [65, 2], [128, 24, 23, 25], [1]])
def test_portions(where, cuts):
    cfg = plain(where)
    w, toks = weights(cfg, 6), tokens(cfg, 200, 7)
    close(feed(make_engine(cfg, w, where[0]), toks, cuts), oracle(cfg, w, toks), where)


@ALL
def test_long_decoding(where):
    cfg = config((lat(heads=2, dim=16, rot=8, vdim=16, q_rank=24, kv_rank=24), moe(2, 2, 24)), dtype=where[1], width=48, vocab=97)
    w, toks = weights(cfg, 8), tokens(cfg, 420, 9)
    close(feed(make_engine(cfg, w, where[0]), toks, [9, 1]), oracle(cfg, w, toks), where)


# ---- batches ----------------------------------------------------------------------------------------------
@ALL
def test_unequal_requests_in_one_step(where):
    """Prompt portions (long and short) and decode rows of several requests share steps; each sees only its own tokens."""
    cfg = plain(where)
    w = weights(cfg, 10)
    eng = make_engine(cfg, w, where[0], seqs=5)
    lens = [1, 250, 37, 190, 64]
    seqs = [tokens(cfg, n, 20 + i) for i, n in enumerate(lens)]
    plans = [[1], [64, 3, 130, 1], [35, 1], [2, 1, 1, 180, 1], [64]]
    reqs = [eng.open_sequence() for _ in lens]
    got, at, turn = [[] for _ in lens], [0] * 5, [0] * 5
    while any(a < n for a, n in zip(at, lens)):
        spans = []
        for i in range(5):
            if at[i] < lens[i]:
                spans.append((i, min(plans[i][min(turn[i], len(plans[i]) - 1)], lens[i] - at[i])))
        rows = eng.feed([(reqs[i], seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in spans]).double().cpu()
        for i, n in spans:
            got[i].append(rows[:n])
            rows, at[i], turn[i] = rows[n:], at[i] + n, turn[i] + 1
    for i in range(5):
        close(torch.cat(got[i]), oracle(cfg, w, seqs[i]), where)


@ALL
def test_pages_and_rows_are_reused(where):
    """Later requests run in pages that earlier ones filled; a diverged predecessor leaves nothing behind."""
    cfg = plain(where)
    w = weights(cfg, 11)
    eng = make_engine(cfg, w, where[0], ctx=256, seqs=1, chunk=256)
    toks = tokens(cfg, 190, 12)
    ref = oracle(cfg, w, toks)
    pages = eng.kv.full.num_pages
    assert sorted(eng.kv.kv_cache) == [0, 1]                # the layers that cache latents of their own
    for i in range(4):
        feed(eng, tokens(cfg, 200 - 31 * i, 30 + i), [50, 1, 20])
    for cuts in ([100, 7, 1], [80, 110], [1]):
        for cache in eng.kv.kv_cache.values():
            cache.fill_(float("nan"))                       # whatever is left in freed pages must not be read
        close(feed(eng, toks, cuts), ref, where)
    assert len(eng.kv.full.free) == pages and len(eng.kv.free_rows) == 1


@ALL
def test_shared_latents_come_from_the_named_layer(where):
    cfg = config(lat(), lat(), lat(kv_from=0), lat(kv_from=1), dtype=where[1])
    w, toks = weights(cfg, 13), tokens(cfg, 90, 14)
    for cuts in (None, [70, 3, 1]):
        close(feed(make_engine(cfg, w, where[0]), toks, cuts), oracle(cfg, w, toks), where)
    swapped = config(lat(), lat(), lat(kv_from=1), lat(kv_from=0), dtype=where[1])
    assert error(oracle(swapped, w, toks), oracle(cfg, w, toks)) > 3 * TOL[where[1]]


# ---- what a position sees -----------------------------------------------------------------------------------
@ALL
def test_far_key_on_both_sides_of_page_borders(where):
    """A key that stands out is found at page and block borders, in a prompt, a short portion and in decoding."""
    cfg = config((lat(heads=2, dim=32, rot=16, vdim=32), None), dtype=where[1])
    eng = None
    _, without = U.needle(cfg, None, 300)
    for at in (0, 1, 63, 64, 127, 128, 191, 255, 256, 298):
        w, toks = U.needle(cfg, at, 300)
        eng = eng or make_engine(cfg, w, where[0])
        ref = oracle(cfg, w, toks)[-1:]
        for cuts in (None, [299, 1], [297, 3], [200, 100]):
            got = feed(eng, toks, cuts)[-1:]
            close(got, ref, where)
            assert error(got, feed(eng, without, cuts)[-1:]) > 0.3


@ALL
def test_first_tokens(where):
    cfg = plain(where)
    w, toks = weights(cfg, 15), tokens(cfg, 6, 16)
    eng = make_engine(cfg, w, where[0])
    for cuts in (None, [1], [2]):
        close(feed(eng, toks, cuts), oracle(cfg, w, toks), where)


@ALL
@pytest.mark.parametrize("part", ["scale", "negative_scale", "rot.base", "norm.eps", "embedding.scale"])
def test_every_constant_counts(where, part):
    """The logits follow each constant of the configuration."""
    from stkernel_b200.models.registry import config_from_json
    cfg = plain(where)
    other = json.loads(json.dumps(domilix_config_to_json(cfg)))
    if part == "scale":
        other["layers"][0]["mixer"]["scale"] *= 0.5
    elif part == "negative_scale":
        other["layers"][0]["mixer"]["scale"] *= -1
    elif part == "rot.base":
        for l in other["layers"]:
            l["mixer"]["rot"]["base"] = 20.0
    elif part == "norm.eps":
        other["norm"]["eps"] = 0.8
    else:
        other["embedding"]["scale"] = 2.5
    cfg2 = config_from_json(other, where[1])
    w, toks = weights(cfg, 17, sharp=1.2), tokens(cfg, 80, 18)
    ref = O.logits(other, w, toks)
    close(feed(make_engine(cfg2, w, where[0]), toks), ref, where)
    assert error(oracle(cfg, w, toks), ref) > 2 * TOL[where[1]]


# ---- generation -----------------------------------------------------------------------------------------------
@EXACT
@pytest.mark.parametrize("sched", [dict(), dict(chunk=24), dict(seqs=2), dict(async_scheduling=True)])
def test_greedy_generation_equals_the_oracle(where, sched):
    cfg = mixed(where)
    w = weights(cfg, 19)
    prompts = [tokens(cfg, n, 40 + n) for n in (5, 1, 81, 26)]
    eng = make_engine(cfg, w, where[0], graph_cap=4, **sched)
    got = eng.generate(prompts, SamplingParams(max_tokens=9))
    for p, g in zip(prompts, got):
        assert g == O.greedy(domilix_config_to_json(cfg), w, p, 9)
    assert eng.kv.full.pages_in_use == 0 and not eng.kv.reserved
    assert len(eng.kv.free_rows) == eng.cfg.sched.max_num_seqs


@ALL
def test_batch_and_alone_sample_the_same_text(where):
    cfg = plain(where)
    w = weights(cfg, 20)
    prompts = [tokens(cfg, n, 60 + n) for n in (30, 4, 77)]
    par = SamplingParams(temperature=0.7, seed=5, max_tokens=12, top_k=20)
    alone = [make_engine(cfg, w, where[0], graph_cap=4).generate([p], par)[0] for p in prompts]
    together = make_engine(cfg, w, where[0], graph_cap=4, chunk=40).generate(prompts, par)
    if where[1] == "float32":
        assert together == alone
    else:                       # rounding may flip a sampled token; the first ones agree
        assert all(a[:2] == b[:2] for a, b in zip(alone, together))


@pytest.mark.gpu
def test_captured_decode_steps_follow_a_growing_context():
    """Graphs of several batch sizes and context buckets, replayed in turn, give what eager steps give."""
    cfg = plain(("cuda:0", "bfloat16"))
    w = weights(cfg, 21)
    prompts = [tokens(cfg, n, 80 + n) for n in (1000, 1015, 30, 2)]
    outs = []
    for cap in (0, 4):
        eng = make_engine(cfg, w, "cuda:0", ctx=1200, chunk=1200, graph_cap=cap)
        outs.append([eng.generate(prompts[:k], SamplingParams(max_tokens=20)) for k in (1, 4, 2, 1)])
    flat = [[t for run in o for text in run for t in text] for o in outs]
    same = sum(a == b for a, b in zip(*flat)) / len(flat[0])
    assert len(flat[0]) == len(flat[1]) and same > 0.7
    assert outs[1][0][0] == outs[1][3][0]                   # the same graph before and after the larger ones were captured


@EXACT
def test_requests_wait_for_pages(where):
    """A pool smaller than all contexts together: requests are admitted as others end, and give the same text."""
    from stkernel_b200.models.hybrid import build_hybrid_weights
    from stkernel_b200.models.sources import DictSource
    from stkernel_b200.runtime.engine import Engine
    cfg = plain(where)
    w = weights(cfg, 22)
    prompts = [tokens(cfg, n, 90 + n) for n in (120, 60, 100, 10)]
    want = make_engine(cfg, w, where[0]).generate(prompts, SamplingParams(max_tokens=6))
    ec = EngineConfig(model=cfg, sched=SchedulerConfig(max_model_len=192, max_num_seqs=4, max_num_batched_tokens=64, graph_cap=0),
                      cache=CacheConfig(kv_pool_tokens=256)).validate()
    eng = Engine(ec, build_hybrid_weights(cfg, DictSource(w), where[0]), where[0], max_context=192)
    assert eng.kv.full.num_pages <= 5 and not eng.kv.fits(1000)
    ids = [eng.add_request(p, SamplingParams(max_tokens=6)) for p in prompts]
    most = 0
    while eng.has_work():
        eng.step()
        most = max(most, eng.sched.num_running)
    assert [eng.requests[i].output for i in ids] == want and 1 < most < 4
    assert eng.kv.full.pages_in_use == 0 and eng.kv.usage() == 0


# ---- product interfaces -----------------------------------------------------------------------------------------
def save_model(path, cfg, w):
    from stkernel_b200.models.loader import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}, {})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(domilix_config_to_json(cfg), f)


@ALL
def test_trace_replay(where, tmp_path):
    """Logits of a replayed trace are the engine's; requests come and go, portions longer than a step are cut."""
    import numpy as np
    from stkernel_b200.models.loader import CheckpointSource
    from stkernel_b200.models.registry import family_of, load_model_config
    from stkernel_b200.runtime.engine import Engine
    from stkernel_b200.serve.trace_run import run
    cfg = plain(where)
    w = weights(cfg, 23)
    save_model(tmp_path / "m", cfg, w)
    loaded = load_model_config(str(tmp_path / "m"), where[1])
    assert loaded == cfg
    src = CheckpointSource(str(tmp_path / "m"))
    assert not src.missing(loaded) and not src.unexpected(loaded)
    ec = make_engine(cfg, w, "cpu", chunk=90, seqs=2).cfg
    eng = Engine(ec, family_of(loaded).build_weights(loaded, src, where[0]), where[0], max_context=640)
    a, b = tokens(cfg, 110, 1), tokens(cfg, 30, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:100], "want": [99, 0, 41]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:20], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[100:], "want": [3]}, {"id": "b", "tokens": b[20:], "want": [9]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": b, "want": [5]}], "end": ["a"]}]
    done = []
    run(eng, [json.dumps(s) for s in steps], str(tmp_path), done.append)
    assert done == [0, 1, 2, 3] and not (tmp_path / "1.f32").exists()
    ra, rb = oracle(cfg, w, a), oracle(cfg, w, b)
    for n, ref in ((0, ra[[99, 0, 41]]), (2, torch.stack([ra[103], rb[29]])), (3, rb[[5]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").copy()).view(-1, cfg.vocab_size).double()
        assert error(got, ref) < TOL[where[1]]
    assert len(eng.kv.free_rows) == 2


def test_greedy_text_over_http(tmp_path):
    """The server command on a checkpoint of weights alone: tokens are the oracle's."""
    from fastapi.testclient import TestClient
    from stkernel_b200.serve.api_server import create_app
    from stkernel_b200.serve.tp_worker import build_engine, make_parser, make_tokenizer
    cfg = mixed((None, "float32"), vocab=400)
    w = weights(cfg, 24)
    save_model(tmp_path, cfg, w)
    a = make_parser().parse_args(["--model", str(tmp_path), "--dtype", "float32", "--max-model-len", "256", "--max-num-seqs", "3",
                                  "--max-num-batched-tokens", "64"])
    eng, mcfg = build_engine(a, 0, 1, torch.device("cpu"))
    assert mcfg == cfg
    tok = make_tokenizer(a, mcfg)
    with TestClient(create_app(eng, tok, "domilix")) as c:
        ids = tok.encode("a text to continue")
        want = tok.decode(O.greedy(domilix_config_to_json(cfg), w, ids, 6))
        body = {"prompt": ["a text to continue", "b"], "max_tokens": 6, "temperature": 0, "ignore_eos": True}
        r = c.post("/v1/completions", json=body).json()
        assert r["choices"][0]["text"].rstrip("�") == want.rstrip("�")
        assert "vllm:gpu_cache_usage_perc" in c.get("/metrics").text


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "attention", "mixer"), (("layers", 1, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 1, "mixer", "kv_from"), 5, "kv_from"), (("layers", 1, "mixer", "kv_rank"), 40, "kv_from"),
    (("layers", 0, "mixer", "rot", "dims"), 6, "rot.dims"), (("layers", 0, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 0, "mixer", "extra"), 1, "extra"), (("layers", 1, "mlp", "kind"), "conv", "feed-forward"),
    (("layers", 1, "mlp", "router", "top"), 7, "top"), (("layers", 1, "mlp", "expert"), {}, "ff"),
    (("layers", 0, "mixer", "scale"), "x", "scale"), (("vocab",), None, "vocab")])
def test_bad_configurations_name_the_field(path, value, word):
    from stkernel_b200.config import ConfigError, tiny_latent_config
    from stkernel_b200.models.registry import config_from_json
    d = json.loads(json.dumps(domilix_config_to_json(tiny_latent_config())))
    assert config_from_json(d) == tiny_latent_config()
    at = d
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        config_from_json(d)


def test_configuration_round_trips_and_sources_follow_the_mechanisms():
    from stkernel_b200.config import tiny_hybrid_config, tiny_latent_config
    from stkernel_b200.csrc.build import sources
    from stkernel_b200.models.registry import config_from_json, family_of
    cfg = tiny_latent_config()
    e = EngineConfig(model=cfg, sched=SchedulerConfig(max_num_seqs=3)).validate()
    assert EngineConfig.from_dict(json.loads(e.resolved())) == e
    assert config_from_json(domilix_config_to_json(cfg), "float32") == dataclasses.replace(cfg, dtype="float32")
    name, files = family_of(cfg).native_sources(cfg)
    other, theirs = family_of(tiny_hybrid_config()).native_sources(tiny_hybrid_config())
    assert name != other and "latent_prompt_tc.cu" in files and "mlstm.cu" not in files and "latent_attention.cu" not in theirs
    assert all(f.exists() for f in sources(files) + sources(theirs))
