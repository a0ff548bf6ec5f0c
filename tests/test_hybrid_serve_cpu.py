"""The hybrid decoder through configuration, checkpoint reader, server command and HTTP interface (CPU)."""
import dataclasses
import json

import pytest
import torch

import timalorn_oracle as O
from hybrid_util import attn, config, make_engine, rec, tokens, weights
from stkernel_b200.config import (ConfigError, EngineConfig, ParallelConfig, SchedulerConfig, SpecConfig, tiny_hybrid_config,
                                  timalorn_config_to_json)
from stkernel_b200.models.registry import FAMILIES, config_from_json, family_of, load_model_config
from test_hybrid import save_model


def test_config_round_trips():
    cfg = tiny_hybrid_config()
    assert config_from_json(json.loads(json.dumps(timalorn_config_to_json(cfg)))) == cfg
    e = EngineConfig(model=cfg, sched=SchedulerConfig(max_num_seqs=3)).validate()
    assert EngineConfig.from_dict(json.loads(e.resolved())) == e
    assert config_from_json(timalorn_config_to_json(cfg), "float32") == dataclasses.replace(cfg, dtype="float32")
    assert family_of(cfg) is FAMILIES["hybrid"] and cfg.weight_layer(2) == 1 and cfg.windows() == [40]


@pytest.mark.parametrize("path,value,word", [
    (("architecture",), "Unknown", "architecture"), (("vocab",), 0, "vocab"), (("vocab",), None, "vocab"),
    (("layers", 1, "type"), "conv", "mixer"), (("layers", 1, "mixer", "heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), 7, "vdim"), (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 26, "rot.dims"), (("layers", 1, "mixer", "mask"), {"size": 0}, "mask.size"),
    (("layers", 1, "mixer", "mask"), {"size": 4, "first": 1}, "first"), (("layers", 1, "mixer", "extra"), 1, "extra"),
    (("layers", 0, "mixer", "gate_cap"), -1.0, "gate_cap"), (("layers", 0, "mixer", "dim"), "16", "dim"),
    (("layers", 2, "weights_of"), 9, "weights_of"), (("layers", 2, "weights_of"), 0, "equal"),
    (("layers", 0, "mlp", "kind"), "moe", "feed-forward"), (("norm",), {}, "eps"), (("layers",), [], "layers")])
def test_bad_configurations_name_the_field(path, value, word):
    d = timalorn_config_to_json(tiny_hybrid_config())
    at = d
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        config_from_json(d)


def test_engine_settings_the_family_refuses():
    cfg = tiny_hybrid_config()
    for kw in (dict(parallel=ParallelConfig(tp_size=2)), dict(parallel=ParallelConfig(pp_size=2)),
               dict(spec=SpecConfig(method="dspark")), dict(parallel=ParallelConfig(eplb_record=True))):
        with pytest.raises(ConfigError):
            EngineConfig(model=cfg, **kw).validate()
    with pytest.raises(ConfigError):
        config_from_json({"vocab_size": 64}, "float32")          # the other family has no float32 form


def test_missing_and_misshapen_tensors_are_named(tmp_path):
    from stkernel_b200.models.loader import CheckpointSource
    cfg = config(rec(), attn())
    w = weights(cfg)
    del w["l1.mix.sink"]
    w["l0.mix.o"] = w["l0.mix.o"][:, :-1]
    save_model(tmp_path, cfg, w)
    src = CheckpointSource(str(tmp_path))
    assert src.missing(cfg) == ["l1.mix.sink"] and not src.unexpected(cfg)
    with pytest.raises(ValueError, match="l0.mix.o"):
        family_of(cfg).build_weights(cfg, src, "cpu")


def test_server_command_serves_a_checkpoint(tmp_path):
    """--model with weights alone (no tokenizer): greedy tokens over HTTP are the oracle's, and decode beside other requests."""
    from fastapi.testclient import TestClient
    from stkernel_b200.serve.api_server import create_app
    from stkernel_b200.serve.tp_worker import build_engine, make_parser, make_tokenizer
    cfg = config(rec(), attn(), (attn(), 72, 1), vocab=400)
    w = weights(cfg, 22)
    save_model(tmp_path, cfg, w)
    a = make_parser().parse_args(["--model", str(tmp_path), "--dtype", "float32", "--max-model-len", "256", "--max-num-seqs", "3",
                                  "--max-num-batched-tokens", "64"])
    eng, mcfg = build_engine(a, 0, 1, torch.device("cpu"))
    assert mcfg == cfg and eng.cfg.model.dtype == "float32"
    tok = make_tokenizer(a, mcfg)
    with TestClient(create_app(eng, tok, "timalorn")) as c:
        ids = tok.encode("a text to continue")
        ref = O.greedy(timalorn_config_to_json(cfg), w, ids, 6)
        body = {"prompt": ["a text to continue", "b", "a text to continue"], "max_tokens": 6, "temperature": 0, "ignore_eos": True}
        r = c.post("/v1/completions", json=body).json()
        want = tok.decode(ref)
        assert r["choices"][0]["text"] == r["choices"][2]["text"]
        # an unfinished multi-byte character at the end is held back
        assert r["choices"][0]["text"].rstrip("\ufffd") == want.rstrip("\ufffd")
        chat = {"messages": [{"role": "user", "content": "hello"}], "max_tokens": 4, "temperature": 0.5, "seed": 3, "ignore_eos": True}
        r1, r2 = (c.post("/v1/chat/completions", json=chat).json() for _ in range(2))
        assert r1["usage"]["completion_tokens"] == 4 and r1["choices"][0]["message"] == r2["choices"][0]["message"]
        assert c.post("/reset_prefix_cache").status_code == 200
        assert "vllm:gpu_cache_usage_perc" in c.get("/metrics").text


def test_server_command_with_random_weights(tmp_path):
    from stkernel_b200.serve.tp_worker import build_engine, make_parser
    cfg = tiny_hybrid_config()
    (tmp_path / "config.json").write_text(json.dumps(timalorn_config_to_json(cfg)))
    a = make_parser().parse_args(["--model-config", str(tmp_path / "config.json"), "--max-model-len", "128"])
    eng, mcfg = build_engine(a, 0, 1, torch.device("cpu"))
    assert mcfg == cfg
    assert len(eng.generate([tokens(cfg, 9)])[0]) == 16
    assert load_model_config(str(tmp_path)) == cfg


def test_sequences_fed_by_the_caller_share_the_engine_with_sampling():
    """Rows and pages of fed sequences and of scheduled requests do not mix."""
    from stkernel_b200.runtime.engine import SamplingParams
    from stkernel_b200.runtime.kv import OutOfPages
    cfg = config(rec(), attn())
    w = weights(cfg, 23)
    eng = make_engine(cfg, w, seqs=2)
    p, t = tokens(cfg, 20, 1), tokens(cfg, 30, 2)
    want = make_engine(cfg, w).generate([p], SamplingParams(max_tokens=5))[0]
    ref = O.logits(timalorn_config_to_json(cfg), w, t)
    s = eng.open_sequence()
    rid = eng.add_request(p, SamplingParams(max_tokens=5))
    for i in range(30):
        got = eng.feed([(s, t[i:i + 1], [0])])
        assert (got.double() - ref[i]).abs().max() < 1e-2
        if eng.has_work():
            eng.step()
    assert eng.requests[rid].output == want
    other = eng.open_sequence()
    with pytest.raises(OutOfPages):
        eng.open_sequence()
    with pytest.raises(ValueError):
        eng.feed([(other, [1, 2], [2])])
    assert eng.feed([(other, [], [])]) is None
    eng.close_sequence(s)
    eng.close_sequence(other)
    eng.close_sequence(other)
    assert len(eng.kv.free_rows) == 2
