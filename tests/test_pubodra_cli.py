"""Pubodra around the graph: configuration reader, registry, synthetic folders, command line, trace replay."""
import io
import json
import os

import numpy as np
import pytest
import torch

import pubodra_oracle as oracle
from design_util import ARMS, TOL, logit_error, tokens_of, write_folder
from machx_inference_engine_b200.cli import trace_run
from machx_inference_engine_b200.cli.main import main as ie
from machx_inference_engine_b200.formats.memory_plan import plan_placement
from machx_inference_engine_b200.formats.model_config import ConfigError, config_to_json, preset, read_json_config
from machx_inference_engine_b200.formats.safetensors import SafetensorsModel
from machx_inference_engine_b200.models import build_model, load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine

L = oracle.latent_layer
CFG = oracle.random_config([L(3, 12, 6, 20, 28, 40, 56, scaling=(4.0, 64, 16.0, 1.0)), L(2, 16, 4, 8, 24, 70, (5, 2, 40)), L(1, 8, 8, 12, 16, 9, None)],
                           vocab=77, width=60, eps=1e-5, loop=(0, 2, 2))


def test_config_round_trip_and_derived_sizes():
    c = read_json_config(CFG)
    assert config_to_json(c) == CFG
    assert (c.arch, c.n_layers, c.hidden, c.vocab, c.rms_eps, c.tie_embeddings) == ("pubodra", 3, 60, 77, 1e-5, True)
    assert c.layer_runs() == [(0, 0), (1, None), (0, 1), (1, None), (2, None)] and [c.layer_window(i) for i in range(3)] == [40, 70, 9]
    s = c.layer_specs
    assert (s[0].yarn, s[1].yarn, s[1].experts, s[1].experts_used, s[2].ffn, s[2].experts) == ((4.0, 64.0, 16.0, 1.0), None, 5, 2, 0, 0)
    assert [x.kv_width() for x in s] == [34, 28, 24] and c.n_experts == 5
    plain = json.loads(json.dumps(CFG))
    plain["loop"] = None
    del plain["layers"][2]["mixer"]["mask"]
    p = read_json_config(plain)
    assert p.layer_runs() == [(0, None), (1, None), (2, None)] and p.layer_window(2) == 0


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="attention"), lambda d: d["layers"][0]["mlp"].update(kind="swiglu"),
                                    lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), lambda d: d["layers"][0]["mixer"]["mask"].update(size=0),
                                    lambda d: d["layers"][1]["mixer"].pop("kv_rank"), lambda d: d.update(layers=[]), lambda d: d["loop"].update(stop=4),
                                    lambda d: d["loop"].update(times=0), lambda d: d["layers"][1]["mlp"]["router"].update(top=6), lambda d: d.pop("norm"),
                                    lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0)])
def test_malformed_configs_are_refused(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ConfigError):
        read_json_config(d)


def test_loader_checks_tensors_and_limits(tmp_path):
    w = oracle.random_weights(CFG)
    for name, cut in (("l0.mix.dkv", lambda a: a[:-1]), ("l1.mlp.e4.up", lambda a: a[:-1]), ("loop.step", lambda a: a[:1]), ("final.norm.alpha", lambda a: a.reshape(1))):
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / name, CFG, {**w, name: cut(w[name])}), "cpu")
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / (name + "-missing"), CFG, {n: a for n, a in w.items() if n != name}), "cpu")
    model, _ = load_model(write_folder(tmp_path / "good", CFG, w), "cpu", max_ctx=256)
    with pytest.raises(ValueError, match="int8"):
        model.new_kv_cache(2, "int8")
    with pytest.raises(ValueError, match="latent"):
        build_model(read_json_config(oracle.random_config([L(1, 8, 8, 8, 520, 16, None)])), "cpu", quant="bf16")


def test_synthetic_folder_inspect_and_plan(tmp_path, capsys):
    out = str(tmp_path / "m")
    assert ie(["synth", "tiny-pubodra", out]) == 0
    assert ie(["inspect", out, "--tensors"]) == 0
    text = capsys.readouterr().out
    assert "arch=pubodra" in text and "l1.mlp.e5.down" in text and "loop=1..2 x 2" in text and "experts=6 (top 2)" in text
    plan = plan_placement(out, ctx=1024)
    cfg = json.load(open(os.path.join(out, "config.json")))
    assert plan.n_gpus == 1 and plan.fits and plan.kv_bytes == 5 * (48 + 8) * 1024 * 2
    m = SafetensorsModel(out)
    W = {n: m.float32(n).copy() for n in m.names()}
    model, _ = load_model(out, "cpu", max_ctx=256, dtype="fp32")
    eng = LLMEngine(model, EngineOptions(max_ctx=256, max_seqs=1))
    toks = tokens_of(100, cfg["vocab"])
    assert logit_error(eng.feed([(eng.open_sequence(), toks, list(range(100)))]).numpy(), oracle.forward(W, cfg, toks)[0]) < TOL["fp32"]


def test_presets_build_and_weights_may_be_random():
    c = preset("tiny-pubodra")
    eng = LLMEngine(build_model(c, "cpu", quant="bf16", max_ctx=256), EngineOptions(max_ctx=256, max_seqs=1))
    lg = eng.feed([(eng.open_sequence(), tokens_of(90, c.vocab), list(range(90)))])
    assert lg.shape == (90, c.vocab) and bool(torch.isfinite(lg).all()) and float(lg.std()) > 0
    assert eng.model.weight_bytes() > 0
    for name in ("pubodra-1b", "pubodra-8b"):
        assert preset(name).layer_specs[1].kv_width() == 576


def test_repl_takes_token_ids_without_a_tokenizer(tmp_path, monkeypatch, capsys):
    w = oracle.random_weights(CFG, seed=3)
    path = write_folder(tmp_path / "m", CFG, w)
    monkeypatch.setattr("sys.stdin", io.StringIO("5 6 7 8\nhello\n/quit\n"))
    assert ie(["run", path, "--cpu", "--ctx", "128", "--gpus", "1", "--max-tokens", "5", "--temperature", "0", "--dtype", "fp32"]) == 0
    got = [int(t) for t in capsys.readouterr().out.replace(">", "").split()]
    want, ids = [], [5, 6, 7, 8]
    for _ in range(5):
        want.append(int(oracle.forward(w, CFG, ids)[0][-1].argmax()))
        ids.append(want[-1])
    assert got == want


@pytest.mark.parametrize("arm", ARMS)
def test_trace_replay(tmp_path, arm):
    """Steps on standard input -> one file of logits per step that wants some, in the order of the entries although the engine runs short queries
    first; pages of ended requests serve the next."""
    device, dtype = arm
    w = oracle.random_weights(CFG, seed=4, clear_routing=True)
    eng = trace_run.build_engine(write_folder(tmp_path / "m", CFG, w), dtype, 320, torch.device(device))
    toks = {k: tokens_of(n, 77, i) for i, (k, n) in enumerate({"x": 130, "y": 20, "z": 190}.items())}
    steps = [([("x", 100), ("y", 3)], []), ([("x", 1), ("y", 15)], []), ([("y", 2)], ["y"]), ([("x", 29)], ["x"]), ([("z", 150)], []),
             ([("z", 2)], []), ([("z", 38)], ["z"])]
    at, lines, rows = dict.fromkeys(toks, 0), [], {}
    for i, (entries, end) in enumerate(steps):
        es = []
        for k, n in entries:
            want = [0, n - 1] if n > 1 and i != 4 else []
            es.append({"id": k, "tokens": toks[k][at[k]:at[k] + n], "want": want})
            rows.setdefault(i, []).extend((k, at[k] + p) for p in want)
            at[k] += n
        lines.append(json.dumps({"step": i, "entries": es, "end": end}))
    said = []
    trace_run.replay(eng, lines, str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(len(steps))]
    full = {k: oracle.forward(w, CFG, t)[0] for k, t in toks.items()}
    for i in range(len(steps)):
        path = tmp_path / f"{i}.f32"
        assert path.exists() == bool(rows[i])
        if rows[i]:
            got = np.fromfile(path, "<f4").reshape(len(rows[i]), 77)
            assert logit_error(got, np.stack([full[k][p] for k, p in rows[i]])) < TOL[dtype]
    assert eng.bm.n_free() == eng.bm.num_blocks - 1
