"""Zegelix around the graph: configuration reader, registry, synthetic folders, command line, trace replay."""
import io
import json
import os

import numpy as np
import pytest
import torch

import zegelix_oracle as oracle
from design_util import ARMS, TOL, logit_error, tokens_of, write_folder
from machx_inference_engine_b200.cli import trace_run
from machx_inference_engine_b200.cli.main import main as ie
from machx_inference_engine_b200.formats.memory_plan import plan_placement
from machx_inference_engine_b200.formats.model_config import ConfigError, config_to_json, preset, read_json_config
from machx_inference_engine_b200.formats.safetensors import SafetensorsModel
from machx_inference_engine_b200.models import build_model, load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine

CFG = oracle.random_config([oracle.rglru_layer((4, 1, 24, 0.8, 48, 1.25), 36, 3, 4),
                            oracle.attention_layer((5, 2, 40, 3.0, 0, 0.0), 4, 2, 12, 20, 40, 6, 8, base=500.0, cap=15.0),
                            oracle.rglru_layer(None, 20, 1, 2),
                            oracle.attention_layer(None, 2, 1, 20, 16, 70, 30, 20, cap=0.0),
                            oracle.attention_layer(None, 2, 2, 8, 8, 0, 0, 8)], vocab=77, width=60, eps=1e-5, scale=2.5, logit_scale=0.625, loop=(1, 3, 3))


def changed(*path, **values):
    def change(d):
        for p in path:
            d = d[p]
        d.update(values)
    return change


def test_config_round_trip_and_derived_sizes():
    c = read_json_config(CFG)
    assert config_to_json(c) == CFG
    assert (c.arch, c.n_layers, c.hidden, c.vocab, c.rms_eps, c.tie_embeddings, c.embedding_scale, c.logit_scale) == ("zegelix", 5, 60, 77, 1e-5, True, 2.5, 0.625)
    assert [s.mixer for s in c.layer_specs] == ["rglru", "pooled_attention", "rglru", "pooled_attention", "pooled_attention"]
    assert [c.layer_window(i) for i in range(5)] == [0, 40, 0, 70, 0] and [c.layer_is_full_attention(i) for i in range(5)] == [False, True, False, True, True]
    s = c.layer_specs
    assert [(x.pool, x.softcap, x.rot_dim, x.rope_theta) for x in s[1::2]] == [(6, 15.0, 8, 500.0), (30, 0.0, 20, 10000.0)] and s[4].pool == 0
    assert (s[0].experts, s[0].experts_used, s[0].act_limit, s[0].shared_ffn, s[0].shared_limit, s[1].shared_ffn, s[2].experts) == (4, 1, 0.8, 48, 1.25, 0, 0)
    assert (s[0].width, s[0].gate_blocks, s[0].conv_taps) == (36, 3, 4)
    assert [x.state_bytes(60) for x in s] == [4 * 36 * 4, 0, 4 * 20 * 2, 0, 0] and s[1].kv_width() == 2 * 32 * (1 + 1 / 6) and s[4].kv_width() == 32
    assert c.layer_runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]


def test_parts_that_may_be_missing():
    d = json.loads(json.dumps(CFG))
    d["loop"] = None
    d["layers"][1]["mixer"]["mask"] = None
    d["layers"][1]["mixer"]["softcap"] = None
    del d["layers"][0]["mlp"]["shared"]
    c = read_json_config(d)
    assert c.loop_times == 0 and c.layer_specs[1].window == c.layer_specs[1].pool == 0 and c.layer_specs[1].softcap == 0.0 and c.layer_specs[0].shared_ffn == 0


@pytest.mark.parametrize("change", [changed("layers", 0, type="mamba"), changed("layers", 0, "mlp", kind="dense"), changed("layers", 1, "mixer", "rot", dims=14),
                                    changed("layers", 1, "mixer", "rot", dims=5), changed("layers", 1, "mixer", "mask", size=0),
                                    changed("layers", 1, "mixer", "mask", pool=-1), changed("layers", 1, "mixer", vdim=13), changed("layers", 1, "mixer", kv_heads=3),
                                    changed("layers", 1, "mixer", softcap=-1.0), changed("layers", 0, "mixer", blocks=5), changed("layers", 0, "mixer", conv=0),
                                    lambda d: d["layers"][0]["mixer"].pop("blocks"), lambda d: d.update(layers=[]), changed("layers", 1, "mlp", "router", top=6),
                                    lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"), lambda d: d["layers"][0]["mlp"]["shared"].pop("limit"),
                                    lambda d: d.pop("norm"), lambda d: d.pop("embedding"), lambda d: d.pop("logit_scale"), changed("loop", stop=6),
                                    changed("loop", times=0)])
def test_malformed_configs_are_refused(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ConfigError):
        read_json_config(d)


def test_loader_checks_tensors(tmp_path):
    w = oracle.random_weights(CFG)
    for name in ("loop.in", "l0.mix.ra", "l0.mix.ri.b", "l0.mix.conv", "l0.mix.lam", "l0.mix.y", "l0.mlp.e3.gate", "l0.mlp.shared.sg", "l0.mlp.router.b", "l1.mix.sink",
                 "l1.mix.temp", "l1.mix.v.b", "l1.mix.o", "final.norm"):
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / name, CFG, {**w, name: w[name][:-1]}), "cpu")
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / (name + "-missing"), CFG, {n: a for n, a in w.items() if n != name}), "cpu")
    model, _ = load_model(write_folder(tmp_path / "good", CFG, w), "cpu", max_ctx=256)
    with pytest.raises(ValueError, match="int8"):
        model.new_kv_cache(2, "int8")


def test_widths_past_the_kernels_are_refused_at_load():
    for layer in (oracle.attention_layer(None, 1, 1, 520, 8, 8, 2, 8), oracle.attention_layer(None, 1, 1, 8, 520, 8, 2, 8), oracle.rglru_layer(None, 1600, 1, 4),
                  oracle.rglru_layer(None, 16, 2, 9)):
        with pytest.raises(ValueError, match="kernels take"):
            build_model(read_json_config(oracle.random_config([layer])), "cpu", quant="bf16")


def test_synthetic_folder_inspect_and_plan(tmp_path, capsys):
    out = str(tmp_path / "m")
    assert ie(["synth", "tiny-zegelix", out]) == 0
    assert ie(["inspect", out, "--tensors"]) == 0
    text = capsys.readouterr().out
    assert "arch=zegelix" in text and "l1.mlp.e5.gate" in text and "l0.mix.lam" in text and "experts=6 (top 2)" in text and "loop=1..2 x 2" in text
    plan = plan_placement(out, ctx=1024)
    cfg = json.load(open(os.path.join(out, "config.json")))
    assert plan.n_gpus == 1 and plan.fits and plan.kv_bytes == int(2 * 2 * 96 * 1.2 * 1024 * 2)
    assert plan.state_bytes == 3 * 4 * 192 * 4
    m = SafetensorsModel(out)
    W = {n: m.float32(n).copy() for n in m.names()}
    model, _ = load_model(out, "cpu", max_ctx=256, dtype="fp32")
    eng = LLMEngine(model, EngineOptions(max_ctx=256, max_seqs=1))
    toks = tokens_of(100, cfg["vocab"])
    assert logit_error(eng.feed([(eng.open_sequence(), toks, list(range(100)))]).numpy(), oracle.forward(cfg, W, toks)) < 5 * TOL["fp32"]


def test_presets_build_and_weights_may_be_random():
    c = preset("tiny-zegelix")
    eng = LLMEngine(build_model(c, "cpu", quant="bf16", max_ctx=256), EngineOptions(max_ctx=256, max_seqs=1))
    lg = eng.feed([(eng.open_sequence(), tokens_of(90, c.vocab), list(range(90)))])
    assert lg.shape == (90, c.vocab) and bool(torch.isfinite(lg).all()) and float(lg.std()) > 0
    pages = [t for d in (eng.kv.k, eng.kv.v) for t in d.values()] + [t for p in eng.kv.pools.values() for t in (p.k, p.v)]
    assert eng.model.weight_bytes() > 0 and eng.model.kv_bytes_per_block() == sum(t[0].numel() * 2 for t in pages)
    for name in ("zegelix-1b", "zegelix-8b"):
        assert {s.mixer for s in preset(name).layer_specs} == {"pooled_attention", "rglru"}


def test_repl_takes_token_ids_without_a_tokenizer(tmp_path, monkeypatch, capsys):
    w = oracle.random_weights(CFG, seed=3)
    path = write_folder(tmp_path / "m", CFG, w)
    monkeypatch.setattr("sys.stdin", io.StringIO("5 6 7 8\nhello\n/quit\n"))
    assert ie(["run", path, "--cpu", "--ctx", "128", "--gpus", "1", "--max-tokens", "5", "--temperature", "0", "--dtype", "fp32"]) == 0
    got = [int(t) for t in capsys.readouterr().out.replace(">", "").split()]
    assert got == oracle.greedy(CFG, w, [5, 6, 7, 8], 5)


@pytest.mark.parametrize("arm", ARMS)
def test_trace_replay(tmp_path, arm):
    """Steps on standard input -> one file of logits per step that wants some; pages and slots of ended requests serve the next."""
    device, dtype = arm
    w = oracle.random_weights(CFG, seed=4)
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
    full = {k: oracle.forward(CFG, w, t) for k, t in toks.items()}
    for i in range(len(steps)):
        path = tmp_path / f"{i}.f32"
        assert path.exists() == bool(rows[i])
        if rows[i]:
            got = np.fromfile(path, "<f4").reshape(len(rows[i]), 77)
            assert logit_error(got, np.stack([full[k][p] for k, p in rows[i]])) < TOL[dtype]
    assert eng.bm.n_free() == eng.bm.num_blocks - 1 and len(eng.sched.free_state) == trace_run.MAX_LIVE
