"""Beputar around the graph: configuration reader, registry, synthetic folders, command line, trace replay."""
import io
import json
import os

import numpy as np
import pytest
import torch

import beputar_oracle as oracle
from design_util import ARMS, TOL, logit_error, tokens_of, write_folder
from machx_inference_engine_b200.cli import trace_run
from machx_inference_engine_b200.cli.main import main as ie
from machx_inference_engine_b200.formats.memory_plan import plan_placement
from machx_inference_engine_b200.formats.model_config import ConfigError, config_to_json, preset, read_json_config
from machx_inference_engine_b200.formats.safetensors import SafetensorsModel
from machx_inference_engine_b200.models import build_model, load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine

CFG = oracle.random_config([oracle.parallel_layer(56, oracle.attention_sizes(4, 2, 12, 40, 6, keep_first=3), 3, 8, 20, (0.5, 0.75, 0.96875)),
                            oracle.wkv_layer((5, 2, 40, 0), 2, 12),
                            oracle.attention_layer((4, 1, 24, 48), 3, 3, 16, 70, 16, base=500.0, scaling=(4.0, 64, 16.0, 1.0)),
                            oracle.attention_layer(None, 2, 1, 20, 0, 10)], vocab=77, width=60, eps=1e-5, scale=2.5)


def changed(*path, **values):
    def change(d):
        for p in path:
            d = d[p]
        d.update(values)
    return change


def test_config_round_trip_and_derived_sizes():
    c = read_json_config(CFG)
    assert config_to_json(c) == CFG
    assert (c.arch, c.n_layers, c.hidden, c.vocab, c.rms_eps, c.tie_embeddings, c.embedding_scale) == ("beputar", 4, 60, 77, 1e-5, True, 2.5)
    assert [s.mixer for s in c.layer_specs] == ["parallel", "wkv", "rotary_attention", "rotary_attention"]
    assert [c.layer_window(i) for i in range(4)] == [40, 0, 70, 0] and [c.layer_is_full_attention(i) for i in range(4)] == [True, False, True, True]
    s = c.layer_specs
    assert (s[0].keep_first, s[0].rot_dim, s[0].lin_decay, s[2].yarn, s[3].yarn) == (3, 6, (0.5, 0.75, 0.96875), (4.0, 64.0, 16.0, 1.0), None)
    assert (s[1].experts, s[1].experts_used, s[1].shared_ffn, s[2].shared_ffn, s[3].ffn, s[3].experts) == (5, 2, 0, 48, 0, 0)
    assert [x.kv_width() for x in s] == [48, 0, 96, 40] and [x.state_bytes(60) for x in s] == [4 * 480, 4 * (288 + 60), 0, 0]


@pytest.mark.parametrize("change", [changed("layers", 0, type="mamba"), changed("layers", 0, "mlp", kind="swiglu"), changed("layers", 2, "mixer", "rot", dims=18),
                                    changed("layers", 2, "mixer", "rot", dims=5), changed("layers", 2, "mixer", "mask", size=0),
                                    changed("layers", 2, "mixer", vdim=12), changed("layers", 0, "mixer", "left", kv_heads=3),
                                    changed("layers", 0, "mixer", "left", "mask", keep_first=-1), changed("layers", 0, "mixer", "right", decay=[0.5]),
                                    changed("layers", 0, "mixer", "right", dim=0), lambda d: d["layers"][1]["mixer"].pop("heads"), lambda d: d.update(layers=[]),
                                    lambda d: d["layers"][0]["mixer"].pop("right"), changed("layers", 1, "mlp", "router", top=6), lambda d: d.pop("norm"),
                                    lambda d: d.pop("embedding"), changed("layers", 2, "mixer", "rot", "scaling", factor=0)])
def test_malformed_configs_are_refused(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ConfigError):
        read_json_config(d)


def test_loader_checks_tensors(tmp_path):
    w = oracle.random_weights(CFG)
    for name in ("l0.mix.left.k", "l0.mix.right.norm", "l0.ls1", "l1.mix.mu.w", "l1.mix.u", "l1.mix.w2", "l1.mlp.e4.gate", "l2.mix.q.b", "l2.mlp.shared.up", "final.norm"):
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / name, CFG, {**w, name: w[name][:-1]}), "cpu")
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            load_model(write_folder(tmp_path / (name + "-missing"), CFG, {n: a for n, a in w.items() if n != name}), "cpu")
    model, _ = load_model(write_folder(tmp_path / "good", CFG, w), "cpu", max_ctx=256)
    with pytest.raises(ValueError, match="int8"):
        model.new_kv_cache(2, "int8")


def test_widths_past_the_kernels_are_refused_at_load():
    for layer in (oracle.attention_layer(None, 1, 1, 520, 8, 8), oracle.wkv_layer(None, 1, 264),
                  oracle.parallel_layer(None, oracle.attention_sizes(1, 1, 8, 8, 8), 1, 264, 8, (0.5,))):
        with pytest.raises(ValueError, match="kernels take"):
            build_model(read_json_config(oracle.random_config([layer])), "cpu", quant="bf16")


@pytest.mark.parametrize("rank", [1, 8, 33])
def test_inner_width_of_the_decay_comes_from_its_tensors(tmp_path, rank):
    w = oracle.random_weights(CFG, rank=rank)
    toks = tokens_of(20, 77)
    model, _ = load_model(write_folder(tmp_path / "m", CFG, w), "cpu", max_ctx=128, dtype="fp32")
    eng = LLMEngine(model, EngineOptions(max_ctx=128, max_seqs=1))
    assert logit_error(eng.feed([(eng.open_sequence(), toks, list(range(20)))]).numpy(), oracle.forward(w, CFG, toks)[0]) < TOL["fp32"]


def test_synthetic_folder_inspect_and_plan(tmp_path, capsys):
    out = str(tmp_path / "m")
    assert ie(["synth", "tiny-beputar", out]) == 0
    assert ie(["inspect", out, "--tensors"]) == 0
    text = capsys.readouterr().out
    assert "arch=beputar" in text and "l1.mlp.e5.gate" in text and "l2.mix.w1" in text and "experts=6 (top 2)" in text
    plan = plan_placement(out, ctx=1024)
    cfg = json.load(open(os.path.join(out, "config.json")))
    assert plan.n_gpus == 1 and plan.fits and plan.kv_bytes == 3 * 2 * 2 * 40 * 1024 * 2
    assert plan.state_bytes == 4 * (2 * 5 * 24 * 40 + 3 * 40 * 40 + 160)
    m = SafetensorsModel(out)
    W = {n: m.float32(n).copy() for n in m.names()}
    model, _ = load_model(out, "cpu", max_ctx=256, dtype="fp32")
    eng = LLMEngine(model, EngineOptions(max_ctx=256, max_seqs=1))
    toks = tokens_of(100, cfg["vocab"])
    assert logit_error(eng.feed([(eng.open_sequence(), toks, list(range(100)))]).numpy(), oracle.forward(W, cfg, toks)[0]) < 5 * TOL["fp32"]


def test_presets_build_and_weights_may_be_random():
    c = preset("tiny-beputar")
    eng = LLMEngine(build_model(c, "cpu", quant="bf16", max_ctx=256), EngineOptions(max_ctx=256, max_seqs=1))
    lg = eng.feed([(eng.open_sequence(), tokens_of(90, c.vocab), list(range(90)))])
    assert lg.shape == (90, c.vocab) and bool(torch.isfinite(lg).all()) and float(lg.std()) > 0
    assert eng.model.weight_bytes() > 0 and eng.model.kv_bytes_per_block() == sum(t[0].numel() * 2 for d in (eng.kv.k, eng.kv.v) for t in d.values())
    for name in ("beputar-1b", "beputar-8b"):
        assert {s.mixer for s in preset(name).layer_specs} == {"parallel", "rotary_attention", "wkv"}


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
    full = {k: oracle.forward(w, CFG, t)[0] for k, t in toks.items()}
    for i in range(len(steps)):
        path = tmp_path / f"{i}.f32"
        assert path.exists() == bool(rows[i])
        if rows[i]:
            got = np.fromfile(path, "<f4").reshape(len(rows[i]), 77)
            assert logit_error(got, np.stack([full[k][p] for k, p in rows[i]])) < TOL[dtype]
    assert eng.bm.n_free() == eng.bm.num_blocks - 1 and len(eng.sched.free_state) == trace_run.MAX_LIVE
