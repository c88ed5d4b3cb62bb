"""Tikarax around the graph: configuration reader, registry, synthetic folders, command line, trace replay, component build list."""
import io
import json
import os

import numpy as np
import pytest
import torch

import tikarax_oracle as oracle
from design_util import ARMS, TOL, logit_error, tokens_of, write_folder
from machx_inference_engine_b200 import _build
from machx_inference_engine_b200.cli import trace_run
from machx_inference_engine_b200.cli.inspect_gguf import inspect
from machx_inference_engine_b200.cli.main import main as ie
from machx_inference_engine_b200.formats.memory_plan import plan_placement
from machx_inference_engine_b200.formats.model_config import ConfigError, config_to_json, preset, read_json_config
from machx_inference_engine_b200.formats.safetensors import SafetensorsModel
from machx_inference_engine_b200.models import build_model, load_model

A, M = oracle.attention_layer, oracle.mingru_layer
CFG = oracle.random_config([A(3, 1, 12, 20, 56, coef=0.7, every=9), M(44, None), A(4, 4, 16, 8, 24)], vocab=77, width=60, groups=4, eps=1e-5)


def test_config_round_trip_and_derived_sizes():
    c = read_json_config(CFG)
    assert config_to_json(c) == CFG
    assert (c.arch, c.n_layers, c.hidden, c.vocab, c.norm_groups, c.rms_eps) == ("tikarax", 3, 60, 77, 4, 1e-5)
    assert [c.layer_is_full_attention(i) for i in range(3)] == [True, False, True]
    assert (c.layer_specs[0].q_temp_coef, c.layer_specs[0].q_temp_every, c.layer_specs[1].ffn, c.layer_specs[1].width) == (0.7, 9.0, 0, 44)


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="lstm"), lambda d: d["layers"][0]["mlp"].update(kind="moe"),
                                    lambda d: d["layers"][0]["mixer"].update(kv_heads=2), lambda d: d["norm"].update(groups=7),
                                    lambda d: d["layers"][1]["mixer"].pop("width"), lambda d: d.update(architecture="Other"), lambda d: d.update(layers=[]),
                                    lambda d: d["layers"][2]["mixer"]["q_temp"].update(every=0)])
def test_malformed_configs_are_refused(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ConfigError):
        read_json_config(d)


def test_loader_checks_tensors_and_dtype(tmp_path):
    w = oracle.random_weights(CFG)
    bad = dict(w)
    bad["l0.mix.g"] = bad["l0.mix.g"][:-1]
    with pytest.raises(ValueError, match="l0.mix.g"):
        load_model(write_folder(tmp_path / "shape", CFG, bad), "cpu")
    del bad["l0.mix.g"]
    with pytest.raises(ValueError, match="l0.mix.g"):
        load_model(write_folder(tmp_path / "missing", CFG, bad), "cpu")
    with pytest.raises(ValueError, match="fp32"):
        build_model(preset("tiny-llama"), "cpu", dtype="fp32")
    model, _ = load_model(write_folder(tmp_path / "good", CFG, w), "cpu", max_ctx=256)
    with pytest.raises(ValueError, match="int8"):
        model.new_kv_cache(2, "int8")
    kv = model.new_kv_cache(3)
    assert sum(t.numel() * 2 for d in (kv.k, kv.v) for t in d.values()) == 3 * model.kv_bytes_per_block()


def test_synthetic_folder_inspect_and_plan(tmp_path, capsys):
    out = str(tmp_path / "m")
    assert ie(["synth", "tiny-tikarax", out]) == 0
    assert ie(["inspect", out, "--tensors"]) == 0
    text = capsys.readouterr().out
    assert "arch=tikarax" in text and "l0.mix.z.b" in text
    plan = plan_placement(out, ctx=1024)
    assert plan.n_gpus == 1 and plan.fits and plan.weights_bytes > 0 and plan.state_bytes > 0
    m = SafetensorsModel(out)
    W = {n: m.float32(n).copy() for n in m.names()}
    cfg = json.load(open(os.path.join(out, "config.json")))
    model, _ = load_model(out, "cpu", max_ctx=256, dtype="fp32")
    from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine
    eng = LLMEngine(model, EngineOptions(max_ctx=256, max_seqs=1))
    toks = tokens_of(60, cfg["vocab"])
    seq = eng.open_sequence()
    assert logit_error(eng.feed([(seq, toks, list(range(60)))]).numpy(), oracle.forward(W, cfg, toks)[0]) < TOL["fp32"]


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
    """Steps on standard input -> one file of logits per step that wants some; pages of ended requests serve the next."""
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
    assert eng.bm.n_free() == eng.bm.num_blocks - 1


def test_pool_is_made_for_the_tokens_of_live_requests(tmp_path):
    """Four live requests whose counts, rounded up to 64, add up to the limit always fit; the pool is not made for more than that."""
    path = write_folder(tmp_path / "m", CFG, oracle.random_weights(CFG))
    for limit, lens in ((256, (64, 64, 64, 64)), (448, (64, 64, 64, 256)), (1152, (1, 65, 129, 700))):
        eng = trace_run.build_engine(path, "bf16", limit, torch.device("cpu"))
        seqs = [(eng.open_sequence(), [1] * n) for n in lens]
        eng.sched.admit([(s, len(t)) for s, t in seqs])
        assert eng.bm.num_blocks * 128 <= limit + 4 * 64 + 256


def test_quantised_weights_need_widths_that_are_not_padded():
    from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine
    aligned = read_json_config(oracle.random_config([A(4, 2, 32, 64, 128), M(96, 64)], vocab=96, width=64))
    toks, out = tokens_of(50, 96), {}
    for quant in ("bf16", "q8_0"):
        eng = LLMEngine(build_model(aligned, "cpu", quant=quant, max_ctx=128), EngineOptions(max_ctx=128, max_seqs=1))
        out[quant] = eng.feed([(eng.open_sequence(), toks, list(range(50)))]).numpy()
    assert 1e-4 < logit_error(out["q8_0"], out["bf16"]) < 0.1
    with pytest.raises(ValueError, match="padded"):
        build_model(read_json_config(oracle.random_config([A(4, 2, 36, 64, 128)], vocab=96, width=64)), "cpu", quant="q8_0")


@pytest.mark.gpu
@pytest.mark.parametrize("quant", ["bf16", "q8_0"])
def test_quantised_weights_on_the_gpu(quant):
    from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine
    aligned = read_json_config(oracle.random_config([A(4, 2, 32, 64, 128), M(96, 64)], vocab=96, width=64))
    toks, out = tokens_of(90, 96), {}
    for dev in ("cpu", "cuda:0"):
        eng = LLMEngine(build_model(aligned, torch.device(dev), quant=quant, max_ctx=128, gen_device="cpu"), EngineOptions(max_ctx=128, max_seqs=1))
        seq = eng.open_sequence()
        out[dev] = torch.cat([eng.feed([(seq, toks[:80], list(range(80)))])] + [eng.feed([(seq, [t], [0])]) for t in toks[80:]]).cpu().numpy()
    assert logit_error(out["cuda:0"], out["cpu"]) < TOL["bf16"]


def test_component_names_existing_sources():
    have = {p.stem for p in (_build.CSRC / "cuda").glob("*.cu")}
    assert all(set(v) <= have for v in _build.COMPONENTS.values())
