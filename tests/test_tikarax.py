"""Tikarax models through the framework: checkpoint folder -> loader -> engine (cache pages, state slots, batches, graphs), against the
plain restatement in tikarax_oracle.py, in 16-bit and in 32-bit."""
import numpy as np
import pytest
import torch

import tikarax_oracle as oracle
from design_util import ARMS, TOL, engine, logit_error, run_portions, tokens_of, write_folder
from machx_inference_engine_b200.models import load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine, OutOfBlocks, SamplingParams

A, M = oracle.attention_layer, oracle.mingru_layer
CONFIGS = {
    # both mixers, different sizes per layer, a layer without feed-forward, widths that fill no vector
    "mixed": oracle.random_config([M(72, 96), A(4, 2, 24, 40, 100), M(50, None), A(6, 1, 20, 12, 64, coef=0.8, every=10)], vocab=131, width=84, groups=3, eps=1e-4),
    "attention-only": oracle.random_config([A(2, 2, 72, 16, 48, coef=0.3, every=33), A(3, 3, 16, 80, None)], vocab=64, width=64, groups=1),
    "mingru-only": oracle.random_config([M(34, 40), M(128, 72)], vocab=90, width=96, groups=12),
    "one-group-odd-width": oracle.random_config([A(4, 4, 8, 8, 30, coef=-0.2, every=5), M(20, 30)], vocab=70, width=50, groups=5),
}
_cache = {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    """name -> (folder, config, weights), written once."""
    def get(name, cfg=None):
        if name not in _cache:
            c = cfg or CONFIGS[name]
            w = oracle.random_weights(c, seed=len(name))
            _cache[name] = (write_folder(tmp_path_factory.mktemp("tikarax") / name, c, w), c, w)
        return _cache[name]
    return get


def expected(folder_entry, tokens):
    _, cfg, w = folder_entry
    return oracle.forward(w, cfg, tokens)[0]


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(folder, arm, name):
    f = folder(name)
    toks = tokens_of(150, f[1]["vocab"], 1)
    assert logit_error(run_portions(engine(f[0], arm), toks, [150]), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
def test_residual_after_every_layer(folder, arm):
    path, cfg, w = folder("mixed")
    toks = tokens_of(30, cfg["vocab"], 2)
    eng = engine(path, arm)
    seen = []

    def tap(li, mixer_out, ffn_out, x):          # x lacks the layer's last branch: add it the way the next norm does
        L = eng.model.layers[li]
        last, wt = (ffn_out, L["norm2b"]) if "ffn" in L else (mixer_out, L["norm1b"])
        n = oracle.grouped_norm(last[:, :cfg["width"]].double().cpu().numpy(), wt.double().cpu().numpy(), cfg["norm"]["eps"], cfg["norm"]["groups"])
        seen.append(x[:, :cfg["width"]].double().cpu().numpy() + n)
    eng.model.tap = tap
    run_portions(eng, toks, [30])
    want = oracle.forward(w, cfg, toks)[1]
    assert len(seen) == len(want)
    for got, ref in zip(seen, want):
        assert np.linalg.norm(got - ref) / np.linalg.norm(ref) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "mingru-only"])
@pytest.mark.parametrize("sizes", [[], [1, 2, 2, 3, 5], [2] * 20, [64, 64, 1, 12], [127, 2, 3], [128, 1, 4], [100, 37]])
def test_portions_and_token_by_token(folder, arm, name, sizes):
    f = folder(name)
    toks = tokens_of(141, f[1]["vocab"], 3)
    assert logit_error(run_portions(engine(f[0], arm), toks, sizes), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
def test_first_tokens_of_a_sequence(folder, arm):
    f = folder("mixed")
    eng = engine(f[0], arm)
    for n in (1, 2, 3):
        toks = tokens_of(n, f[1]["vocab"], 10 + n)
        for sizes in ([n], []):
            assert logit_error(run_portions(eng, toks, sizes), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
def test_long_decoding(folder, arm):
    """Hundreds of single tokens after a short prompt, over two page borders."""
    f = folder("one-group-odd-width")
    n = 300 if arm[0] != "cpu" else 140
    toks = tokens_of(n, f[1]["vocab"], 4)
    eng = engine(f[0], arm)
    assert logit_error(run_portions(eng, toks, [3]), expected(f, toks)) < TOL[arm[1]]
    if arm[0] != "cpu":
        assert eng.stats["graph_replays"] >= n - 3               # decoding went through the CUDA graph that generation replays


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_graphed_prefill_chunk(folder, dtype):
    """A single-sequence portion of a graphed size runs as a graph replay when its last token is all that is wanted."""
    f = folder("mixed")
    toks = tokens_of(700, f[1]["vocab"], 5)
    eng = engine(f[0], ("cuda:0", dtype))
    want = expected(f, toks)
    for start in (0, 130):
        seq = eng.open_sequence()
        if start:
            eng.feed([(seq, toks[:start], [])])
        before = eng.stats["graph_replays"]
        got = eng.feed([(seq, toks[start:start + 512], [511])])
        assert eng.stats["graph_replays"] == before + 1
        assert logit_error(got.cpu().numpy(), want[start + 511:start + 512]) < TOL[dtype]
        eng.abort(seq)


# ------------------------------------------------------------------ batches, pages, slots
@pytest.mark.parametrize("arm", ARMS)
def test_batches_of_unequal_requests_against_each_alone(folder, arm):
    """Portions of some requests beside single tokens of others; requests rest, end, and their pages and slots go to the next ones.  The
    pool holds just what the live requests need."""
    f = folder("mixed")
    V = f[1]["vocab"]
    lens = {"a": 200, "b": 30, "c": 131, "d": 1, "e": 140, "f": 66}
    toks = {k: tokens_of(n, V, 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: expected(f, t) for k, t in toks.items()}
    eng = engine(f[0], arm, num_blocks=1 + 2 + 1 + 2 + 1, max_seqs=4)
    live, at, rng = {}, dict.fromkeys(lens, 0), np.random.default_rng(0)
    queue, held = list(lens), set()
    while queue or live:
        room = eng.bm.n_free() - sum((lens[k] + 127) // 128 - len(s.blocks) for k, s in live.items())
        while queue and len(live) < 4 and (lens[queue[0]] + 127) // 128 <= room:
            room -= (lens[queue[0]] + 127) // 128
            live[queue.pop(0)] = eng.open_sequence()
        picks = [k for k in live if rng.random() < 0.8] or list(live)
        entries, rows = [], []
        for k in picks:
            n = min(int(rng.choice([1, 1, 2, 3, 17, 70, 90])), lens[k] - at[k])
            w = list(range(0, n, 3))
            entries.append((live[k], toks[k][at[k]:at[k] + n], w))
            rows += [(k, at[k] + i) for i in w]
            at[k] += n
        got = eng.feed(entries).cpu().numpy()
        held |= {(k, b) for k in picks for b in live[k].blocks}
        assert logit_error(got, np.stack([want[k][p] for k, p in rows])) < TOL[arm[1]], rows
        for k in picks:
            if at[k] == lens[k]:
                eng.abort(live.pop(k))
    blocks = [b for _, b in held]
    assert len(blocks) > len(set(blocks))                            # some page served two requests
    assert eng.bm.n_free() == 6 and len(eng.sched.free_state) == 4      # everything came back


@pytest.mark.parametrize("arm", ARMS)
def test_used_pages_and_slots_leave_nothing_behind(folder, arm):
    """The same request before and after others have used its pages and its slot, bit for bit."""
    f = folder("mixed")
    toks, other = tokens_of(135, f[1]["vocab"], 6), tokens_of(250, f[1]["vocab"], 7)
    eng = engine(f[0], arm, num_blocks=3, max_seqs=1)
    first = run_portions(eng, toks, [70, 2, 60])
    run_portions(eng, other, [250])
    assert np.array_equal(first, run_portions(eng, toks, [70, 2, 60]))


def test_a_step_that_does_not_fit_is_refused_before_it_runs(folder):
    f = folder("mixed")
    eng = engine(f[0], ("cpu", "fp32"), num_blocks=2, max_seqs=1)
    seq = eng.open_sequence()
    with pytest.raises(OutOfBlocks):
        eng.feed([(seq, tokens_of(129, f[1]["vocab"]), [])])
    assert seq.tokens == []
    eng.abort(seq)
    toks = tokens_of(20, f[1]["vocab"], 8)
    assert logit_error(run_portions(eng, toks, [20]), expected(f, toks)) < TOL["fp32"]
    with pytest.raises(ValueError):
        eng.feed([(eng.open_sequence(), [1, 2], [2])])


# ------------------------------------------------------------------ far keys, long memory
def _needle_model():
    """One attention layer whose query on token QUERY and key on token NEEDLE meet in one dimension, and a head that reads the values."""
    cfg = oracle.random_config([A(2, 1, 16, 24, 32, coef=0.05, every=64, scale=1.0)], vocab=40, width=48, groups=1)
    w = oracle.random_weights(cfg, seed=9)
    e = np.zeros((40, 48), dtype=np.float32)
    e[:, 2:] = w["embed"][:, 2:]
    QUERY, NEEDLE = 38, 39
    e[QUERY, 0] = e[NEEDLE, 1] = 12.0
    for t in ("q", "k"):
        w[f"l0.mix.{t}"] *= 0.0
        w[f"l0.mix.{t}.b"] *= 0.0
    w["l0.mix.q"][::16, 0] = 4.0
    w["l0.mix.k"][0, 1] = 4.0
    w["embed"] = oracle.round_bf16(e)
    return cfg, w, QUERY, NEEDLE


@pytest.mark.parametrize("arm", ARMS)
def test_a_far_key_shows_in_the_logits(folder, arm):
    cfg, w, QUERY, NEEDLE = _needle_model()
    if "needle" not in _cache:
        folder("needle", cfg)                        # (its random weights are replaced by the arranged ones)
        write_folder(_cache["needle"][0], cfg, w)
        _cache["needle"] = (_cache["needle"][0], cfg, w)
    f = _cache["needle"]
    eng = engine(f[0], arm)
    base = tokens_of(400, 38, 11)
    base[399] = base[300] = QUERY
    for place in (0, 1, 127, 128, 255, 256, 299):
        toks = list(base)
        toks[place] = NEEDLE
        want = expected(f, toks)
        moved = logit_error(expected(f, base)[399:], want[399:])      # what losing the key would change
        assert moved > 5 * TOL["bf16"]
        for sizes in ([400], [399], [150, 2, 240]):
            seq, at, got = eng.open_sequence(), 0, None
            for n in list(sizes) + [1] * (400 - sum(sizes)):
                got = eng.feed([(seq, toks[at:at + n], [n - 1])])
                at += n
            eng.abort(seq)
            assert logit_error(got.cpu().numpy(), want[399:]) < TOL[arm[1]], (place, sizes)


@pytest.mark.parametrize("arm", ARMS)
def test_state_remembers_across_portions(folder, arm):
    """A minGRU channel that opens only on one token: its trace decides later logits, and must survive portions, decoding and batches."""
    cfg = oracle.random_config([M(40, None)], vocab=30, width=32, groups=1)
    w = oracle.random_weights(cfg, seed=12)
    w["l0.mix.z"] = w["l0.mix.z"] * 0.0
    w["l0.mix.z.b"] = w["l0.mix.z.b"] * 0.0 - 12.0
    w["embed"] = w["embed"].copy()
    w["embed"][:, 0] = 0.0
    w["embed"][29, 0] = 20.0
    w["l0.mix.z"][:, 0] = 8.0
    w["embed"], w["l0.mix.z"] = oracle.round_bf16(w["embed"]), oracle.round_bf16(w["l0.mix.z"])
    if "memory" not in _cache:
        folder("memory", cfg)
        write_folder(_cache["memory"][0], cfg, w)
    f = (_cache["memory"][0], cfg, w)
    toks = tokens_of(300, 29, 13)
    lost = expected(f, toks)
    toks[2] = 29
    want = expected(f, toks)
    assert logit_error(lost[250:], want[250:]) > 5 * TOL["bf16"]
    for sizes in ([300], [5, 130, 2, 3, 100]):
        assert logit_error(run_portions(engine(f[0], arm), toks, sizes)[250:], want[250:]) < TOL[arm[1]]


# ------------------------------------------------------------------ generation through the scheduler
@pytest.mark.parametrize("arm", ARMS)
def test_greedy_generation_through_the_scheduler(folder, arm):
    """Three requests over chunked prompts; every generated token is the oracle's best (or within rounding of it) in its own context."""
    f = folder("mixed")
    V = f[1]["vocab"]
    prompts = [tokens_of(n, V, 30 + n) for n in (5, 140, 33)]
    device, dtype = arm
    model, _ = load_model(f[0], torch.device(device), max_ctx=512, dtype=dtype)
    eng = LLMEngine(model, EngineOptions(max_ctx=512, max_batch_tokens=48, max_seqs=3))
    outs = eng.generate(prompts, SamplingParams(max_tokens=20, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 20
        lg = oracle.forward(f[2], f[1], p + o[:-1])[0][len(p) - 1:]
        picked = lg[np.arange(20), o]
        assert (lg.max(-1) - picked < 3 * TOL[dtype] * lg.std()).all()
    if device != "cpu":
        assert eng.stats["graph_replays"] > 0


@pytest.mark.parametrize("arm", ARMS)
def test_shared_prefix_resumes_pages_and_state(folder, arm):
    f = folder("mixed")
    shared = tokens_of(270, f[1]["vocab"], 40)
    sp = SamplingParams(max_tokens=4, ignore_eos=True)
    opts = lambda **k: dict(max_ctx=512, max_batch_tokens=128, max_seqs=2, **k)
    model, _ = load_model(f[0], torch.device(arm[0]), max_ctx=512, dtype=arm[1])
    cold = LLMEngine(model, EngineOptions(**opts(enable_prefix_cache=False))).generate([shared + [3, 4]], sp)[0]
    eng = LLMEngine(model, EngineOptions(**opts()))
    eng.generate([shared + [7]], sp)
    seq = eng.add_request(shared + [3, 4], sp)
    while not seq.finished:
        eng.step()
    assert seq.n_cached_prefix == 256 and seq.tokens[len(seq.prompt):] == cold


def test_engine_api_and_sampling(folder):
    from machx_inference_engine_b200.runtime.api import Engine
    f = folder("mixed")
    eng = Engine.load(f[0], "cpu", EngineOptions(max_ctx=256, max_batch_tokens=64, max_seqs=2), dtype="fp32")
    prompt = tokens_of(40, f[1]["vocab"], 50)
    res = eng.generate(prompt, SamplingParams(max_tokens=6, ignore_eos=True))
    lg = oracle.forward(f[2], f[1], prompt + res.token_ids)[0]
    assert res.token_ids == lg[39:45].argmax(-1).tolist()
    a = eng.generate(prompt, SamplingParams(max_tokens=8, temperature=1.0, seed=3, ignore_eos=True)).token_ids
    assert len(a) == 8 and all(0 <= t < f[1]["vocab"] for t in a)
    assert eng.generate("text").error and "tokenizer" in eng.generate("text").error
