"""Pubodra models through the framework: checkpoint folder -> loader -> engine (cache pages, batches, graphs), against the plain restatement in
pubodra_oracle.py, in 16-bit and in 32-bit."""
import numpy as np
import pytest
import torch

import pubodra_oracle as oracle
from design_util import ARMS, engine, logit_error, run_portions, tokens_of, write_folder
from machx_inference_engine_b200.models import load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine, OutOfBlocks, SamplingParams

TOL = {"fp32": 1e-5, "bf16": 1.5e-2}      # of the logits, whose size the tied table sets
L = oracle.latent_layer
YARN = (4.0, 100, 16.0, 1.0)
CONFIGS = {
    # layers that differ in every size; experts, dense and no feed-forward; a loop in the middle; widths that fill no vector
    "mixed": oracle.random_config([L(3, 20, 6, 28, 36, 50, 100), L(5, 16, 8, 24, 40, 129, (6, 2, 40), base=5000.0, scaling=YARN),
                                   L(2, 40, 10, 12, 20, 7, None, scaling=(2.0, 64, 8.0, 2.0)), L(4, 24, 16, 40, 64, 90, 72)],
                                  vocab=131, width=84, eps=1e-3, loop=(1, 3, 2)),
    "no-loop": oracle.random_config([L(4, 32, 16, 48, 64, 128, 64, scaling=YARN), L(2, 64, 64, 64, 128, 200, (4, 4, 64))], vocab=64, width=64),
    "all-looped": oracle.random_config([L(2, 16, 8, 16, 24, 33, (5, 1, 24)), L(3, 8, 4, 20, 16, 64, 50)], vocab=90, width=50, loop=(0, 2, 3)),
    # widths that the expanded form does not take
    "latent-space-only": oracle.random_config([L(2, 200, 72, 264, 40, 60, 64), L(1, 24, 8, 16, 24, 100, 40)], vocab=60, width=64),
    "one-pass-loop-at-the-end": oracle.random_config([L(2, 24, 8, 32, 48, 1, 40), L(1, 100, 12, 72, 88, 140, 96)], vocab=70, width=96, loop=(1, 2, 1)),
}
_cache = {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    """name -> (folder, config, weights), written once."""
    def get(name, cfg=None, weights=None):
        if name not in _cache:
            c = cfg or CONFIGS[name]
            w = weights or oracle.random_weights(c, seed=len(name), clear_routing=True)
            _cache[name] = (write_folder(tmp_path_factory.mktemp("pubodra") / name, c, w), c, w)
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
    for n in (150, 40):                       # expanded keys, latent space
        toks = tokens_of(n, f[1]["vocab"], n)
        assert logit_error(run_portions(engine(f[0], arm), toks, [n]), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "all-looped"])
def test_residual_after_every_layer_run(folder, arm, name):
    path, cfg, w = folder(name)
    toks = tokens_of(30, cfg["vocab"], 2)
    eng = engine(path, arm)
    seen = []
    last = {}

    def tap(i, mixer_out, ffn_out, x):          # x holds the mixer's output already when the layer has a feed-forward
        branch = ffn_out if "norm2" in eng.model.layers[eng.model.runs[i][0]] else mixer_out
        seen.append((x + branch.float())[:, :cfg["width"]].double().cpu().numpy())
        last["n"] = i
    eng.model.tap = tap
    run_portions(eng, toks, [30])
    want = oracle.forward(w, cfg, toks)[1]
    assert len(seen) == len(want) == last["n"] + 1
    for got, ref in zip(seen, want):
        assert np.linalg.norm(got - ref) / np.linalg.norm(ref) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "no-loop"])
@pytest.mark.parametrize("sizes", [[], [1, 2, 2, 3, 5], [2] * 20, [64, 64, 1, 12], [127, 2, 3], [128, 1, 4], [100, 37], [63, 70], [3, 130]])
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
    """Hundreds of single tokens after a short prompt, over two page borders; every window passes over decoded tokens."""
    f = folder("mixed")
    n = 300 if arm[0] != "cpu" else 150
    toks = tokens_of(n, f[1]["vocab"], 4)
    eng = engine(f[0], arm)
    assert logit_error(run_portions(eng, toks, [3]), expected(f, toks)) < TOL[arm[1]]
    if arm[0] != "cpu":
        assert eng.stats["graph_replays"] >= n - 3               # decoding went through the CUDA graph that generation replays


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_graphed_prefill_chunk(folder, dtype):
    """A single-sequence portion of a graphed size runs as a graph replay when its last token is all that is wanted; the page list of a portion is
    formed anew by every replay."""
    f = folder("mixed")
    toks = tokens_of(900, f[1]["vocab"], 5)
    eng = engine(f[0], ("cuda:0", dtype))
    want = expected(f, toks)
    for start in (0, 130, 333):
        seq = eng.open_sequence()
        if start:
            eng.feed([(seq, toks[:start], [])])
        before = eng.stats["graph_replays"]
        got = eng.feed([(seq, toks[start:start + 512], [511])])
        assert eng.stats["graph_replays"] == before + 1
        assert logit_error(got.cpu().numpy(), want[start + 511:start + 512]) < TOL[dtype]
        eng.abort(seq)


# ------------------------------------------------------------------ batches, pages
@pytest.mark.parametrize("arm", ARMS)
def test_batches_of_unequal_requests_against_each_alone(folder, arm):
    """Long portions of some requests beside short ones and single tokens of others, in any order; requests rest, end, and their pages go to the
    next ones.  The pool holds just what the live requests need."""
    f = folder("mixed")
    V = f[1]["vocab"]
    lens = {"a": 200, "b": 30, "c": 131, "d": 1, "e": 140, "f": 66}
    toks = {k: tokens_of(n, V, 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: expected(f, t) for k, t in toks.items()}
    eng = engine(f[0], arm, num_blocks=1 + 2 + 1 + 2 + 1, max_seqs=4)
    live, at, rng = {}, dict.fromkeys(lens, 0), np.random.default_rng(1)
    queue, held, both = list(lens), set(), 0
    while queue or live:
        room = eng.bm.n_free() - sum((lens[k] + 127) // 128 - len(s.blocks) for k, s in live.items())
        while queue and len(live) < 4 and (lens[queue[0]] + 127) // 128 <= room:
            room -= (lens[queue[0]] + 127) // 128
            live[queue.pop(0)] = eng.open_sequence()
        picks = [k for k in live if rng.random() < 0.8] or list(live)
        rng.shuffle(picks)
        entries, rows, ns = [], [], []
        for k in picks:
            n = min(int(rng.choice([1, 1, 2, 17, 66, 70, 90])), lens[k] - at[k])
            w = list(range(0, n, 3))
            entries.append((live[k], toks[k][at[k]:at[k] + n], w))
            rows += [(k, at[k] + i) for i in w]
            at[k] += n
            ns.append(n)
        both += min(ns) < 64 <= max(ns)
        got = eng.feed(entries).cpu().numpy()
        held |= {(k, b) for k in picks for b in live[k].blocks}
        assert logit_error(got, np.stack([want[k][p] for k, p in rows])) < TOL[arm[1]], rows
        for k in picks:
            if at[k] == lens[k]:
                eng.abort(live.pop(k))
    blocks = [b for _, b in held]
    assert both >= 3                                                 # long and short queries met in a batch
    assert len(blocks) > len(set(blocks))                            # some page served two requests
    assert eng.bm.n_free() == 6                                      # everything came back


@pytest.mark.parametrize("arm", ARMS)
def test_used_pages_leave_nothing_behind(folder, arm):
    """The same request before and after others have used its pages, bit for bit."""
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


@pytest.mark.parametrize("arm", ARMS)
def test_every_pass_has_its_own_cache(folder, arm):
    """Three passes over two layers: as many caches as layer runs, all of them different after a prompt."""
    f = folder("all-looped")
    eng = engine(f[0], arm)
    seq = eng.open_sequence()
    eng.feed([(seq, tokens_of(40, f[1]["vocab"], 9), [])])
    assert len(eng.kv.k) == 6 and eng.kv.v[0].numel() == 0
    pages = [eng.kv.k[i][seq.blocks[0], 0, :40].float().cpu() for i in range(6)]
    for a, b in ((0, 2), (0, 4), (2, 4), (1, 3), (3, 5)):
        assert float((pages[a] - pages[b]).abs().max()) > 0.1
    assert eng.model.kv_bytes_per_block() == sum(t[0].numel() * t.element_size() for t in eng.kv.k.values())


# ------------------------------------------------------------------ far keys, window edges
def _needle_model(window):
    """One attention layer whose query on token QUERY and key on token NEEDLE meet in one dimension; the values reach the logits."""
    cfg = oracle.random_config([L(2, 16, 8, 24, 32, window, 32, scale=1.0)], vocab=40, width=48)
    w = oracle.random_weights(cfg, seed=9)
    e = np.array(w["embed"])
    e[:, :2] = 0.0
    QUERY, NEEDLE = 38, 39
    e[QUERY, 0] = e[NEEDLE, 1] = 4.0
    w["embed"] = oracle.round_bf16(e)
    for n in ("l0.norm1", "l0.norm1.b"):
        w[n] = w[n] * 0.0 + (1.0 if n == "l0.norm1" else 0.0)
    w["l0.mix.q"] *= 0.0
    w["l0.mix.q"][[0, 24], 0] = 8.0                                  # unrotated element 0 of both heads
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, 1] = 40.0                                     # latent element 0 marks the needle ...
    w["l0.mix.uk"] *= 0.0
    w["l0.mix.uk"][[0, 16], 0] = 4.0                                 # ... and is unrotated key element 0
    return cfg, w, QUERY, NEEDLE


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("window", [100, 128, 300])
def test_a_far_key_shows_in_the_logits_until_the_window_has_passed(folder, arm, window):
    cfg, w, QUERY, NEEDLE = _needle_model(window)
    f = folder(f"needle-{window}", cfg, w)
    eng = engine(f[0], arm)
    base = tokens_of(400, 38, 11)
    base[399] = base[350] = QUERY
    for gap in (1, window - 2, window - 1, window, 127, 128, 271):
        toks = list(base)
        toks[399 - gap] = NEEDLE
        want = expected(f, toks)
        moved = logit_error(expected(f, base)[399:], want[399:])      # what the needle changes
        assert moved > 5 * TOL["bf16"] if gap < window else moved < 1e-9, (gap, moved)
        for sizes in ([400], [399], [150, 2, 240], [330, 69]):
            seq, at, got = eng.open_sequence(), 0, None
            for n in list(sizes) + [1] * (400 - sum(sizes)):
                got = eng.feed([(seq, toks[at:at + n], [n - 1])])
                at += n
            eng.abort(seq)
            assert logit_error(got.cpu().numpy(), want[399:]) < TOL[arm[1]], (gap, sizes)


# ------------------------------------------------------------------ generation through the scheduler
@pytest.mark.parametrize("arm", ARMS)
def test_greedy_generation_through_the_scheduler(folder, arm):
    """Four requests over chunked prompts, long portions beside decoding; every generated token is the oracle's best (or within rounding of it) in
    its own context."""
    f = folder("mixed")
    V = f[1]["vocab"]
    prompts = [tokens_of(n, V, 30 + n) for n in (5, 140, 33, 200)]
    device, dtype = arm
    model, _ = load_model(f[0], torch.device(device), max_ctx=512, dtype=dtype)
    eng = LLMEngine(model, EngineOptions(max_ctx=512, max_batch_tokens=80, max_seqs=3))
    outs = eng.generate(prompts, SamplingParams(max_tokens=20, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 20
        lg = oracle.forward(f[2], f[1], p + o[:-1])[0][len(p) - 1:]
        picked = lg[np.arange(20), o]
        assert (lg.max(-1) - picked < 3 * TOL[dtype] * lg.std()).all()
    if device != "cpu":
        assert eng.stats["graph_replays"] > 0


@pytest.mark.parametrize("arm", ARMS)
def test_shared_prefix_is_not_computed_again(folder, arm):
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
