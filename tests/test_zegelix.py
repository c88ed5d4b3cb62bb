"""Zegelix models through the framework: checkpoint folder -> loader -> engine (cache and pool pages, state slots, batches, graphs), against the plain
restatement in zegelix_oracle.py, in 16-bit and in 32-bit."""
import numpy as np
import pytest
import torch

import zegelix_oracle as oracle
from design_util import ARMS, engine, logit_error, run_portions, tokens_of, write_folder
from machx_inference_engine_b200.models import load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine, OutOfBlocks, SamplingParams

TOL = {"fp32": 2e-5, "bf16": 3e-2}
A, R = oracle.attention_layer, oracle.rglru_layer
CONFIGS = {
    # layers that differ in every size, a loop in the middle, layers without a feed-forward; widths and heads that fill no vector
    "mixed": oracle.random_config([R((6, 2, 40, 1.0, 24, 0.5), 60, 3, 4), A((5, 1, 32, 3.0, 0, 0.0), 6, 2, 20, 36, 50, 7, 12, base=500.0, cap=12.0),
                                   A(None, 3, 3, 40, 24, 129, 12, 40), R(None, 40, 1, 2), A((4, 4, 24, 0.7, 40, 7.0), 2, 1, 24, 24, 20, 33, 24, cap=0.0),
                                   R((3, 1, 20, 2.0, 16, 2.0), 96, 4, 1)], vocab=131, width=84, eps=1e-3, scale=5.0, logit_scale=0.3, loop=(1, 4, 2)),
    "tensor-core-widths": oracle.random_config([A((8, 2, 64, 7.0, 64, 7.0), 4, 2, 64, 128, 100, 16, 32, cap=50.0), R((8, 2, 32, 1.0, 0, 0.0), 128, 2, 3),
                                                A((4, 2, 32, 1.0, 32, 1.0), 4, 2, 128, 64, 128, 8, 128)], vocab=64, width=128, loop=(0, 3, 2)),
    "whole-loop-once": oracle.random_config([A(None, 2, 2, 32, 16, 0, 0, 8), R((3, 2, 32, 1.0, 0, 0.0), 48, 2, 5)], vocab=90, width=50, eps=1e-2, scale=1.0,
                                            logit_scale=4.0, loop=(0, 2, 1)),
    "recurrent-only": oracle.random_config([R((4, 2, 24, 1.5, 8, 1.5), 64, 8, 4), R(None, 24, 1, 3)], vocab=60, width=64, loop=(1, 2, 2)),
    "attention-only": oracle.random_config([A((4, 2, 24, 1.5, 8, 1.5), 3, 1, 28, 20, 33, 0, 28), A(None, 2, 1, 16, 40, 30, 140, 6)], vocab=60, width=40),
}
_cache = {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    """name -> (folder, config, weights), written once."""
    def get(name, cfg=None, weights=None):
        if name not in _cache:
            c = cfg or CONFIGS[name]
            w = weights or oracle.random_weights(c, seed=len(name))
            _cache[name] = (write_folder(tmp_path_factory.mktemp("zegelix") / name, c, w), c, w)
        return _cache[name]
    return get


_logits = {}


def expected(entry, tokens):
    path, cfg, w = entry
    key = (path, tuple(tokens))
    if key not in _logits:
        _logits[key] = oracle.forward(cfg, w, tokens)
    return _logits[key]


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(folder, arm, name):
    f = folder(name)
    for n in (150, 40):
        toks = tokens_of(n, f[1]["vocab"], n)
        assert logit_error(run_portions(engine(f[0], arm), toks, [n]), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "whole-loop-once"])
def test_residual_after_every_layer_run(folder, arm, name):
    path, cfg, w = folder(name)
    toks = tokens_of(30, cfg["vocab"], 2)
    eng = engine(path, arm)
    seen, H = [], cfg["width"]

    def tap(i, mixer_out, ffn_out, x):          # x holds the mixer's branch already when the layer has a feed-forward
        second = "moe" in eng.model.layers[eng.model.runs[i][0]]
        seen.append((x + (ffn_out if second else mixer_out)).double().cpu().numpy()[:, :H])
    eng.model.tap = tap
    run_portions(eng, toks, [30])
    want = []
    oracle.forward(cfg, w, toks, want)
    assert len(seen) == len(want) == len(oracle.runs(cfg))
    for got, ref in zip(seen, want):
        assert np.linalg.norm(got - ref) / np.linalg.norm(ref) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "tensor-core-widths"])
@pytest.mark.parametrize("sizes", [[], [1, 2, 2, 3, 5], [2] * 20, [64, 64, 1, 12], [127, 2, 3], [128, 1, 4], [100, 37], [63, 70], [3, 130]])
def test_portions_and_token_by_token(folder, arm, name, sizes):
    f = folder(name)
    toks = tokens_of(141, f[1]["vocab"], 3)
    assert logit_error(run_portions(engine(f[0], arm), toks, sizes), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "recurrent-only", "attention-only"])
def test_first_tokens_of_a_sequence(folder, arm, name):
    f = folder(name)
    eng = engine(f[0], arm)
    for n in (1, 2, 3):
        toks = tokens_of(n, f[1]["vocab"], 10 + n)
        for sizes in ([n], []):
            assert logit_error(run_portions(eng, toks, sizes), expected(f, toks)) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
def test_long_decoding(folder, arm):
    """Hundreds of single tokens after a short prompt, over page borders; every window passes over decoded tokens, whose blocks become visible."""
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
    """A single-sequence portion of a graphed size runs as a graph replay when its last token is all that is wanted, from zeros or from a carried state."""
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


# ------------------------------------------------------------------ batches, pages, slots
@pytest.mark.parametrize("arm", ARMS)
def test_batches_of_unequal_requests_against_each_alone(folder, arm):
    """Long portions of some requests beside short ones and single tokens of others, in any order; requests rest, end, and their pages and state slots go
    to the next ones.  The pool holds just what the live requests need."""
    f = folder("mixed")
    V = f[1]["vocab"]
    lens = {"a": 200, "b": 30, "c": 131, "d": 1, "e": 140, "f": 66}
    toks = {k: tokens_of(n, V, 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: expected(f, t) for k, t in toks.items()}
    eng = engine(f[0], arm, num_blocks=1 + 2 + 1 + 2 + 1, max_seqs=4)
    live, at, rng = {}, dict.fromkeys(lens, 0), np.random.default_rng(1)
    queue, held, slots = list(lens), set(), []
    while queue or live:
        room = eng.bm.n_free() - sum((lens[k] + 127) // 128 - len(s.blocks) for k, s in live.items())
        while queue and len(live) < 4 and (lens[queue[0]] + 127) // 128 <= room:
            room -= (lens[queue[0]] + 127) // 128
            live[queue.pop(0)] = eng.open_sequence()
        picks = [k for k in live if rng.random() < 0.8] or list(live)
        rng.shuffle(picks)
        entries, rows = [], []
        for k in picks:
            n = min(int(rng.choice([1, 1, 2, 17, 66, 70, 90])), lens[k] - at[k])
            w = list(range(0, n, 3))
            entries.append((live[k], toks[k][at[k]:at[k] + n], w))
            rows += [(k, at[k] + i) for i in w]
            at[k] += n
        got = eng.feed(entries).cpu().numpy()
        held |= {(k, b) for k in picks for b in live[k].blocks}
        assert logit_error(got, np.stack([want[k][p] for k, p in rows])) < TOL[arm[1]], rows
        for k in picks:
            if at[k] == lens[k]:
                slots.append(live[k].state_slot)
                eng.abort(live.pop(k))
    blocks = [b for _, b in held]
    assert len(blocks) > len(set(blocks)) and len(slots) > len(set(slots))     # some page and some slot served two requests
    assert eng.bm.n_free() == 6 and len(eng.sched.free_state) == 4             # everything came back


@pytest.mark.parametrize("arm", ARMS)
def test_used_pages_and_slots_leave_nothing_behind(folder, arm):
    """The same request before and after others have used its pages and its slot, bit for bit."""
    f = folder("mixed")
    toks, other = tokens_of(135, f[1]["vocab"], 6), tokens_of(250, f[1]["vocab"], 7)
    eng = engine(f[0], arm, num_blocks=3, max_seqs=1)
    first = run_portions(eng, toks, [70, 2, 60])
    run_portions(eng, other, [250])
    assert np.array_equal(first, run_portions(eng, toks, [70, 2, 60]))
    run_portions(eng, other, [3])
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


def test_every_run_of_a_layer_has_its_own_cache_and_state(folder):
    assert engine(folder("attention-only")[0], ("cpu", "fp32")).state is None
    eng = engine(folder("mixed")[0], ("cpu", "fp32"))
    # runs: 0 | 1 2 3, twice | 4 5
    assert {l: tuple(k.shape[1:]) for l, k in eng.kv.k.items()} == {**{i: (2, 128, 24) for i in (1, 4)}, **{i: (3, 128, 40) for i in (2, 5)}, 7: (1, 128, 24)}
    assert {l: tuple(v.shape[1:]) for l, v in eng.kv.v.items()} == {**{i: (2, 128, 40) for i in (1, 4)}, **{i: (3, 128, 24) for i in (2, 5)}, 7: (1, 128, 24)}
    assert {l: tuple(p.v.shape[1:]) for l, p in eng.kv.pools.items()} == {**{i: (2, 19, 40) for i in (1, 4)}, **{i: (3, 11, 24) for i in (2, 5)}, 7: (1, 4, 24)}
    shapes = {n: {l: tuple(t.shape[1:]) for l, t in d.items()} for n, d in eng.state.tensors.items()}
    assert shapes["S"] == {0: (96,), 3: (64,), 6: (64,), 8: (96,)}
    assert shapes["conv"] == {0: (3, 96), 3: (1, 64), 6: (1, 64), 8: (0, 96)}


# ------------------------------------------------------------------ far keys, window and block edges, sinks, long memory
def _needle_model(window, pool):
    """One layer whose query on token QUERY and key on token NEEDLE meet in one dimension that is not rotated; the needle's value reaches the logits."""
    QUERY, NEEDLE, H = 38, 39, 48
    cfg = oracle.random_config([A(None, 2, 1, 24, 16, window, pool, 4, scale=3.0, cap=60.0)], vocab=40, width=H, scale=1.0)
    w, p = oracle.random_weights(cfg, seed=9), "l0.mix"
    for n in ("q.b", "k.b"):
        w[f"{p}.{n}"] *= 0.0
    w[f"{p}.sink"][:] = -2.0
    w[f"{p}.temp"][:] = 1.0
    e = np.array(w["embed"])
    e[:, :2] = 0.0
    e[QUERY, 0] = e[NEEDLE, 1] = 8.0
    w["embed"] = oracle.round_bf16(e)
    for n in ("q", "k"):
        w[f"{p}.{n}"] = oracle.round_bf16(w[f"{p}.{n}"] * 0.05)
    w[f"{p}.q"][[20, 44], 0] = 4.0
    w[f"{p}.k"][20, 1] = 4.0
    w[f"{p}.v"][:, 1] = oracle.round_bf16(8.0 * w[f"{p}.v"][:, 1])
    return cfg, w, QUERY, NEEDLE


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("window,pool", [(100, 6), (128, 4), (61, 5), (130, 8)])
def test_a_far_key_shows_while_it_or_its_block_is_seen(folder, arm, window, pool):
    cfg, w, QUERY, NEEDLE = _needle_model(window, pool)
    f = folder(f"needle-{window}-{pool}", cfg, w)
    eng = engine(f[0], arm)
    n = 400
    base = tokens_of(n, 38, 11)
    base[n - 1] = QUERY
    newest = (n - 1 - window - pool + 1) // pool                       # the last block that the query sees
    for at in (n - 2, n - window, n - window - 1, (newest + 1) * pool, (newest + 1) * pool - 1, newest * pool, 272, 140, 128, 127, pool, pool - 1, 0):
        toks = list(base)
        toks[at] = NEEDLE
        want = expected(f, toks)
        moved = logit_error(expected(f, base)[n - 1:], want[n - 1:])  # what the needle changes
        seen = n - 1 - at < window or (at // pool + 1) * pool - 1 <= n - 1 - window
        assert moved > 3 * TOL["bf16"] if seen else moved < 0.02, (at, moved, seen)
        for sizes in ([n], [n - 1], [150, 2, 240], [330, 69]):
            seq, done, got = eng.open_sequence(), 0, None
            for k in list(sizes) + [1] * (n - sum(sizes)):
                got = eng.feed([(seq, toks[done:done + k], [k - 1])])
                done += k
            eng.abort(seq)
            assert logit_error(got.cpu().numpy(), want[n - 1:]) < TOL[arm[1]], (at, sizes)


@pytest.mark.parametrize("arm", ARMS)
def test_the_sink_takes_its_share(folder, arm):
    """Sinks that outweigh every score: a model that left them out, scaled, capped or counted them per tile or block would be far off."""
    cfg = oracle.random_config([A(None, 4, 2, 16, 16, 40, 5, 16, cap=2.0)], vocab=40, width=48, scale=1.0)
    w = oracle.random_weights(cfg, seed=5)
    w["l0.mix.sink"] = oracle.round_bf16(np.array([4.0, -30.0, 5.0, 2.0]))
    f = folder("sink", cfg, w)
    toks = tokens_of(200, 40, 13)
    want = expected(f, toks)
    assert logit_error(oracle.forward(cfg, {**w, "l0.mix.sink": w["l0.mix.sink"] * 0.0}, toks), want) > 3 * TOL["bf16"]
    for sizes in ([200], [199], [64, 2, 100]):
        assert logit_error(run_portions(engine(f[0], arm), toks, sizes), want) < TOL[arm[1]]


@pytest.mark.parametrize("arm", ARMS)
def test_a_slow_state_remembers_hundreds_of_tokens(folder, arm):
    """The first token decides a logit 299 tokens later, through the state alone; the whole prompt, portions and decoding agree."""
    cfg = oracle.random_config([R(None, 32, 2, 3)], vocab=40, width=48, scale=1.0)
    w = oracle.random_weights(cfg, seed=3)
    w["l0.mix.lam"][:] = -9.0                                        # a decay of at most e^-0.001 a token
    w["l0.mix.ri.b"][:] = -2.0
    w["embed"][:39, 40:] = w["embed"][39, :40] = 0.0                 # a token with columns of its own, which the recurrence reads loudly
    w["l0.mix.x"][:, 40:] = oracle.round_bf16(5.0 * w["l0.mix.x"][:, 40:])
    f = folder("memory", cfg, w)
    toks = tokens_of(300, 39, 12)
    other = [39] + toks[1:]
    want = expected(f, other)
    assert logit_error(expected(f, toks)[299:], want[299:]) > 2 * TOL["bf16"]
    for sizes in ([300], [299], [64, 2, 3, 231], [100]):
        assert logit_error(run_portions(engine(f[0], arm), other, sizes)[-1:], want[-1:]) < TOL[arm[1]]


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
        lg = oracle.forward(f[1], f[2], p + o[:-1])[len(p) - 1:]
        picked = lg[np.arange(20), o]
        assert (lg.max(-1) - picked < 3 * TOL[dtype] * lg.std()).all()
    if device != "cpu":
        assert eng.stats["graph_replays"] > 0


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("name", ["mixed", "attention-only"])
def test_shared_prefix_is_not_computed_again(folder, arm, name):
    """Pages, the pooled rows in them and the state's snapshot at a page border serve the next request with the same beginning."""
    f = folder(name)
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


def test_pooled_rows_move_with_their_pages(folder):
    eng = engine(folder("mixed")[0], ("cpu", "fp32"))
    for p in eng.kv.pools.values():
        p.k[2], p.v[2] = 3.0, 4.0
    eng.kv.copy_blocks([2], [5])
    assert all(bool((p.k[5] == 3.0).all()) and bool((p.v[5] == 4.0).all()) for p in eng.kv.pools.values())


def test_engine_api_and_sampling(folder):
    from machx_inference_engine_b200.runtime.api import Engine
    f = folder("mixed")
    eng = Engine.load(f[0], "cpu", EngineOptions(max_ctx=256, max_batch_tokens=64, max_seqs=2), dtype="fp32")
    prompt = tokens_of(40, f[1]["vocab"], 50)
    res = eng.generate(prompt, SamplingParams(max_tokens=6, ignore_eos=True))
    lg = oracle.forward(f[1], f[2], prompt + res.token_ids)
    assert res.token_ids == lg[39:45].argmax(-1).tolist()
    a = eng.generate(prompt, SamplingParams(max_tokens=8, temperature=1.0, seed=3, ignore_eos=True)).token_ids
    assert len(a) == 8 and all(0 <= t < f[1]["vocab"] for t in a)
