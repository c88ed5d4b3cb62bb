"""The mechanisms of Zegelix one by one, as the operators the graph calls, against the plain restatement in zegelix_oracle.py; on a GPU these are the
sm_100a kernels, on the CPU their PyTorch twins."""
import numpy as np
import pytest
import torch

import zegelix_oracle as oracle
from design_util import DEVICES
from machx_inference_engine_b200 import ops
from machx_inference_engine_b200.models.hybrid import RecurrentState, RglruBlock
from machx_inference_engine_b200.models.transformer import ClampedMoEFFN, ForwardBatch, KVCache, PooledAttentionBlock, pair_order
from machx_inference_engine_b200.ops import QuantWeight, WFormat
from machx_inference_engine_b200.utils.rope import rope_tables

DT = {"bf16": torch.bfloat16, "fp32": torch.float32}
TOL = {"bf16": 8e-3, "fp32": 3e-6}
DTYPES = pytest.mark.parametrize("dtype", ["bf16", "fp32"])
ON = pytest.mark.parametrize("device", DEVICES)
PAGE = KVCache.BLOCK


def f64(t):
    return t.detach().double().cpu().numpy()


def rel(got, want):
    got, want = (f64(t) if isinstance(t, torch.Tensor) else np.asarray(t, dtype=np.float64) for t in (got, want))
    return float(np.linalg.norm(got - want) / (np.linalg.norm(want) + 1e-30))


def rnd(shape, seed, device, dtype="fp32", std=1.0, mean=0.0):
    return (torch.from_numpy(np.asarray(np.random.default_rng(seed).standard_normal(shape))).float() * std + mean).to(DT[dtype]).to(device)


def i32(v, device):
    return torch.tensor(v, dtype=torch.int32, device=device)


def pad_cols(t, to):
    return torch.nn.functional.pad(t, (0, to - t.shape[-1])).contiguous()


class Weights:
    """A source of named arrays, as the blocks ask for them."""

    def __init__(self, arrays, device):
        self.a, self.device = arrays, device

    def matrix(self, name, N, K, E=1, experts=None):
        if "*" in name:
            return QuantWeight(WFormat.BF16, N, K, E, torch.cat([self.matrix(name.replace("*", str(e)), N, K).p0 for e in range(E)]).contiguous())
        assert self.a[name].shape == (N, K)
        return QuantWeight(WFormat.BF16, N, K, 1, torch.from_numpy(self.a[name]).to(torch.bfloat16).reshape(1, N, K).to(self.device).contiguous())

    def table(self, name, shape):
        assert self.a[name].shape == tuple(shape)
        return torch.from_numpy(np.array(self.a[name], dtype=np.float32)).to(self.device)

    def vector(self, name, n):
        return self.table(name, (n,))


class Batch:
    """Sequences over one pool of pages (in scattered order), stepped by :meth:`step`."""

    def __init__(self, lens, device, slots=None):
        self.device, self.done, n = device, [0] * len(lens), [(x + PAGE - 1) // PAGE for x in lens]
        order = np.random.default_rng(sum(lens)).permutation(np.arange(1, sum(n) + 1))
        self.pages, width = sum(n) + 1, max(n)
        self.table = np.zeros((len(lens), width), dtype=np.int32)
        at = 0
        for i, k in enumerate(n):
            self.table[i, :k] = order[at:at + k]
            at += k
        self.slots = slots or list(range(len(lens)))[::-1]

    def step(self, counts):
        """counts: new tokens per sequence (0: it rests).  ForwardBatch of the step and the positions of its rows."""
        live = [i for i, c in enumerate(counts) if c]
        pos = [np.arange(self.done[i], self.done[i] + counts[i]) for i in live]
        slot = [self.table[i][p // PAGE].astype(np.int64) * PAGE + p % PAGE for i, p in zip(live, pos)]
        for i in live:
            self.done[i] += counts[i]
        at, d = np.concatenate(pos), self.device
        return ForwardBatch(i32([0] * len(at), d), i32(at.tolist(), d), torch.tensor(np.concatenate(slot), device=d), torch.tensor(self.table[live], device=d),
                            i32([self.done[i] for i in live], d), i32(np.cumsum([0] + [counts[i] for i in live]).tolist(), d), max(counts),
                            state_slots=i32([self.slots[i] for i in live], d), max_kv_len=max(self.done[i] for i in live)), live, pos


# ------------------------------------------------------------------ residual add + norm
@ON
@DTYPES
@pytest.mark.parametrize("width,rows", [(64, 1), (50, 7), (4096, 3), (260, 33), (9000, 2)])
def test_branches_join_the_residual_as_they_are(device, dtype, width, rows):
    ld, eps, K = (width + 31) // 32 * 32, 1e-3, 3
    x0, w = rnd((rows, width), 1, device, std=2.0), rnd((width,), 2, device, mean=1.0, std=0.3)
    a, y = rnd((rows, width), 3, device, dtype), rnd((rows * K + 5, width), 4, device, dtype)
    pos = torch.from_numpy(np.random.default_rng(9).permutation(rows * K + 5)[:rows * K]).to(torch.int32).to(device)
    pw = torch.rand(rows, K, generator=torch.Generator().manual_seed(1)).to(device)
    z = rnd((rows, 12), 5, device, std=2.0)
    picked = (f64(y)[f64(pos).astype(int)].reshape(rows, K, width) * f64(pw)[..., None]).sum(1)
    shared = f64(a) * oracle.sigmoid(f64(z)[:, 7:8])
    cases = [(None, 0.0), (pad_cols(a, ld), f64(a)), (ops.ExpertSum(pad_cols(y, ld), pos, K, w=pw), picked),
             (ops.ExpertSum(pad_cols(y, ld), pos, K, pad_cols(a, ld), pw, z[:, 7]), picked + shared)]
    for delta, d in cases:
        for final in (None, w):
            x, both = pad_cols(x0, ld), torch.full((rows, 2 * ld), 5.0, dtype=DT[dtype], device=device)
            got = ops.sublayer_norm(x, delta, None, eps, w=None if final is None else pad_cols(w, ld), width=width, out_dtype=DT[dtype], out=both[:, ld:])
            want = f64(x0) + d
            assert rel(x[:, :width], want) < 1e-6
            assert got.data_ptr() == both[:, ld:].data_ptr() and bool((both[:, :ld] == 5.0).all())
            assert rel(got[:, :width], want if final is None else oracle.rms_norm(want, f64(w), eps)) < TOL[dtype]
            assert bool((got[:, width:] == 0).all()) and bool((x[:, width:] == 0).all())


@ON
def test_weighted_rows_of_some_tokens_only(device):
    y, pos, s, w, z = rnd((12, 32), 1, device), i32([3, 0, 7, 9, 2, 11], device), rnd((3, 32), 2, device), torch.rand(3, 2, device=device), rnd((3, 4), 3, device)
    rows = torch.tensor([2, 0], device=device)
    whole = ops.ExpertSum(y, pos, 2, s, w, z[:, 1])
    assert torch.equal(whole.rows(rows).materialize(), whole.materialize()[rows])


# ------------------------------------------------------------------ head epilogue
@ON
@DTYPES
@pytest.mark.parametrize("T", [1, 6, 700])
@pytest.mark.parametrize("dim,rot,vdim", [(40, 24, 56), (64, 64, 64), (128, 64, 96), (20, 6, 18), (200, 120, 264), (8, 0, 8), (96, 96, 24)])
def test_head_epilogue_with_values_of_their_own(device, dtype, T, dim, rot, vdim):
    nq, nkv, base = 6, 2, 3000.0
    dk, dv = (dim + 7) // 8 * 8, (vdim + 7) // 8 * 8
    kr, vr = rope_tables(900, rot, base, device=device), rope_tables(900, vdim, base, device=device)
    y = rnd((T, nq * dk + nkv * (dk + dv) + 8), 1, device, dtype)
    q, k = y[:, :nq * dk].unflatten(1, (nq, dk)), y[:, nq * dk:(nq + nkv) * dk].unflatten(1, (nkv, dk))
    v = y[:, (nq + nkv) * dk:(nq + nkv) * dk + nkv * dv].unflatten(1, (nkv, dv))
    for t, d in ((q, dim), (k, dim), (v, vdim)):
        t[..., d:] = 0
    temp = rnd((nq,), 2, device, mean=1.0, std=0.5)
    temp[1] = -0.7
    pos = np.random.default_rng(T).permutation(900)[:T]
    pos[0] = 0
    slots = np.random.default_rng(3).permutation(np.arange(PAGE, 8 * PAGE))[:T]
    if T > 2:
        slots[2] = -1
    pages = lambda d: torch.zeros(8, nkv, PAGE, d, dtype=DT[dtype], device=device)
    kc, vc = pages(dk), pages(dv)
    order = lambda x, d, r: np.argsort(pair_order(d, r).numpy())          # from neighbouring pairs back to half splits
    raw = {n: f64(t)[..., :d][..., order(t, d, r)] for n, t, d, r in (("q", q, dim, rot), ("k", k, dim, rot), ("v", v, vdim, vdim))}
    got = ops.qk_post(q, k, i32(pos.tolist(), device), *kr, torch.tensor(slots.astype(np.int64), device=device), kc, vc, dim, rot, interleaved=True, v=v, v_rope=vr,
                      q_scale=temp)
    want = oracle.turn(raw["q"], pos, rot, base) if rot else raw["q"]
    assert rel(f64(got)[..., :dim][..., order(q, dim, rot)], want * f64(temp)[:, None]) < TOL[dtype] and bool((got[..., dim:] == 0).all())
    for cache, d, r, n in ((kc, dim, rot, "k"), (vc, vdim, vdim, "v")):
        want = oracle.turn(raw[n], pos, r, base) if r else raw[n]
        for t in range(T):
            if slots[t] < 0:
                continue
            row = f64(cache[slots[t] // PAGE, :, slots[t] % PAGE])
            assert rel(row[:, :d][:, order(cache, d, r)], want[t]) < TOL[dtype] and not row[:, d:].any()
        assert not cache[0].any()


# ------------------------------------------------------------------ attention with pooled blocks
def attention_setup(device, dtype, lens, heads, kv_heads, dk, dv, window, pool, seed=0, std=1.0):
    b = Batch(lens, device)
    kv = KVCache(1, b.pages, kv_heads, dk, torch.device(device), [0], dtype=dtype, geometry={0: (kv_heads, dk, dv)}, pools={0: (pool, window)} if pool else None)
    mk = lambda i, n, w, s: rnd((lens[i], n, w), seed + 10 * i + s, device, dtype, std=std)
    seqs = [(mk(i, heads, dk, 1), mk(i, kv_heads, dk, 2), mk(i, kv_heads, dv, 3), mk(i, heads, dv, 4)) for i in range(len(lens))]
    return b, kv, seqs


def attention_step(b, kv, seqs, counts, device, dtype, window, scale, cap=0.0, sinks=None, out_rope=None, gated=False, n_splits=None):
    """One step: keys and values into the pages, pooled blocks formed, attention.  Returns the rows per live sequence."""
    fb, live, pos = b.step(counts)
    cut = lambda j: torch.cat([seqs[i][j][p[0]:p[-1] + 1] for i, p in zip(live, pos)])
    q, k, v, g = (cut(j) for j in range(4))
    nkv, pools, dense = k.shape[1], kv.pools.get(0), None
    if fb.max_q_len == 1 and pools is not None:
        flat = torch.cat([k.flatten(1), v.flatten(1)], dim=1)
        none = rope_tables(4, 0, 10.0, device=device)
        ops.qk_post(q.clone(), flat[:, :nkv * k.shape[2]].unflatten(1, k.shape[1:]), fb.positions, *none, fb.slot_map, kv.k[0], kv.v[0], k.shape[2], 0, interleaved=True,
                    v=flat[:, nkv * k.shape[2]:].unflatten(1, v.shape[1:]), v_rope=none, pools=pools, block_table=fb.block_table)
    else:
        ops.kv_store(k.flatten(1), v.flatten(1), fb.slot_map, kv.k[0], kv.v[0])
        if pools is not None:
            dense = ops.pool_blocks(kv.k[0], kv.v[0], pools, fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, max_kv_len=fb.max_kv_len)
    kw = {} if n_splits is None else {"n_splits": n_splits}
    out = ops.attention(q, kv.k[0], kv.v[0], fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, sinks=sinks, window=window, scale=scale, softcap=cap,
                        max_kv_len=fb.max_kv_len, gate=g.flatten(1) if gated else None, pools=pools, pool_dense=dense, out_rope=out_rope, **kw)
    return {i: o for i, o in zip(live, torch.split(out, [len(p) for p in pos]))}


def attention_want(seq, window, pool, scale, cap, sinks, base, gated):
    q, k, v, g = (f64(t) for t in seq)
    mask = {"size": window, **({"pool": pool} if pool else {})} if window else None
    o = oracle.attend(q, k, v, scale, mask, cap, None if sinks is None else f64(sinks))
    if base:
        dv = v.shape[2]
        order = pair_order(dv, dv).numpy()
        o = oracle.turn(o[..., np.argsort(order)], -np.arange(q.shape[0]), dv, base)[..., order]
    return o * oracle.sigmoid(g) if gated else o


@ON
@DTYPES
@pytest.mark.parametrize("heads,kv_heads,dk,dv", [(6, 2, 40, 56), (4, 4, 64, 64), (4, 1, 128, 128), (2, 1, 72, 24), (3, 3, 48, 136)])
@pytest.mark.parametrize("window,pool", [(50, 5), (1, 3), (128, 16), (136, 12), (100, 1), (40, 150), (33, 0), (0, 0)])
def test_window_and_pooled_blocks(device, dtype, heads, kv_heads, dk, dv, window, pool):
    """Every piece at once, whole prompts of unequal lengths, then single tokens."""
    lens, base, scale, cap = [330, 70, 201], 500.0, dk ** -0.5, 8.0
    if device == "cpu" and dk != 40:
        lens = [150, 9]
    b, kv, seqs = attention_setup(device, dtype, lens, heads, kv_heads, dk, dv, window, pool, std=2.0)
    sinks, turn = rnd((heads,), 77, device), rope_tables(400, dv, base, device=device)
    want = [attention_want(s, window, pool, scale, cap, sinks, base, True) for s in seqs]
    first = [n - 3 for n in lens]
    kw = dict(cap=cap, sinks=sinks, out_rope=turn, gated=True)
    got = [[o] for _, o in sorted(attention_step(b, kv, seqs, first, device, dtype, window, scale, **kw).items())]
    for _ in range(3):
        for i, o in attention_step(b, kv, seqs, [1] * len(lens), device, dtype, window, scale, **kw).items():
            got[i].append(o)
    for g, w in zip(got, want):
        g = torch.cat(g)
        assert rel(g, w) < 1.5 * TOL[dtype]
        assert max(rel(g[t], w[t]) for t in range(len(w))) < 6 * TOL[dtype]           # no row of its own is off


@ON
@DTYPES
@pytest.mark.parametrize("sizes", [[2] * 30, [64, 2, 3, 70], [1] * 40, [100, 1, 1, 66, 5], [63, 129]])
@pytest.mark.parametrize("window,pool", [(50, 7), (20, 12), (5, 40)])
def test_pooled_blocks_over_portions(device, dtype, sizes, window, pool):
    lens = [sum(sizes), max(sum(sizes) // 2, 3)]
    b, kv, seqs = attention_setup(device, dtype, lens, 4, 2, 24, 40, window, pool)
    want = [attention_want(s, window, pool, 0.3, 0.0, None, 0.0, False) for s in seqs]
    got = [[], []]
    for n in sizes:
        other = min(n, lens[1] - b.done[1]) if n % 3 else 0                           # the second request rests now and then
        for i, o in attention_step(b, kv, seqs, [n, other], device, dtype, window, 0.3).items():
            got[i].append(o)
    for g, w in zip(got, want):
        if g:
            g = torch.cat(g)
            assert rel(g, w[:len(g)]) < 1.5 * TOL[dtype]


@ON
@DTYPES
@pytest.mark.parametrize("window,pool", [(50, 5), (130, 12), (64, 128), (7, 33)])
@pytest.mark.parametrize("long", [False, True])
def test_edges_of_window_and_blocks(device, dtype, window, pool, long):
    """One key stands out so far that a query that sees its token, or the block it is pooled into, says so: the token until it has left the window, nothing
    until the whole block lies before the window, then the block."""
    T, dk = 290, 16
    for at in (0, 1, pool - 1, pool, 127, 128, 130, 2 * pool + 1):
        b, kv, seqs = attention_setup(device, dtype, [T], 2, 1, dk, 16, window, pool, std=0.05)
        q, k, v, _ = seqs[0]
        q[..., 3], k[at, :, 3], v[at] = 8.0, 8.0 * pool, 64.0
        want = attention_want(seqs[0], window, pool, 0.5, 0.0, None, 0.0, False)
        block = at // pool
        seen = lambda p: at <= p < at + window or (block + 1) * pool - 1 <= p - window
        assert all((abs(want[p]).max() > 0.3) == seen(p) for p in range(T))
        edges = [p for p in (at, at + window - 1, at + window, (block + 1) * pool - 2 + window, (block + 1) * pool - 1 + window) if 2 <= p < T]
        if long:
            runs = [[T]]
        else:
            runs = [[p - 1, 2, 1] for p in sorted(set(edges))]
        for sizes in runs:
            b.done = [0]
            got = torch.cat([attention_step(b, kv, seqs, [n], device, dtype, window, 0.5)[0] for n in sizes if n])
            n = min(len(got), T)
            assert rel(got[-3:], want[n - 3:n]) < 2 * TOL[dtype] or np.abs(f64(got[-3:]) - want[n - 3:n]).max() < 2e-2 * (dtype == "bf16")
            if long:
                assert all((abs(f64(got[p])).max() > 0.3) == seen(p) for p in range(T))


@ON
@pytest.mark.parametrize("scale,cap", [(0.05, 20.0), (1.0, 20.0), (6.0, 50.0), (3.0, 2.0), (0.0001, 30.0)])
def test_soft_cap_of_small_and_large_scores(device, scale, cap):
    """The tensor-core kernel forms tanh in two ways; rows whose scores are all small and rows that saturate."""
    b, kv, seqs = attention_setup(device, "bf16", [300], 2, 1, 64, 64, 90, 8, std=1.5)
    got = attention_step(b, kv, seqs, [300], device, "bf16", 90, scale, cap=cap)[0]
    assert rel(got, attention_want(seqs[0], 90, 8, scale, cap, None, 0.0, False)) < 8e-3


@ON
@DTYPES
def test_sink_joins_once_whatever_the_ranges(device, dtype):
    lens, window, pool = [400], 60, 4
    for big in (-3.0, 0.0, 6.0):
        sinks = torch.full((4,), big, device=device)
        for n_splits in (None, 1, 3, 7):
            b, kv, seqs = attention_setup(device, dtype, lens, 4, 2, 32, 32, window, pool)
            want = attention_want(seqs[0], window, pool, 0.4, 0.0, sinks, 0.0, False)
            attention_step(b, kv, seqs, [399], device, dtype, window, 0.4, sinks=sinks)
            got = attention_step(b, kv, seqs, [1], device, dtype, window, 0.4, sinks=sinks, n_splits=n_splits)[0]
            assert rel(got, want[399:]) < 2 * TOL[dtype]


@ON
@DTYPES
@pytest.mark.parametrize("pool,window", [(5, 20), (12, 1), (128, 30), (150, 40), (3, 200)])
def test_rows_of_pool_pages(device, dtype, pool, window):
    """What the pages hold after prompts in portions and after decoding: the means, each at its place beside the page of the block's last token."""
    n = 420
    for sizes in ([n], [70, 2, 348], [400] + [1] * 20):
        b, kv, seqs = attention_setup(device, dtype, [n], 2, 2, 16, 8, window, pool)
        for s in sizes:
            attention_step(b, kv, seqs, [s], device, dtype, window, 1.0)
        pages = kv.pools[0]
        assert pages.k.shape[2] == -(-PAGE // pool)
        for which, x in ((pages.k, seqs[0][1]), (pages.v, seqs[0][2])):
            means = oracle.pooled(f64(x), pool)
            for blk in range(max(n - window, 0) // pool):
                page = (blk * pool + pool - 1) // PAGE
                first = next(i for i in range(blk + 1) if (i * pool + pool - 1) // PAGE == page)
                assert rel(which[int(b.table[0, page]), :, blk - first], means[blk]) < TOL[dtype], blk


# ------------------------------------------------------------------ the attention block
@ON
@DTYPES
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,window,pool", [(4, 2, 20, 36, 12, 30, 7), (3, 1, 40, 24, 40, 60, 12)])
def test_attention_block(device, dtype, heads, kv_heads, dim, vdim, rot, window, pool):
    H, row, T = 50, 64, 150
    cfg = oracle.random_config([oracle.attention_layer(None, heads, kv_heads, dim, vdim, window, pool, rot, base=700.0, cap=10.0)], width=H)
    W, m = oracle.random_weights(cfg, seed=2), cfg["layers"][0]["mixer"]
    blk = PooledAttentionBlock(Weights(W, device), "l0.mix", H, row, heads, kv_heads, dim, vdim, m["scale"], window, 10.0, rot,
                               rope_tables(300, rot, 700.0, device=device), rope_tables(300, vdim, 700.0, device=device))
    b = Batch([T], device)
    kv = KVCache(1, b.pages, kv_heads, blk.dk, torch.device(device), [3], dtype=dtype, geometry={3: (kv_heads, blk.dk, blk.dv)}, pools={3: (pool, window)})
    h = rnd((T, H), 5, device, dtype)
    want = oracle.attention({n: np.float64(a) for n, a in W.items()}, "l0.mix", m, f64(h))
    got, at = [], 0
    for n in (70, 3, 1, 1, 74, 1):
        fb, _, _ = b.step([n])
        got.append(blk(pad_cols(h[at:at + n], row), fb, kv, 3))
        at += n
    got = torch.cat(got)
    assert rel(got[:, :H], want) < 2 * TOL[dtype] and bool((got[:, H:] == 0).all())


# ------------------------------------------------------------------ convolution and recurrence
@ON
@DTYPES
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("C", [32, 160])
def test_causal_convolution(device, dtype, taps, C):
    lens = [45, 1, 7, 130]
    x = [rnd((n, C + 32), i, device, dtype) for i, n in enumerate(lens)]
    w, bias = rnd((C, taps), 50, device), rnd((C,), 51, device)
    want = [oracle.causal_conv(f64(t)[:, :C], f64(w), f64(bias)) for t in x]
    state = torch.full((5, taps - 1, C), 3.0, dtype=DT[dtype], device=device)        # slots are not reset: a start does not read them
    b, got = Batch(lens, device, slots=[2, 0, 4, 1]), [[] for _ in lens]
    for counts in ([20, 1, 2, 64], [1, 0, 1, 1], [2, 0, 1, 2], [1, 0, 0, 60], [21, 0, 3, 3]):
        fb, live, pos = b.step(counts)
        y = ops.causal_conv(torch.cat([x[i][p[0]:p[-1] + 1] for i, p in zip(live, pos)])[:, :C], w, bias, state, fb.state_slots, fb.cu_q, fb.seq_lens, fb.max_q_len)
        for i, o in zip(live, torch.split(y, [len(p) for p in pos])):
            got[i].append(o)
    for g, ref in zip(got, want):
        assert rel(torch.cat(g), ref) < TOL[dtype]
    assert bool((state[3] == 3.0).all())
    for i, slot in enumerate([2, 0, 4, 1]):
        tail = np.concatenate([np.zeros((taps - 1, C)), f64(x[i])[:, :C]])[len(x[i]):]
        assert rel(state[slot], tail) < 1e-30 + TOL[dtype] or taps == 1


@ON
@DTYPES
@pytest.mark.parametrize("blocks,n", [(3, 16), (1, 40), (16, 8), (2, 256)])
def test_recurrence(device, dtype, blocks, n):
    W, lens = blocks * n, [300, 1, 65, 140] if device != "cpu" else [60, 1, 20]
    r, i = (rnd((sum(lens), blocks, n), s, device) for s in (1, 2))
    gates, bias = torch.cat([r, i], dim=2).contiguous(), rnd((blocks, 2 * n), 3, device)
    u, y = rnd((sum(lens), W + 8), 4, device, dtype), rnd((sum(lens), W + 16), 5, device, dtype, std=2.0)
    lam = np.random.default_rng(6).uniform(-9.0, 2.0, W)
    coef = torch.from_numpy(-8.0 * np.logaddexp(0.0, lam)).float().to(device)
    act = oracle.sigmoid(f64(gates + bias))
    r64, i64 = act[..., :n].reshape(-1, W), act[..., n:].reshape(-1, W)
    state = torch.full((len(lens) + 1, W), 9.0, device=device)
    b, start, got = Batch(lens, device), np.cumsum([0] + lens), [[] for _ in lens]
    for part in (0.4, 0.05, 1.0):
        counts = [min(max(int(k * part), 1), k - d) if part < 1 else k - d for k, d in zip(lens, b.done)]
        fb, live, pos = b.step(counts)
        rows = np.concatenate([start[j] + p for j, p in zip(live, pos)])
        o = ops.rglru_scan(gates[rows], u[rows][:, :W], y[rows][:, 8:8 + W], bias, coef, state, fb.state_slots, fb.cu_q, fb.seq_lens, fb.max_q_len)
        for j, t in zip(live, torch.split(o, [len(p) for p in pos])):
            got[j].append(t)
    for j in range(len(lens)):
        s = slice(start[j], start[j + 1])
        S = oracle.gated_recurrence(f64(u)[s, :W], r64[s], i64[s], lam)
        assert rel(torch.cat(got[j]), S * oracle.gelu_tanh(f64(y)[s, 8:8 + W])) < TOL[dtype]
        assert rel(state[b.slots[j]], S[-1]) < 2e-6 if dtype == "fp32" or device == "cpu" else 1e-5
    assert bool((state[len(lens)] == 9.0).all())


@ON
@DTYPES
def test_slow_and_fast_decays(device, dtype):
    """Gates from closed to open over decays from "hundreds of thousands of tokens" to "at once": 1 - a^2 where a is all but one, and where it is zero."""
    n, T = 64, 200
    lam = np.linspace(-14.0, 6.0, n)
    coef = torch.from_numpy(-8.0 * np.logaddexp(0.0, lam)).float().to(device)
    gates = torch.zeros(T, 1, 2 * n, device=device)
    gates[..., :n] = torch.linspace(-6, 6, T, device=device).reshape(T, 1, 1)
    u = rnd((T, n), 1, device, dtype)
    y = torch.full((T, n), 3.0, dtype=DT[dtype], device=device)
    state, b = torch.zeros(1, n, device=device), Batch([T], device)
    fb, _, _ = b.step([T])
    got = ops.rglru_scan(gates, u, y, torch.zeros(1, 2 * n, device=device), coef, state, fb.state_slots, fb.cu_q, fb.seq_lens, T)
    act = oracle.sigmoid(f64(gates))
    want = oracle.gated_recurrence(f64(u), act[:, 0, :n], act[:, 0, n:], lam)
    err = np.abs(f64(state[0]) - want[-1]) / np.abs(want).max(0)
    assert err.max() < (2e-6 if dtype == "fp32" else 2e-5)
    assert rel(got, want * oracle.gelu_tanh(3.0)) < TOL[dtype]


@ON
@DTYPES
@pytest.mark.parametrize("batch", [1, 2, 3, 5, 8, 19])
@pytest.mark.parametrize("width,blocks,taps", [(60, 3, 4), (20, 1, 2), (160, 2, 3), (96, 12, 1), (512, 2, 4)])
def test_recurrent_block_decodes_as_it_reads(device, dtype, batch, width, blocks, taps):
    """Prompts of unequal lengths, then single tokens through the one-kernel form, against the restatement."""
    H, row = 44, 64
    cfg = oracle.random_config([oracle.rglru_layer(None, width, blocks, taps)], width=H)
    W = oracle.random_weights(cfg, seed=batch)
    blk = RglruBlock(Weights(W, device), "l0.mix", H, row, width, blocks, taps)
    lens = [2 + (7 * i) % 23 for i in range(batch)]
    total = [k + 4 for k in lens]
    h = [rnd((k, H), 100 + i, device, dtype) for i, k in enumerate(total)]
    tensors = blk.state_tensors(batch + 2, DT[dtype], device)
    for t in tensors.values():
        t.fill_(5.0)
    state = RecurrentState(batch + 2, {n: {1: t} for n, t in tensors.items()}, device)
    b, got = Batch(total, device), [[] for _ in lens]
    lens[0] = 1                                           # one sequence starts in a step of single tokens, beside a row of the batch that does not
    for counts in ([0] + lens[1:], *[[1] * batch] * 3):
        if not any(counts):
            continue
        fb, live, pos = b.step(counts)
        o = blk(torch.cat([pad_cols(h[i][p[0]:p[-1] + 1], row) for i, p in zip(live, pos)]), fb, state, 1)
        for i, t in zip(live, torch.split(o, [len(p) for p in pos])):
            got[i].append(t)
    W64 = {k: np.float64(a) for k, a in W.items()}
    for g, x in zip(got, h):
        g = torch.cat(g)
        want = oracle.rglru(W64, "l0.mix", cfg["layers"][0]["mixer"], f64(x))[:len(g)]
        assert rel(g[:, :H], want) < 2.5 * TOL[dtype] and bool((g[:, H:] == 0).all())
    assert bool((state.tensors["S"][1][batch:] == 5.0).all())


# ------------------------------------------------------------------ projections, experts
@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 3, 5, 70, 200])
def test_per_block_products_in_fp32(device, dtype, rows):
    for blocks, n in ((3, 32), (2, 80), (16, 8)):
        x = rnd((rows, blocks * n + 16), 1, device, dtype)
        w = QuantWeight(WFormat.BF16, 2 * n, n, blocks, rnd((blocks, 2 * n, n), 2, device, "bf16", std=n ** -0.5))
        got = ops.head_linear(x[:, :blocks * n].unflatten(1, (blocks, n)), w, out_f32=True)
        assert got.dtype == torch.float32
        assert rel(got, np.einsum("tbk,bnk->tbn", f64(x)[:, :blocks * n].reshape(rows, blocks, n), f64(w.p0))) < 2e-6


@ON
@pytest.mark.parametrize("E,top,ld", [(8, 1, 8), (8, 3, 16), (5, 5, 8), (64, 6, 72), (1, 1, 8)])
def test_routing_over_the_first_columns(device, E, top, ld):
    z = rnd((37, ld), 1, device, std=3.0)
    z[:, E:] = 100.0                                     # columns that are no experts
    idx, w = ops.moe_route(z, None, top, experts=E)
    want_i, want_w = oracle.route(f64(z)[:, :E], top)
    assert np.array_equal(f64(idx).astype(int), want_i) and np.allclose(f64(w), want_w, rtol=2e-6, atol=1e-12)


@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 3, 5, 9, 40, 200])
@pytest.mark.parametrize("E,top,f,limit,shared,shared_limit", [(6, 2, 40, 1.0, 24, 0.4), (8, 1, 64, 7.0, 0, 0.0), (3, 3, 20, 0.3, 64, 2.0), (9, 4, 32, 2.0, 32, 2.0)])
def test_clamped_experts(device, dtype, rows, E, top, f, limit, shared, shared_limit):
    H, row = 60, 64
    g = np.random.default_rng(2)
    mlp = oracle.feed_forward((E, top, f, limit, shared, shared_limit))
    W = {"m.router": oracle.round_bf16(g.standard_normal((E, H)) / 4), "m.router.b": oracle.round_bf16(g.standard_normal(E))}
    for p, n in [(f"m.e{e}", f) for e in range(E)] + ([("m.shared", shared)] if shared else []):
        for name, s in ((".gate", (n, H)), (".up", (n, H)), (".down", (H, n))):
            W[p + name] = oracle.round_bf16(g.standard_normal(s) / 6)
    if shared:
        W["m.shared.sg"] = oracle.round_bf16(g.standard_normal((1, H)) / 5)
    h = rnd((rows, H), 4, device, dtype, std=2.0)
    z = np.sort(f64(h) @ W["m.router"].T.astype(np.float64) + W["m.router.b"], axis=1)[:, ::-1]
    clear = np.ones(rows, bool) if top == E else (z[:, top - 1] - z[:, top] > 1e-3)           # a choice within rounding of another says nothing
    got = ClampedMoEFFN(Weights(W, device), "m", H, row, E, top, f, limit, shared, shared_limit)(pad_cols(h, row)).materialize()
    want = oracle.experts({n: a.astype(np.float64) for n, a in W.items()}, "m", mlp, f64(h))
    assert clear.any() and rel(f64(got)[clear, :H], want[clear]) < 2 * TOL[dtype]
    assert bool((got[:, H:] == 0).all())
