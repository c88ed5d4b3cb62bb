"""The mechanisms of Beputar one by one, as the operators the graph calls, against the plain restatement in beputar_oracle.py; on a GPU these are the
sm_100a kernels, on the CPU their PyTorch twins."""
import math

import numpy as np
import pytest
import torch

import beputar_oracle as oracle
from design_util import DEVICES
from machx_inference_engine_b200 import ops
from machx_inference_engine_b200.models.transformer import GatedFFN, ScaledInputMoEFFN
from machx_inference_engine_b200.ops import QuantWeight, WFormat
from machx_inference_engine_b200.utils.rope import rope_tables

DT = {"bf16": torch.bfloat16, "fp32": torch.float32}
TOL = {"bf16": 8e-3, "fp32": 3e-6}
DTYPES = pytest.mark.parametrize("dtype", ["bf16", "fp32"])
ON = pytest.mark.parametrize("device", DEVICES)


def f64(t):
    return t.detach().double().cpu().numpy()


def rel(got, want):
    got, want = (f64(t) if isinstance(t, torch.Tensor) else np.asarray(t, dtype=np.float64) for t in (got, want))
    return float(np.linalg.norm(got - want) / (np.linalg.norm(want) + 1e-30))


def rnd(shape, seed, device, dtype="fp32", std=1.0, mean=0.0):
    return (torch.from_numpy(np.asarray(np.random.default_rng(seed).standard_normal(shape))).float() * std + mean).to(DT[dtype]).to(device)


def weight(n, k, seed, device, e=1):
    return QuantWeight(WFormat.BF16, n, k, e, rnd((e, n, k), seed, device, "bf16", std=k ** -0.5))


def i32(v, device):
    return torch.tensor(v, dtype=torch.int32, device=device)


def layout(lens, before, device):
    """(cu_q, lengths after the step, slots) of a batch: ``lens`` new tokens after ``before`` old ones, slots in reverse order."""
    return i32(np.cumsum([0] + list(lens)).tolist(), device), i32([a + b for a, b in zip(lens, before)], device), i32(list(range(len(lens)))[::-1], device)


class Weights:
    """A source of named arrays, as the blocks ask for them."""

    def __init__(self, arrays, device):
        self.a, self.device = arrays, device

    def matrix(self, name, N, K, E=1, experts=None):
        if "*" in name:
            return QuantWeight(WFormat.BF16, N, K, E, torch.cat([self.matrix(name.replace("*", str(e)), N, K).p0 for e in range(E)]).contiguous())
        return QuantWeight(WFormat.BF16, N, K, 1, torch.from_numpy(self.a[name]).to(torch.bfloat16).reshape(1, N, K).to(self.device).contiguous())


# ------------------------------------------------------------------ norms on a sublayer's output
@ON
@DTYPES
@pytest.mark.parametrize("width,rows", [(64, 1), (50, 7), (4096, 3), (260, 33), (9000, 2)])
def test_sublayer_norm_of_every_kind_of_branch(device, dtype, width, rows):
    ld, eps, K = (width + 31) // 32 * 32, 1e-3, 3
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width)).contiguous()
    vec = lambda s: rnd((width,), s, device, mean=1.0, std=0.3)
    x0, scale, w, wa, wb = rnd((rows, width), 1, device, std=2.0), vec(2), vec(3), vec(4), vec(5)
    a, b = rnd((rows, width), 6, device, dtype, std=0.1), rnd((rows, width), 7, device, dtype, std=3.0)
    y = rnd((rows * K + 5, width), 8, device, dtype)
    pos = torch.from_numpy(np.random.default_rng(9).permutation(rows * K + 5)[:rows * K]).to(torch.int32).to(device)
    picked = f64(y)[f64(pos).astype(int)].reshape(rows, K, width).sum(1)
    norm = lambda t, g: oracle.rms_norm(t, f64(g), eps)
    cases = [(None, None), (pad(a), f64(a)), (ops.ExpertSum(pad(y), pos, K), picked), (ops.ExpertSum(pad(y), pos, K, pad(b)), picked + f64(b)),
             (ops.BranchMean(pad(a), pad(wa), pad(b), pad(wb)), 0.5 * (norm(f64(a), wa) + norm(f64(b), wb)))]
    for delta, d in cases:
        for final in (None, w):
            x = pad(x0)
            got = ops.sublayer_norm(x, delta, pad(scale), eps, w=None if final is None else pad(final), width=width, out_dtype=DT[dtype])
            want = f64(x0) + (0 if d is None else norm(d, scale))
            assert rel(x[:, :width], want) < 1e-6
            assert got.dtype == DT[dtype] and rel(got[:, :width], want if final is None else norm(want, final)) < TOL[dtype]
            assert bool((got[:, width:] == 0).all()) and bool((x[:, width:] == 0).all())
        x = pad(x0)
        assert ops.sublayer_norm(x, delta, pad(scale), eps, width=width, out_dtype=DT[dtype], want_out=False) is None
        assert rel(x[:, :width], f64(x0) + (0 if d is None else norm(d, scale))) < 1e-6


@ON
def test_branches_of_some_rows_only(device):
    y, pos, s = rnd((12, 32), 1, device), i32([3, 0, 7, 9, 2, 11], device), rnd((3, 32), 2, device)
    rows = torch.tensor([2, 0], device=device)
    whole = ops.ExpertSum(y, pos, 2, s)
    assert torch.equal(whole.rows(rows).materialize(), whole.materialize()[rows])
    one = torch.ones(32, device=device)
    m = ops.BranchMean(s, one, 2 * s, one)
    assert torch.equal(m.rows(rows).materialize(1e-6), m.materialize(1e-6)[rows])


# ------------------------------------------------------------------ head epilogue
@ON
@DTYPES
@pytest.mark.parametrize("dim,rot", [(40, 24), (64, 64), (128, 64), (20, 6), (200, 120), (264, 264), (8, 2)])
@pytest.mark.parametrize("interleaved,weighted,after", [(True, False, True), (False, True, False), (False, False, False), (True, True, True)])
def test_head_epilogue(device, dtype, dim, rot, interleaved, weighted, after):
    T, nq, nkv, bs, eps = 5, 3, 2, 128, 1e-2
    dp = (dim + 7) // 8 * 8
    spec = {"base": 5000.0, "dims": rot, "scaling": {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0}}
    cos, sin = rope_tables(600, rot, 5000.0, scaling_type="yarn", scaling_factor=4.0, orig_ctx=64, beta_fast=16.0, beta_slow=1.0, device=device)
    y = rnd((T, (nq + nkv) * dp + 8), 1, device, dtype)
    heads = y[:, :(nq + nkv) * dp].view(T, nq + nkv, dp)
    heads[..., dim:] = 0
    raw = f64(heads)[..., :dim]
    positions = [0, 1, 130, 511, 77]
    w = [torch.nn.functional.pad(rnd((dim,), s, device, mean=1.0, std=0.3), (0, dp - dim)) if weighted else None for s in (2, 3)]
    kc, vc = torch.zeros(4, nkv, bs, dp, dtype=DT[dtype], device=device), torch.zeros(4, nkv, bs, dp, dtype=DT[dtype], device=device)
    slots = [128, 255, 384, -1, 300]
    q = ops.qk_post(y[:, :nq * dp].unflatten(1, (nq, dp)), y[:, nq * dp:(nq + nkv) * dp].unflatten(1, (nkv, dp)), i32(positions, device), cos, sin,
                    torch.tensor(slots, device=device), kc, vc, dim, rot, interleaved=interleaved, q_norm=w[0], k_norm=w[1], norm_after=after, eps=eps)

    def want(x, wn):
        if wn is not None:
            x = oracle.rms_norm(x, f64(wn)[:dim], eps)
        x = oracle.rotate(x, positions, spec, interleaved)
        return oracle.rms_norm(x, 1.0, eps) if after else x
    k = want(raw[:, nq:], w[1])
    assert rel(q[..., :dim], want(raw[:, :nq], w[0])) < TOL[dtype] and bool((q[..., dim:] == 0).all())
    for t, s in enumerate(slots):
        if s >= 0:
            assert rel(kc[s // bs, :, s % bs, :dim], k[t]) < TOL[dtype]
            assert np.array_equal(f64(vc[s // bs, :, s % bs, :dim]), raw[t, nq:])
    assert int((kc.abs().sum(-1) != 0).sum()) == int((vc.abs().sum(-1) != 0).sum()) == 4 * nkv


# ------------------------------------------------------------------ attention: kept first tokens, a score of zero, a gate per head
def _paged(rows, lens, device, dtype, seed):
    """Keys of every sequence [len, G, dim] spread over shuffled pages: (cache, block table)."""
    G, d = rows[0].shape[1:]
    need = [(n + 127) // 128 for n in lens]
    order = (np.random.default_rng(seed).permutation(sum(need)) + 1).tolist()
    cache = torch.full((sum(need) + 1, G, 128, d), 3.0, dtype=DT[dtype], device=device)       # what other requests left in the pages
    table = torch.zeros(len(lens), max(need) + 2, dtype=torch.int32)
    for b, r in enumerate(rows):
        for j in range(need[b]):
            table[b, j] = page = order.pop()
            part = r[j * 128:(j + 1) * 128]
            cache[page, :, :part.shape[0]] = part.permute(1, 0, 2).to(cache.dtype)
    return cache, table.to(device)


@ON
@DTYPES
@pytest.mark.parametrize("window,keep", [(70, 5), (41, 0), (128, 128), (100, 200), (1, 1), (200, 65), (64, 64), (0, 0)])
@pytest.mark.parametrize("H,G,dim,lens,new", [(4, 2, 64, (300, 130, 41), (1, 1, 1)), (6, 1, 40, (300, 200, 7), (150, 2, 7)), (3, 3, 128, (257,), (257,)),
                                              (8, 4, 128, (390, 129), (130, 1)), (2, 1, 24, (140, 70), (5, 3))])
def test_attention_window_with_kept_first_tokens(device, dtype, window, keep, H, G, dim, lens, new):
    g = np.random.default_rng(1)
    dt = DT[dtype]
    keys = [torch.from_numpy(g.standard_normal((n, G, dim))).float().to(dt).to(device) for n in lens]
    vals = [torch.from_numpy(g.standard_normal((n, G, dim))).float().to(dt).to(device) for n in lens]
    q = torch.from_numpy(g.standard_normal((sum(new), H, dim))).float().to(dt).to(device)
    gate = torch.from_numpy(g.standard_normal((sum(new), H + 8))).float().to(dt).to(device)[:, 3:3 + H]
    kc, table = _paged(keys, lens, device, dtype, 2)
    vc, _ = _paged(vals, lens, device, dtype, 2)
    cu = i32(np.cumsum([0] + list(new)).tolist(), device)
    scale = 1.7 / math.sqrt(dim)
    got = ops.attention(q, kc, vc, table, i32(list(lens), device), cu, max(new), sinks=torch.zeros(H, device=device), window=window, scale=scale, gate=gate,
                        keep_first=keep)
    mask = {"size": window, "keep_first": keep} if window else None
    at = 0
    for b, n in enumerate(new):
        want = oracle.attend(f64(q[at:at + n]), f64(keys[b]), f64(vals[b]), scale, mask, sink=True, first_query=lens[b] - n)
        want *= oracle.sigmoid(f64(gate[at:at + n]))[:, :, None]
        assert rel(got[at:at + n], want) < TOL[dtype], b
        at += n


@ON
@DTYPES
@pytest.mark.parametrize("n", [1, 3, 90])
def test_every_edge_of_the_mask_shows(device, dtype, n):
    """One key stands out; it must count just inside the window and among the kept tokens, and not one place further."""
    window, keep, L, d = 100, 5, 391, 32
    for at in (0, 4, 5, 6, L - n - window, L - n - window + 1, L - window - 1, L - window, L - window + 1, 255, 256, L - 1):
        k, v = torch.zeros(L, 1, d), torch.zeros(L, 1, d)
        k[at, 0, 0], v[at, 0, 0] = 12.0, 1.0
        q = torch.zeros(n, 1, d)
        q[:, 0, 0] = 1.0
        kc, table = _paged([k.to(device)], [L], device, dtype, 4)
        vc, _ = _paged([v.to(device)], [L], device, dtype, 4)
        got = ops.attention(q.to(DT[dtype]).to(device), kc, vc, table, i32([L], device), i32([0, n], device), n, sinks=torch.zeros(1, device=device), window=window,
                            scale=1.0, keep_first=keep)
        want = oracle.attend(q.double().numpy(), k.double().numpy(), v.double().numpy(), 1.0, {"size": window, "keep_first": keep}, sink=True, first_query=L - n)
        assert set((want[:, 0, 0] > 0.9).tolist()) <= {True, False} and np.abs(f64(got)[:, 0, 0] - want[:, 0, 0]).max() < 1e-2, at


@ON
@DTYPES
def test_the_zero_score_weighs_what_it_should(device, dtype):
    """With all scores very low the output goes to zero; with equal scores of zero n keys share n / (n + 1)."""
    for shift, total in ((0.0, 30 / 31), (-40.0, 0.0), (40.0, 1.0)):
        k, v = torch.full((30, 1, 16), shift / 16), torch.ones(30, 1, 16)
        for n in (1, 30):
            q = torch.ones(n, 1, 16).to(DT[dtype]).to(device)
            kc, table = _paged([k.to(device)], [30], device, dtype, 5)
            vc, _ = _paged([v.to(device)], [30], device, dtype, 5)
            got = ops.attention(q, kc, vc, table, i32([30], device), i32([0, n], device), n, sinks=torch.zeros(1, device=device), scale=1.0)
            assert abs(float(got[-1].float().mean()) - total) < 5e-3


# ------------------------------------------------------------------ token shift
@ON
@DTYPES
@pytest.mark.parametrize("width,lens,before", [(64, (5,), (0,)), (320, (1, 7, 1, 3), (0, 4, 9, 0)), (2080, (1300, 2, 900), (3, 0, 0)), (32, (1,) * 6, (1, 0, 2, 0, 5, 1))])
def test_token_shift(device, dtype, width, lens, before):
    n = 5
    x, mu = rnd((sum(lens), width), 1, device), rnd((n, width), 2, device, std=0.5)
    state = rnd((len(lens) + 1, width), 3, device)
    old = f64(state)
    cu, sl, slots = layout(lens, before, device)
    got = ops.token_shift(x, mu, state, slots, cu, sl, out_dtype=DT[dtype])
    at = 0
    for b, m in enumerate(lens):
        slot = int(slots[b])
        h = f64(x)[at:at + m]
        first = old[slot:slot + 1] if before[b] else np.zeros((1, width))
        for i in range(n):
            full = oracle.token_shift(np.concatenate([first, h]), f64(mu)[i])[1:]
            assert rel(got[i, at:at + m], full) < TOL[dtype]
        assert np.array_equal(f64(state)[slot], h[-1])
        at += m
    assert np.array_equal(f64(state)[-1], old[-1])


# ------------------------------------------------------------------ recurrences
def _scan_inputs(T, H, dk, dv, seed, device, dtype):
    row = rnd((T, H * (2 * dk + dv) + 8), seed, device, dtype, std=0.7)                      # columns of one projection
    q, k, v = row[:, :H * dk], row[:, H * dk:2 * H * dk], row[:, 2 * H * dk:H * (2 * dk + dv)]
    return q.unflatten(1, (H, dk)), k.unflatten(1, (H, dk)), v.unflatten(1, (H, dv))


SHAPES = [(2, 32, 32), (3, 40, 24), (1, 64, 64), (2, 128, 128), (2, 8, 72), (1, 200, 40), (1, 136, 128), (4, 64, 32)]


@ON
@DTYPES
@pytest.mark.parametrize("H,dk,dv", SHAPES)
@pytest.mark.parametrize("kind", ["fixed", "data"])
def test_decay_scan_whole_and_in_portions(device, dtype, kind, H, dk, dv):
    """Portions of any size, the state carried in a slot, against the whole sequence."""
    T = 70 if device == "cpu" else 333
    q, k, v = _scan_inputs(T, H, dk, dv, 1, device, dtype)
    decay = torch.linspace(0.3, 0.999, H, device=device)
    z, u = rnd((T, H * dk), 2, device, mean=-2.0), rnd((H, dk), 3, device)
    if kind == "fixed":
        s = lambda t: oracle.silu(f64(t))
        want = oracle.decayed_sum(s(q), s(k), s(v), f64(decay))
    else:
        want = oracle.wkv_recurrence(f64(q), f64(k), f64(v), np.exp(-np.exp(f64(z))).reshape(T, H, dk), f64(u))
    for sizes in ([T], [1] * 20 + [T - 20], [2, 3, 16, 17, T - 38], [T - 2, 1, 1]):
        state = torch.full((3, H, dk, dv), 7.0, device=device)                               # what an earlier request left
        at, outs = 0, []
        for n in sizes:
            r = slice(at, at + n)
            kw = dict(decay=decay, silu=True) if kind == "fixed" else dict(z=z[r].contiguous(), u=u)
            outs.append(ops.decay_scan(q[r], k[r], v[r], state, i32([1], device), i32([0, n], device), i32([at + n], device), n, **kw))
            at += n
        got = torch.cat(outs)
        assert got.dtype == torch.float32 and rel(got.view(T, H, dv), want) < (2e-5 if dtype == "fp32" else 8e-3)
        assert bool((state[0] == 7.0).all()) and bool((state[2] == 7.0).all())


@ON
@pytest.mark.parametrize("kind", ["fixed", "data"])
@pytest.mark.parametrize("H,dk,dv", [(2, 64, 64), (2, 128, 128), (3, 40, 24)])
def test_decay_scan_batches_against_each_alone(device, kind, H, dk, dv):
    lens, before = (140, 1, 2, 65, 1, 128), (0, 5, 3, 0, 0, 9)
    T = sum(lens)
    q, k, v = _scan_inputs(T, H, dk, dv, 4, device, "bf16")
    z, u, decay = rnd((T, H * dk), 5, device, mean=-1.0), rnd((H, dk), 6, device), torch.linspace(0.6, 1.0, H, device=device)
    cu, sl, slots = layout(lens, before, device)
    state0 = rnd((len(lens), H, dk, dv), 7, device)
    kw = lambda r: dict(decay=decay, silu=True) if kind == "fixed" else dict(z=z[r].contiguous(), u=u)
    state = state0.clone()
    got = ops.decay_scan(q, k, v, state, slots, cu, sl, max(lens), **kw(slice(0, T)))
    at = 0
    for b, n in enumerate(lens):
        r, alone = slice(at, at + n), state0.clone()
        one = ops.decay_scan(q[r], k[r], v[r], alone, slots[b:b + 1], i32([0, n], device), sl[b:b + 1], n, **kw(r))
        assert rel(got[r], one) < 6e-3 and rel(state[int(slots[b])], alone[int(slots[b])]) < 6e-3      # (long batches run in chunks)
        at += n


@pytest.mark.gpu
@pytest.mark.parametrize("H,dk,dv", [(2, 64, 64), (2, 128, 128), (3, 40, 24), (1, 8, 72), (2, 32, 136), (1, 104, 64)])
@pytest.mark.parametrize("kind", ["fixed", -6.0, -1.0, 1.5, 4.0, "mixed"])
@pytest.mark.parametrize("lens,before", [((64,), (0,)), ((300,), (5,)), ((1, 63, 65, 128, 17, 200), (3, 0, 0, 7, 9, 0))])
def test_chunked_scan_on_the_tensor_cores(kind, H, dk, dv, lens, before):
    """Any mix of chunk lengths, and decays from nearly none to a key channel that forgets at once, in some channels or in all."""
    dev, T, B = "cuda:0", sum(lens), len(lens)
    q, k, v = _scan_inputs(T, H, dk, dv, 8, dev, "bf16")
    decay, u = torch.linspace(0.02, 1.0, H, device=dev), rnd((H, dk), 10, dev)
    z = rnd((T, H * dk), 9, dev, std=0.7, mean=0.0 if isinstance(kind, str) else kind)
    if kind == "mixed":
        z[:, ::3] -= 5.0
        z[:, 1::3] += 5.0
        z[::7, 2::3] = 30.0
    cu, sl, slots = layout(lens, before, dev)
    state0 = rnd((B, H, dk, dv), 7, dev)
    kw = dict(decay=decay, silu=True) if kind == "fixed" else dict(z=z, u=u)
    state, plain = state0.clone(), state0.clone()
    got = ops.decay_scan(q, k, v, state, slots, cu, sl, max(lens), chunked=True, **kw)
    one_by_one = ops.decay_scan(q, k, v, plain, slots, cu, sl, max(lens), chunked=False, **kw)
    at = 0
    for b, n in enumerate(lens):
        r, slot = slice(at, at + n), int(slots[b])
        S = f64(state0)[slot] if before[b] else np.zeros((H, dk, dv))
        want = np.zeros((n, H, dv))
        act = oracle.silu if kind == "fixed" else (lambda x: x)
        qq, kk, vv = (act(f64(t[r])) for t in (q, k, v))
        for t in range(n):
            kv = kk[t][:, :, None] * vv[t][:, None, :]
            if kind == "fixed":
                S = f64(decay)[:, None, None] * S + kv
                want[t] = np.einsum("hd,hdv->hv", qq[t], S)
            else:
                want[t] = np.einsum("hd,hdv->hv", qq[t], S + f64(u)[:, :, None] * kv)
                S = np.exp(-np.exp(f64(z)[at + t])).reshape(H, dk, 1) * S + kv
        assert rel(one_by_one[r].view(n, H, dv), want) < 5e-5 and rel(plain[slot], S) < 5e-5
        assert rel(got[r].view(n, H, dv), want) < 8e-3 and rel(state[slot], S) < 8e-3, b
        at += n


@ON
@pytest.mark.parametrize("n", [1, 200])
def test_slow_decay_remembers_and_fast_decay_forgets(device, n):
    """One key long ago: a head that decays by 0.9999 a token still gives its value, a head that halves does not, and neither overflows."""
    H, d, gap = 3, 64, 600
    decay = torch.tensor([0.9999, 0.5, 1e-6], device=device)
    state = torch.zeros(1, H, d, d, device=device)
    q, k, v = (torch.full((gap, H, d), -30.0, device=device, dtype=torch.bfloat16) for _ in range(3))       # silu(-30) is nearly nothing
    k[0, :, 5], v[0, :, 9] = 1.0, 2.0
    q[:, :, 5] = 1.0
    one = oracle.silu(np.float64(1.0))
    want = np.stack([one * one * oracle.silu(np.float64(2.0)) * np.float64(x) ** (gap - 1) for x in (0.9999, 0.5, 1e-6)])
    at, got = 0, None
    while at < gap:
        m = min(n, gap - at) if at else 300
        got = ops.decay_scan(q[at:at + m], k[at:at + m], v[at:at + m], state, i32([0], device), i32([0, m], device), i32([at + m], device), m, decay=decay, silu=True)
        at += m
    assert bool(torch.isfinite(got).all())
    assert np.abs(f64(got[-1]).reshape(H, d)[:, 9] - want).max() < 1e-2 * want.max()


@ON
def test_the_bonus_belongs_to_the_current_token_only(device):
    H, d = 2, 32
    r = torch.ones(3, H, d, device=device)
    k, v = torch.zeros_like(r), torch.zeros_like(r)
    k[1, :, 3], v[1, :, 7] = 1.0, 1.0
    z = torch.full((3, H * d), math.log(-math.log(0.25)), device=device)                      # a decay of 1/4
    u = torch.full((H, d), 5.0, device=device)
    got = ops.decay_scan(r, k, v, torch.zeros(1, H, d, d, device=device), i32([0], device), i32([0, 3], device), i32([3], device), 3, z=z, u=u)
    col = f64(got).reshape(3, H, d)[:, :, 7]
    assert np.allclose(col, [[0, 0], [5, 5], [1, 1]], atol=1e-5)


# ------------------------------------------------------------------ gated norms
@ON
@DTYPES
@pytest.mark.parametrize("groups,width,live", [(1, 64, 64), (3, 40, 36), (1, 4096, 4096), (64, 64, 64), (1, 192, 150), (2, 9000, 9000)])
@pytest.mark.parametrize("silu", [False, True])
def test_gated_group_norm(device, dtype, groups, width, live, silu):
    T, W, eps = 5, groups * width, 1e-3
    o, w = rnd((T, groups, width), 1, device, std=0.3), rnd((W,), 2, device, mean=1.0)
    o[..., live:] = 0
    gate = rnd((T, W + 16), 3, device, dtype)[:, 8:8 + W]
    got = ops.gated_group_norm(o.reshape(T, W), gate, w, eps, groups=groups, width=live, silu=silu, out_dtype=DT[dtype])
    x = f64(o)
    x = (x / np.sqrt((x[..., :live] ** 2).mean(-1, keepdims=True) + eps)).reshape(T, W) * f64(w)
    assert rel(got, x * (oracle.silu if silu else oracle.sigmoid)(f64(gate))) < TOL[dtype]


# ------------------------------------------------------------------ projections
@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 2, 3, 9, 40, 200])
@pytest.mark.parametrize("N,K", [(64, 64), (96, 160), (200, 320)])
def test_every_matrix_of_a_stack_with_its_own_input(device, dtype, rows, N, K):
    x, w = rnd((4, rows, K), 1, device, dtype), weight(N, K, 2, device, e=4)
    got = ops.stacked_linear(x, w)
    assert got.shape == (4, rows, N) and rel(got, np.einsum("ntk,nmk->ntm", f64(x), f64(w.p0))) < TOL[dtype]


@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 70, 200])
def test_projection_with_tanh_and_the_decay_behind_it(device, dtype, rows):
    """The two small products of a data-dependent decay: a short inner width, the second one with an fp32 offset and fp32 result."""
    for rank, N, K in ((32, 72, 96), (64, 256, 160)):
        x, w1, w2, w0 = rnd((rows, K), 5, device, dtype, std=2.0), weight(rank, K, 6, device), weight(N, rank, 7, device), rnd((N,), 8, device)
        a = ops.linear(x, w1, act=ops.ACT_TANH)
        assert rel(a, np.tanh(f64(x) @ f64(w1.p0[0]).T)) < TOL[dtype]
        z = ops.linear(a, w2, bias=w0, out_f32=True)
        assert z.dtype == torch.float32 and rel(z, f64(a) @ f64(w2.p0[0]).T + f64(w0)) < 1e-5


@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 5, 9, 150])
def test_gated_feed_forward(device, dtype, rows):
    H, row, f = 60, 64, 50
    g = np.random.default_rng(3)
    W = {n: oracle.round_bf16(g.standard_normal(s) / 7) for n, s in {"m.gate": (f, H), "m.up": (f, H), "m.down": (H, f)}.items()}
    h = torch.nn.functional.pad(rnd((rows, H), 1, device, dtype), (0, row - H))
    got = GatedFFN(Weights(W, device), "m", H, row, f)(h)
    assert rel(got[:, :H], oracle.expert({n: a.astype(np.float64) for n, a in W.items()}, "m", f64(h)[:, :H])) < 2 * TOL[dtype]
    assert bool((got[:, H:] == 0).all())


# ------------------------------------------------------------------ routing, experts
@ON
@pytest.mark.parametrize("E,top", [(8, 1), (8, 3), (5, 5), (64, 6), (200, 8), (1, 1)])
def test_sigmoid_routing(device, E, top):
    z = rnd((37, E), 1, device, std=3.0)
    z[0] = 40.0 + torch.arange(E, device=device)                   # scores that all round to one: the order is still the logits'
    z[1] = -40.0 - torch.arange(E, device=device)
    idx, w = ops.moe_route(z, None, top, sigmoid=True)
    want_i, want_w = oracle.route(f64(z), top)
    assert np.array_equal(f64(idx).astype(int), want_i) and np.allclose(f64(w), want_w, rtol=1e-6, atol=0)


@ON
@DTYPES
@pytest.mark.parametrize("packed", [False, True])
def test_rows_scaled_for_their_experts(device, dtype, packed):
    T, K, E, H = 11, 3, 7, 96
    x, w = rnd((T, H), 1, device, dtype), torch.rand(T, K, device=device)
    idx = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:K] for t in range(T)]).to(torch.int32).to(device)
    pk = ops.moe_pack(idx, E) if packed else None
    got = ops.moe_scale_rows(x, w, pk)
    at = pk.pair_to_packed.long() if packed else torch.arange(T * K, device=device)
    assert rel(got[at], (f64(w)[..., None] * f64(x)[:, None]).reshape(T * K, H)) < TOL[dtype]


@ON
@DTYPES
@pytest.mark.parametrize("rows", [1, 3, 5, 9, 40, 200])
@pytest.mark.parametrize("E,top,f,shared", [(6, 2, 40, 24), (8, 1, 64, 0), (3, 3, 20, 64)])
def test_experts_whose_weight_scales_their_input(device, dtype, rows, E, top, f, shared):
    H, row = 60, 64
    g = np.random.default_rng(2)
    mlp = oracle.feed_forward((E, top, f, shared))
    W = {"m.router": oracle.round_bf16(g.standard_normal((E, H)) / 4)}
    for p, n in [(f"m.e{e}", f) for e in range(E)] + ([("m.shared", shared)] if shared else []):
        for name, s in ((".gate", (n, H)), (".up", (n, H)), (".down", (H, n))):
            W[p + name] = oracle.round_bf16(g.standard_normal(s) / 6)
    h = rnd((rows, H), 4, device, dtype, std=2.0)
    z = np.sort(f64(h) @ W["m.router"].T.astype(np.float64), axis=1)[:, ::-1]
    clear = np.ones(rows, bool) if top == E else (z[:, top - 1] - z[:, top] > 1e-3)           # a choice within rounding of another says nothing
    got = ScaledInputMoEFFN(Weights(W, device), "m", H, row, E, top, f, shared)(torch.nn.functional.pad(h, (0, row - H))).materialize()
    want = oracle.moe_mlp({n: a.astype(np.float64) for n, a in W.items()}, "m", mlp, f64(h))
    assert clear.any() and rel(f64(got)[clear, :H], want[clear]) < 2 * TOL[dtype]
    assert bool((got[:, H:] == 0).all())


# ------------------------------------------------------------------ rotation tables
@pytest.mark.parametrize("scaling", [None, (8.0, 1000, 30.0, 1.0), (4.0, 64, 16.0, 1.0), (2.0, 30, 64.0, 0.5), (1.0, 100, 8.0, 2.0)])
@pytest.mark.parametrize("dims,base", [(64, 10000.0), (24, 500.0), (2, 1e6)])
def test_rotation_tables(scaling, dims, base):
    rot = oracle._rot(dims, base, scaling)
    f, mag = oracle.frequencies(rot)
    a = np.arange(700)[:, None] * f
    kw = {} if scaling is None else dict(scaling_type="yarn", scaling_factor=scaling[0], orig_ctx=scaling[1], beta_fast=scaling[2], beta_slow=scaling[3])
    cos, sin = rope_tables(700, dims, base, **kw)
    assert np.abs(f64(cos) - np.cos(a) * mag).max() < 1e-6 and np.abs(f64(sin) - np.sin(a) * mag).max() < 1e-6
