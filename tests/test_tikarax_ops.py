"""The mechanisms of Tikarax one by one, as the operators the graph calls, against the plain restatement in tikarax_oracle.py; on a GPU
these are the sm_100a kernels, on the CPU their PyTorch twins."""
import numpy as np
import pytest
import torch

import tikarax_oracle as oracle
from design_util import DEVICES
from machx_inference_engine_b200 import ops
from machx_inference_engine_b200.ops import QuantWeight, WFormat
from machx_inference_engine_b200.utils.rope import query_temperature_table

DT = {"bf16": torch.bfloat16, "fp32": torch.float32}
TOL = {"bf16": 8e-3, "fp32": 2e-6}


def rel(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.linalg.norm(got.detach().double().cpu().numpy() - want) / (np.linalg.norm(want) + 1e-30))


def f64(t):
    return t.detach().double().cpu().numpy()


def rnd(shape, seed, device, dtype="fp32", std=1.0):
    return (torch.from_numpy(np.random.default_rng(seed).standard_normal(shape)).float() * std).to(DT[dtype]).to(device)


# ------------------------------------------------------------------ norms in groups
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("width,groups", [(64, 1), (160, 5), (90, 3), (70, 7), (96, 12), (640, 20), (33, 1), (4096, 2), (6144, 1), (10240, 1)])
def test_group_norm_with_and_without_a_branch(device, dtype, width, groups):
    T, ld, eps = 5, (width + 31) // 32 * 32, 1e-3
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width))
    x0, d0 = rnd((T, width), 1, device), rnd((T, width), 2, device, dtype, std=0.1)
    w, dw = rnd((width,), 3, device), rnd((width,), 4, device)
    norm = lambda a, g: oracle.grouped_norm(a, f64(g), eps, groups)
    for branch, fresh in ((False, False), (True, False), (True, True)):
        x = pad(x0).contiguous()
        if fresh:
            x.fill_(float("nan"))                      # a fresh residual must not be read
        got = ops.group_norm(x, w, eps, groups, delta=pad(d0).contiguous() if branch else None, delta_w=dw if branch else None, fresh=fresh, width=width,
                             out_dtype=DT[dtype])
        want_x = (0 if fresh else f64(x0)) + (norm(f64(d0), dw) if branch else 0)
        assert rel(x[:, :width], want_x) < 1e-6
        assert got.dtype == DT[dtype] and rel(got[:, :width], norm(want_x, w)) < TOL[dtype]
        assert bool((got[:, width:] == 0).all()) and bool((x[:, width:] == 0).all())


# ------------------------------------------------------------------ xIELU in the projection's epilogue
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 70, 200])
@pytest.mark.parametrize("n,k", [(72, 40), (256, 192)])
def test_xielu_projection(device, dtype, rows, n, k):
    p, q = 0.7, -1.3
    a, b = float(oracle.softplus(p)), 0.5 + float(oracle.softplus(q))
    x, w, bias = rnd((rows, k), 5, device, dtype), rnd((1, n, k), 6, device, "bf16", std=k ** -0.5), rnd((n,), 7, device)
    got = ops.linear(x, QuantWeight(WFormat.BF16, n, k, 1, w), bias=bias, act=ops.ACT_XIELU, act_alpha=a, act_limit=b)
    assert got.shape == (rows, n) and rel(got, oracle.xielu(f64(x) @ f64(w[0]).T + f64(bias), p, q)) < TOL[dtype]


def test_xielu_branches_meet_and_differ():
    z = np.array([-30.0, -1.0, -1e-3, 0.0, 1e-3, 1.0, 30.0])
    got = ops.ref.act_unary(ops.ACT_XIELU, torch.from_numpy(z), float(oracle.softplus(0.2)), 0.5 + float(oracle.softplus(0.9)))
    assert np.allclose(got.numpy(), oracle.xielu(z, 0.2, 0.9), rtol=1e-12, atol=1e-15)


# ------------------------------------------------------------------ query temperature
@pytest.mark.parametrize("coef,every", [(0.5, 1), (0.3, 7), (-0.4, 16), (1.25, 100)])
def test_temperature_steps_where_it_should(coef, every):
    t = query_temperature_table(3 * every + 5, coef, every).numpy()
    assert np.allclose(t, oracle.query_temperature(np.arange(len(t)), coef, every), rtol=1e-6)
    if every > 1:
        assert t[0] == 1.0 and t[every - 2] == 1.0 and t[every - 1] != 1.0      # the first step is taken at p + 1 == every


# ------------------------------------------------------------------ attention: widths, gate, temperature, pages
def paged(rng, lens, q_lens, n_q, n_kv, dk, dv, device, dtype, bs=128):
    """Random keys / values of every sequence, laid into shuffled pages; queries and gate as column ranges of one projection."""
    nb = max((l + bs - 1) // bs for l in lens) + 1
    blocks = torch.from_numpy(rng.permutation(len(lens) * nb) + 1)
    kc = torch.zeros(len(lens) * nb + 1, n_kv, bs, dk, dtype=DT[dtype])
    vc = torch.zeros(len(lens) * nb + 1, n_kv, bs, dv, dtype=DT[dtype])
    table = blocks.reshape(len(lens), nb)
    ks, vs = [], []
    for b, l in enumerate(lens):
        k, v = (torch.from_numpy(rng.standard_normal((l, n_kv, d))).float().to(DT[dtype]) for d in (dk, dv))
        for p in range(l):
            kc[table[b, p // bs], :, p % bs], vc[table[b, p // bs], :, p % bs] = k[p], v[p]
        ks.append(k)
        vs.append(v)
    y = torch.from_numpy(rng.standard_normal((sum(q_lens), n_q * dk + 8 + n_q * dv))).float().to(DT[dtype])
    cu = torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32)
    return y, kc, vc, ks, vs, table.to(torch.int32), torch.tensor(lens, dtype=torch.int32), cu


def oracle_attention(y, ks, vs, lens, q_lens, n_q, dk, dv, scale, temp):
    outs, at = [], 0
    for k, v, l, n in zip(ks, vs, lens, q_lens):
        q = np.zeros((l, n_q, dk))
        q[l - n:] = f64(y[at:at + n, :n_q * dk]).reshape(n, n_q, dk)
        q = q * temp[:l, None, None]
        o = oracle.causal_softmax_attention(q, f64(k), f64(v), scale)[l - n:].reshape(n, n_q * dv)
        outs.append(o * oracle.sigmoid(f64(y[at:at + n, n_q * dk + 8:])))
        at += n
    return np.concatenate(outs)


def run_attention(y, kc, vc, table, sl, cu, n_q, dk, scale, temp, device):
    to = lambda t: t.to(device)
    yd, lens = to(y), (cu[1:] - cu[:-1])
    T = y.shape[0]
    o = ops.attention(yd[:, :n_q * dk].view(T, n_q, dk), to(kc), to(vc), to(table), to(sl), to(cu), int(lens.max()), scale=scale,
                      q_scale=torch.from_numpy(temp).float().to(device), gate=yd[:, n_q * dk + 8:])
    return o.reshape(T, -1)


CASES = [  # n_q, n_kv, dk, dv
    (4, 1, 40, 24), (6, 3, 16, 72), (2, 2, 64, 64), (8, 2, 64, 128), (4, 2, 128, 64), (3, 1, 136, 88), (4, 4, 128, 128), (2, 1, 200, 256), (5, 5, 8, 8), (4, 1, 96, 200)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("n_q,n_kv,dk,dv", CASES)
def test_attention_widths_gate_and_temperature(device, dtype, n_q, n_kv, dk, dv):
    temp = oracle.query_temperature(np.arange(1024), 0.6, 24)
    for lens, q_lens in (([1, 130, 300], [1, 1, 1]), ([9, 129, 260], [9, 2, 37]), ([70, 128, 331], [70, 1, 150])):      # decode, short portions, prompts
        y, kc, vc, ks, vs, table, sl, cu = paged(np.random.default_rng(dk + dv), lens, q_lens, n_q, n_kv, dk, dv, device, dtype)
        got = run_attention(y, kc, vc, table, sl, cu, n_q, dk, dk ** -0.5, temp, device)
        assert rel(got, oracle_attention(y, ks, vs, lens, q_lens, n_q, dk, dv, dk ** -0.5, temp)) < (1e-2 if dtype == "bf16" else 3e-6), q_lens


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("q_lens", [[1, 1], [12, 3], [90, 80]])
def test_attention_temperature_that_changes_sign(device, q_lens):
    """1 + coef ln(.) with a negative coef passes through zero and turns negative: the scores' order turns round with it."""
    n_q, n_kv, dk, dv, lens = 2, 1, 32, 40, [150, 210]
    temp = np.linspace(1.0, -1.0, 211)
    temp[140:145] = 0.0
    y, kc, vc, ks, vs, table, sl, cu = paged(np.random.default_rng(5), lens, q_lens, n_q, n_kv, dk, dv, device, "bf16")
    got = run_attention(y, kc, vc, table, sl, cu, n_q, dk, 0.4, temp, device)
    assert rel(got, oracle_attention(y, ks, vs, lens, q_lens, n_q, dk, dv, 0.4, temp)) < 1e-2


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("n_new", [1, 2, 100])
def test_one_key_that_stands_out_is_found_anywhere(device, dtype, n_new):
    """A single key carries nearly all of the weight; wherever it lies (first token, both sides of page borders, the query's own place, far
    back) the output is its value.  The key one past the last query is given the same pull and must not be seen."""
    n_q, n_kv, dk, dv, L = 2, 1, 24, 16, 390
    for place in (0, 1, 63, 64, 127, 128, 255, 256, L - n_new, L - 1):
        y, kc, vc, ks, vs, table, sl, cu = paged(np.random.default_rng(place), [L + 1], [n_new], n_q, n_kv, dk, dv, device, dtype)
        sl = sl - 1                                                   # token L exists in its page but is not part of the sequence yet
        hot = torch.zeros(dk)
        hot[3] = 12.0
        y[:, :n_q * dk] = 0.1 * y[:, :n_q * dk]
        y[-1, :n_q * dk] = hot.repeat(n_q).to(y.dtype)                # the last query pulls on element 3 ...
        for p, v in ((place, 12.0), (L, 14.0)):                       # ... which two keys carry: `place` and the one beyond the end
            ks[0][p] = 0
            ks[0][p, :, 3] = v
            kc[table[0, p // 128].long(), :, p % 128] = ks[0][p]
        got = run_attention(y, kc, vc, table, sl, cu, n_q, dk, 0.25, np.ones(512), device)
        want = f64(vs[0][place]).repeat(n_q, 0).reshape(-1) * oracle.sigmoid(f64(y[-1, n_q * dk + 8:]))
        assert rel(got[-1], want) < 1e-2, place
        full = oracle_attention(y, [ks[0][:L]], [vs[0][:L]], [L], [n_new], n_q, dk, dv, 0.25, np.ones(512))
        assert rel(got, full) < 1e-2, place


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
def test_kv_rows_land_in_their_slots(device, dtype):
    T, n_kv, dk, dv = 7, 3, 24, 40
    y = rnd((T, 16 + n_kv * (dk + dv)), 8, device, dtype)
    kc, vc = torch.zeros(4, n_kv, 128, dk, dtype=DT[dtype], device=device), torch.zeros(4, n_kv, 128, dv, dtype=DT[dtype], device=device)
    slots = torch.tensor([128 + 127, 256, 257, -1, 384, 128, 511], dtype=torch.int64, device=device)
    k, v = y[:, 16:16 + n_kv * dk], y[:, 16 + n_kv * dk:]
    ops.kv_store(k, v, slots, kc, vc)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(kc[s // 128, :, s % 128], k[t].reshape(n_kv, dk)) and torch.equal(vc[s // 128, :, s % 128], v[t].reshape(n_kv, dv))
    assert int((kc != 0).any(-1).sum()) == 6 * n_kv and int((vc != 0).any(-1).sum()) == 6 * n_kv


# ------------------------------------------------------------------ minGRU recurrence
def mingru_case(lens, W, device, dtype, seed=0):
    y = rnd((sum(lens), 3 * W + 4), seed, device, dtype, std=1.5)
    zb, ub = rnd((W,), seed + 1, device) * 2 - 4, rnd((W,), seed + 2, device)       # slow gates: the state remembers hundreds of tokens
    return y, zb, ub


def mingru_oracle(y, zb, ub, W, state):
    S, last = oracle.mingru_recurrence(f64(y[:, :W]) + f64(zb), f64(y[:, W:2 * W]) + f64(ub), state)
    return S * oracle.silu(f64(y[:, 2 * W:3 * W])), last


def mingru_run(y, zb, ub, W, state, slots, q_lens, start):
    dev = y.device
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    cu = [0] + list(np.cumsum(q_lens))
    return ops.mingru_scan(y[:, :W], y[:, W:2 * W], y[:, 2 * W:3 * W], zb, ub, state, i32(slots), i32(cu), i32([s + n for s, n in zip(start, q_lens)]),
                           max(q_lens))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("W", [2, 40, 96, 5000])
def test_mingru_batch_of_unequal_sequences(device, dtype, W):
    lens = [1, 2, 7, 9, 300, 530] if W < 1000 else [3, 270]
    y, zb, ub = mingru_case(lens, W, device, dtype)
    state = torch.full((len(lens) + 2, W), 50.0, device=device)                      # leftovers of other requests: must not show
    slots = np.random.default_rng(1).permutation(len(lens) + 2)[:len(lens)].tolist()
    got = mingru_run(y, zb, ub, W, state, slots, lens, [0] * len(lens))
    at = 0
    for n, s in zip(lens, slots):
        want, last = mingru_oracle(y[at:at + n], zb, ub, W, np.zeros(W))
        assert rel(got[at:at + n], want) < (8e-3 if dtype == "bf16" else 2e-6)
        assert rel(state[s], last) < 2e-6
        at += n
    untouched = set(range(len(lens) + 2)) - set(slots)
    assert all(bool((state[s] == 50.0).all()) for s in untouched)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("sizes", [[1] * 40, [2, 3, 5, 1, 29], [37, 3], [8, 8, 8, 16], [300, 2, 258, 40]])
def test_mingru_state_carries_across_portions(device, sizes):
    W, n = 24, sum(sizes)
    y, zb, ub = mingru_case([n], W, device, "fp32", seed=7)
    want, last = mingru_oracle(y, zb, ub, W, np.zeros(W))
    state, at, outs = torch.full((3, W), 9.0, device=device), 0, []
    for k in sizes:
        outs.append(mingru_run(y[at:at + k], zb, ub, W, state, [1], [k], [at]))
        at += k
    assert rel(torch.cat(outs), want) < 2e-6 and rel(state[1], last) < 2e-6


@pytest.mark.parametrize("device", DEVICES)
def test_mingru_candidate_switches_at_zero(device):
    """u just below, at and just above zero, with the gate open: the candidate is sigmoid(u) or u + 1/2."""
    W = 8
    u = torch.tensor([-5.0, -1e-3, -0.0, 0.0, 1e-3, 5.0, -0.5, 0.5], device=device)
    y = torch.cat([torch.full((W,), 40.0, device=device), u, torch.full((W,), 3.0, device=device)]).reshape(1, -1).contiguous()
    zero, state = torch.zeros(W, device=device), torch.zeros(1, W, device=device)
    mingru_run(y, zero, zero, W, state, [0], [1], [0])
    un = u.cpu().double().numpy()
    assert np.allclose(state[0].cpu().numpy(), np.where(un >= 0, un + 0.5, oracle.sigmoid(un)), rtol=1e-6)
