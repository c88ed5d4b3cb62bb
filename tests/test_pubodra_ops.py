"""The mechanisms of Pubodra one by one, as the operators the graph calls, against the plain restatement in pubodra_oracle.py; on a GPU these are
the sm_100a kernels, on the CPU their PyTorch twins."""
import math

import numpy as np
import pytest
import torch

import pubodra_oracle as oracle
from design_util import DEVICES
from machx_inference_engine_b200 import ops
from machx_inference_engine_b200.models.transformer import UnaryMoEFFN
from machx_inference_engine_b200.ops import QuantWeight, WFormat
from machx_inference_engine_b200.parallel.comm import ParallelCtx
from machx_inference_engine_b200.utils.rope import rope_tables

DT = {"bf16": torch.bfloat16, "fp32": torch.float32}
TOL = {"bf16": 8e-3, "fp32": 2e-6}


def f64(t):
    return t.detach().double().cpu().numpy()


def rel(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.linalg.norm(f64(got) - want) / (np.linalg.norm(want) + 1e-30))


def rnd(shape, seed, device, dtype="fp32", std=1.0):
    return (torch.from_numpy(np.asarray(np.random.default_rng(seed).standard_normal(shape))).float() * std).to(DT[dtype]).to(device)


def weight(n, k, seed, device, e=1, std=None):
    return QuantWeight(WFormat.BF16, n, k, e, rnd((e, n, k), seed, device, "bf16", std=std or k ** -0.5))


# ------------------------------------------------------------------ dynamic tanh in the place of a norm
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("width,rows", [(64, 1), (50, 7), (4096, 3), (260, 33)])
def test_dyt_norm_adds_branch_and_vector(device, dtype, width, rows):
    ld, alpha = (width + 31) // 32 * 32, 0.83
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width)).contiguous()
    x0, d0, st = rnd((rows, width), 1, device, std=2.0), rnd((rows, width), 2, device, dtype), rnd((width,), 3, device)
    w, b = rnd((width,), 4, device), rnd((width,), 5, device)
    for delta, step in ((None, None), (d0, None), (None, st), (d0, st)):
        x = pad(x0)
        got = ops.dyt_norm(x, alpha, pad(w), pad(b), delta=None if delta is None else pad(delta), step=None if step is None else pad(step), out_dtype=DT[dtype])
        want = f64(x0) + (0 if delta is None else f64(delta)) + (0 if step is None else f64(step))
        assert rel(x[:, :width], want) < 1e-6
        assert got.dtype == DT[dtype] and rel(got[:, :width], oracle.dynamic_tanh(want, alpha, f64(w), f64(b))) < TOL[dtype]
        assert bool((got[:, width:] == 0).all()) and bool((x[:, width:] == 0).all())


@pytest.mark.parametrize("device", DEVICES)
def test_dyt_norm_saturates_and_keeps_small_values(device):
    x = torch.tensor([[-1e4, -20.0, -1e-4, 0.0, 1e-4, 0.5, 20.0, 1e4]], device=device)
    one, zero = torch.ones(8, device=device), torch.zeros(8, device=device)
    got = ops.dyt_norm(x.clone(), 2.0, one, zero, out_dtype=torch.float32)
    assert np.allclose(f64(got), np.tanh(2.0 * f64(x)), rtol=1e-6, atol=0)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
def test_dyt_norm_forms_the_expert_sum(dtype):
    from machx_inference_engine_b200.ops.cuda import CombineDelta
    T, K, ld, dev = 9, 3, 96, "cuda:0"
    y, w = rnd((40, ld), 1, dev, dtype), rnd((T, K), 2, dev)
    pos = torch.from_numpy(np.random.default_rng(3).permutation(40)[:T * K]).to(torch.int32).to(dev)
    x, step = rnd((T, ld), 4, dev), rnd((ld,), 5, dev)
    g, b = rnd((ld,), 6, dev), rnd((ld,), 7, dev)
    want = f64(x) + f64(step) + (f64(w)[..., None] * f64(y)[f64(pos).astype(int)].reshape(T, K, ld)).sum(1)
    d = CombineDelta(y, pos, w)
    assert rel(d.materialize(), want - f64(x) - f64(step)) < 1e-6
    rows = torch.tensor([7, 2], device=dev)
    assert torch.equal(d.rows(rows).materialize(), d.materialize()[rows])
    got = ops.dyt_norm(x, 0.5, g, b, delta=d, step=step, out_dtype=DT[dtype])
    assert rel(x, want) < 1e-6 and rel(got, oracle.dynamic_tanh(want, 0.5, f64(g), f64(b))) < TOL[dtype]


# ------------------------------------------------------------------ activations in the projections
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 70, 200])
@pytest.mark.parametrize("act,fn", [(ops.ACT_GELU_TANH, oracle.gelu_tanh), (ops.ACT_RELU2, oracle.squared_relu)])
def test_projection_with_activation(device, dtype, rows, act, fn):
    for n, k in ((72, 40), (256, 192)):
        x, w = rnd((rows, k), 5, device, dtype, std=2.0), weight(n, k, 6, device)
        got = ops.linear(x, w, act=act)
        assert got.shape == (rows, n) and rel(got, fn(f64(x) @ f64(w.p0[0]).T)) < TOL[dtype]


# ------------------------------------------------------------------ rotation
ROTS = [({"base": 1e4, "dims": 8}, None), ({"base": 5e5, "dims": 64}, (16.0, 1024, 32.0, 1.0)), ({"base": 1e4, "dims": 32}, (4.0, 200, 16.0, 2.0)),
        ({"base": 100.0, "dims": 6}, (1.0, 64, 32.0, 1.0)), ({"base": 3e4, "dims": 48}, (0.5, 300, 8.0, 0.5)), ({"base": 3.1e5, "dims": 20}, (9.0, 12, 64.0, 24.0)),
        ({"base": 1e4, "dims": 4}, (40.0, 4096, 1.0, 1.0)), ({"base": 1e4, "dims": 2}, (2.0, 128, 32.0, 1.0))]


def tables(rot, yarn, n, device):
    f, orig, fast, slow = yarn or (1.0, 0, 32.0, 1.0)
    return rope_tables(n, rot["dims"], rot["base"], scaling_type="yarn" if yarn else "none", scaling_factor=f, orig_ctx=orig, beta_fast=fast, beta_slow=slow,
                       device=device)


def with_scaling(rot, yarn):
    return {**rot, **({"scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))} if yarn else {})}


@pytest.mark.parametrize("rot,yarn", ROTS)
def test_rotation_tables(rot, yarn):
    f, mag = oracle.frequencies(rot["dims"], rot["base"], with_scaling(rot, yarn).get("scaling"))
    c, s = tables(rot, yarn, 700, "cpu")
    a = np.arange(700)[:, None] * f
    assert np.abs(c.numpy() - np.cos(a) * mag).max() < 1e-6 and np.abs(s.numpy() - np.sin(a) * mag).max() < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("H,rank,rot_dim", [(1, 8, 8), (5, 40, 6), (16, 512, 64), (3, 20, 10), (8, 100, 2)])
def test_head_epilogue_norms_rotates_and_stores(device, dtype, H, rank, rot_dim):
    """Strided inputs, padded widths, slots in any order and one that is not stored; rotation in place and into another tensor."""
    T, eps, d = 7, 1e-3, 16
    R, r = (rank + 7) // 8 * 8, (rot_dim + 7) // 8 * 8
    rot, yarn = {"base": 1000.0, "dims": rot_dim}, (4.0, 40, 8.0, 1.0)
    cos, sin = tables(rot, yarn, 64, device)
    y = rnd((T, H * (d + r) + R + r + 8), 1, device, dtype)
    q, ckv = y[:, :H * (d + r)].view(T, H, d + r), y[:, H * (d + r):H * (d + r) + R + r]
    q[..., d + rot_dim:] = 0
    ckv[:, rank:R] = 0
    ckv[:, R + rot_dim:] = 0
    w = torch.zeros(R, device=device)
    w[:rank] = rnd((rank,), 2, device) + 1
    pos = torch.tensor([0, 1, 2, 63, 30, 5, 9], dtype=torch.int32, device=device)
    slots = torch.tensor([128 + 127, 256, 257, -1, 384, 128, 511], dtype=torch.int64, device=device)
    full = with_scaling(rot, yarn)
    p = f64(pos)
    want_q = oracle.rotate_pairs(f64(q)[..., d:d + rot_dim], p, full)
    x = f64(ckv)
    want_row = np.concatenate([oracle.rms_norm(x[:, :rank], f64(w)[:rank], eps), oracle.rotate_pairs(x[:, R:R + rot_dim], p, full)], axis=1)
    for inplace in (False, True):
        cache = torch.zeros(4, 1, 128, R + r, dtype=DT[dtype], device=device)
        out = q[..., d:] if inplace else torch.full((T, H, R + r), 7.0, dtype=DT[dtype], device=device)[..., R:]
        ops.latent_post(q[..., d:], ckv, w, rank, eps, pos, cos, sin, slots, cache, out)
        assert rel(out[..., :rot_dim], want_q) < TOL[dtype] and bool((out[..., rot_dim:] == 0).all())
        for t, s in enumerate(slots.tolist()):
            if s >= 0:
                row = cache[s // 128, 0, s % 128]
                assert rel(torch.cat([row[:rank], row[R:R + rot_dim]]), want_row[t]) < TOL[dtype]
                assert bool((row[rank:R] == 0).all()) and bool((row[R + rot_dim:] == 0).all())
        assert int((cache != 0).any(-1).sum()) == 6


# ------------------------------------------------------------------ per-head products
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("H,N,K", [(3, 24, 40), (8, 512, 128), (5, 128, 512), (1, 8, 8), (2, 72, 200)])
def test_every_head_its_own_matrix(device, dtype, H, N, K):
    for T in (1, 2, 5, 8, 9, 20, 130):
        buf = rnd((T, H, K + 16), T, device, dtype)
        x, w = buf[..., 8:8 + K], weight(N, K, 3, device, e=H)
        gates = rnd((T, H * N + 8), 4, device, dtype)[:, 8:]
        want = np.einsum("thk,hnk->thn", f64(x), f64(w.p0))
        assert rel(ops.head_linear(x, w), want) < TOL[dtype]
        out = torch.full((T, H, N + 8), 3.0, dtype=DT[dtype], device=device)
        ops.head_linear(x, w, gate=gates, out=out[..., :N])
        assert rel(out[..., :N], want * oracle.sigmoid(f64(gates)).reshape(T, H, N)) < TOL[dtype]
        assert bool((out[..., N:] == 3.0).all())


# ------------------------------------------------------------------ attention over latent pages
def paged_latents(rng, lens, width, dtype, bs=128):
    """Random cache rows of every sequence in shuffled pages; rows that belong to nobody hold large numbers."""
    nb = max((l + bs - 1) // bs for l in lens) + 1
    table = torch.from_numpy(rng.permutation(len(lens) * nb) + 1).reshape(len(lens), nb)
    cache = torch.full((len(lens) * nb + 1, 1, bs, width), 30.0, dtype=DT[dtype])
    rows = []
    for b, l in enumerate(lens):
        c = torch.from_numpy(rng.standard_normal((l, width))).float().to(DT[dtype])
        for p in range(l):
            cache[table[b, p // bs], 0, p % bs] = c[p]
        rows.append(c)
    return cache, rows, table.to(torch.int32)


def batch_of(lens, q_lens, device):
    cu = torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32)
    return torch.tensor(lens, dtype=torch.int32, device=device), cu.to(device)


def latent_space_oracle(q, rows, lens, q_lens, rank, scale, window):
    """Heads whose key and value matrices are the identity: keys are the cached rows, values their first part."""
    H, outs, at = q.shape[1], [], 0
    eye = np.stack([np.eye(rank)] * H)
    for c, l, n in zip(rows, lens, q_lens):
        r = f64(c)
        outs.append(oracle.latent_heads(q[at:at + n], r[:, :rank], r[:, rank:], eye, eye, scale, window, first_query=l - n))
        at += n
    return np.concatenate(outs)


SHAPES = [(4, 512, 128), (1, 8, 8), (5, 40, 8), (9, 64, 24), (3, 192, 72), (16, 512, 64), (40, 256, 32), (64, 128, 64), (7, 136, 24)]
BATCHES = [([1, 130, 300, 257], [1, 1, 1, 1]), ([9, 129, 260], [9, 2, 37]), ([1], [1]), ([40, 400], [40, 1])]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("H,rank,rot", SHAPES)
def test_latent_attention(device, dtype, H, rank, rot):
    for window in (0, 1, 60, 128, 129, 1000):
        lens, q_lens = BATCHES[window % len(BATCHES)] if device == "cpu" else (None, None)
        for lens, q_lens in ([(lens, q_lens)] if lens else BATCHES):
            cache, rows, table = paged_latents(np.random.default_rng(rank + window), lens, rank + rot, dtype)
            sl, cu = batch_of(lens, q_lens, device)
            q = rnd((sum(q_lens), H, rank + rot), 2, device, dtype)
            scale = 2.0 / math.sqrt(rank + rot)
            got = ops.latent_attention(q, cache.to(device), table.to(device), sl, cu, max(q_lens), rank, window=window, scale=scale)
            assert rel(got, latent_space_oracle(f64(q), rows, lens, q_lens, rank, scale, window)) < (1e-2 if dtype == "bf16" else 3e-6), (window, q_lens)


@pytest.mark.gpu
@pytest.mark.parametrize("n_splits", [1, 2, 3, 8])
@pytest.mark.parametrize("H,rank,rot", [(32, 512, 64), (9, 64, 24), (48, 128, 64)])
def test_latent_attention_ranges(n_splits, H, rank, rot):
    """Any cut of the keys into ranges, more ranges than pages included, gives the same result."""
    from machx_inference_engine_b200.ops import cuda as K
    lens, q_lens = [1, 700, 129, 384, 1000], [1, 1, 1, 1, 1]
    cache, rows, table = paged_latents(np.random.default_rng(1), lens, rank + rot, "bf16")
    sl, cu = batch_of(lens, q_lens, "cuda:0")
    q = rnd((5, H, rank + rot), 2, "cuda:0", "bf16")
    for window in (0, 300):
        got = K.latent_attention(q, cache.cuda(), table.cuda(), sl, cu, 1, rank, window=window, scale=0.1, n_splits=n_splits)
        assert rel(got, latent_space_oracle(f64(q), rows, lens, q_lens, rank, 0.1, window)) < 1e-2, window


@pytest.mark.gpu
def test_latent_attention_scores_that_grow():
    """Keys sorted so that the maximum rises from tile to tile: the accumulator is rescaled again and again."""
    H, rank, rot, L = 16, 128, 64, 900
    cache, rows, table = paged_latents(np.random.default_rng(3), [L], rank + rot, "bf16")
    q = rnd((1, H, rank + rot), 4, "cuda:0", "bf16")
    ramp = torch.linspace(0.1, 6.0, L).reshape(-1, 1) * q[0, 0].float().cpu().sign()
    rows[0] = (rows[0].float() * 0.3 + ramp * 0.3).to(torch.bfloat16)
    for p in range(L):
        cache[table[0, p // 128].long(), 0, p % 128] = rows[0][p]
    sl, cu = batch_of([L], [1], "cuda:0")
    from machx_inference_engine_b200.ops import cuda as K
    for n_splits in (1, 4):
        got = K.latent_attention(q, cache.cuda(), table.cuda(), sl, cu, 1, rank, scale=1.0, n_splits=n_splits)
        assert rel(got, latent_space_oracle(f64(q), rows, [L], [1], rank, 1.0, 0)) < 1e-2


EXPANDED = [(3, 24, 8, 40, 40), (2, 64, 24, 64, 80), (4, 40, 64, 128, 192), (2, 56, 8, 200, 24), (3, 104, 16, 56, 72), (2, 128, 64, 128, 512), (1, 96, 24, 232, 136),
            (2, 160, 32, 48, 64), (2, 192, 64, 128, 128), (1, 136, 8, 256, 40)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,dim,rot,vdim,rank", EXPANDED)
def test_expanded_attention(device, H, dim, rot, vdim, rank):
    """Per-head keys and values formed from the pages, gate included; long and short segments, some queries left out of the call."""
    wkv = weight(H * (dim + vdim), rank, 5, device)
    uk, uv = f64(wkv.p0[0])[:H * dim].reshape(H, dim, rank), f64(wkv.p0[0])[H * dim:].reshape(H, vdim, rank)
    for window, lens, q_lens in ((0, [70, 300], [70, 150]), (100, [330, 65, 128], [200, 65, 1]), (1, [90], [90]), (129, [400, 260], [128, 260]), (128, [389], [130])):
        cache, rows, table = paged_latents(np.random.default_rng(rank + window), lens, rank + rot, "bf16")
        sl, cu = batch_of(lens, q_lens, device)
        skip = 3
        y = rnd((skip + sum(q_lens), H * (dim + rot) + 16), 2, device, "bf16")
        q = y[:, 8:8 + H * (dim + rot)].view(-1, H, dim + rot)
        gate = rnd((skip + sum(q_lens), H * vdim), 3, device, "bf16")
        out = torch.full((skip + sum(q_lens), H, vdim), 9.0, dtype=torch.bfloat16, device=device)
        scale = 1.5 / math.sqrt(dim + rot)
        plans = {}
        for _ in range(2):                           # the second call finds the page list of the first
            ops.latent_attention_expanded(q, wkv, cache.to(device), table.to(device), sl, cu + skip, max(q_lens), dim, vdim, rank, window=window, scale=scale,
                                          gate=gate, out=out, plans=plans)
        at, qn, gn = skip, f64(q), oracle.sigmoid(f64(gate)).reshape(-1, H, vdim)
        assert bool((out[:skip] == 9.0).all())
        for c, l, n in zip(rows, lens, q_lens):
            r = f64(c)
            want = oracle.latent_heads(qn[at:at + n], r[:, :rank], r[:, rank:], uk, uv, scale, window, first_query=l - n) * gn[at:at + n]
            assert rel(out[at:at + n], want) < 1.2e-2, (window, l, n)
            at += n


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("form", ["latent", "latent-fp32", "expanded"])
@pytest.mark.parametrize("window", [40, 128, 130, 257])
def test_one_key_that_stands_out_at_the_window_edge(device, form, window):
    """One key carries nearly all of the weight of the last query while it lies in the window -- down to its last place -- and none when it lies one
    token further back; a key beyond the sequence, with an even stronger pull, is never seen."""
    H, dim, rank, rot, vdim, L = 2, 24, 24, 8, 16, 390
    dtype = "fp32" if form == "latent-fp32" else "bf16"
    n = 70 if form == "expanded" else 2
    for gap in (0, 1, window - 2, window - 1, window, window + 1):
        place = L - 1 - gap
        cache, rows, table = paged_latents(np.random.default_rng(gap), [L + 1], rank + rot, dtype)
        rows[0] = rows[0] * 0.1
        for p, v in ((place, 12.0), (L, 20.0)):
            rows[0][p] = 0
            rows[0][p, 3] = v
            rows[0][p, 5] = 4.0
        for p in range(L + 1):
            cache[table[0, p // 128].long(), 0, p % 128] = rows[0][p]
        sl, cu = batch_of([L], [n], device)
        eye = np.stack([np.eye(rank)] * H)
        if form == "expanded":
            q = rnd((n, H, dim + rot), 6, device, dtype, std=0.1)
            q[-1] = 0
            q[-1, :, 3] = 8.0
            uk, uv = eye, eye[:, :vdim]
            wkv = QuantWeight(WFormat.BF16, H * (dim + vdim), rank, 1, torch.from_numpy(np.concatenate([uk.reshape(-1, rank), uv.reshape(-1, rank)])[None])
                              .to(torch.bfloat16).to(device))
            got = ops.latent_attention_expanded(q, wkv, cache.to(device), table.to(device), sl, cu, n, dim, vdim, rank, window=window, scale=0.25)
        else:
            q = rnd((n, H, rank + rot), 6, device, dtype, std=0.1)
            q[-1] = 0
            q[-1, :, 3] = 8.0
            uk = uv = eye
            got = ops.latent_attention(q, cache.to(device), table.to(device), sl, cu, n, rank, window=window, scale=0.25)
        r = f64(rows[0][:L])
        want = oracle.latent_heads(f64(q), r[:, :rank], r[:, rank:], uk, uv, 0.25, window, first_query=L - n)
        assert rel(got, want) < 1.2e-2, gap
        assert abs(float(got[-1, 0, 5]) - 4.0) < 0.05 if gap < window else abs(float(got[-1, 0, 5])) < 0.5, gap


# ------------------------------------------------------------------ experts
class _Given:
    """A weight source over a dict of arrays."""

    def __init__(self, W, device):
        self.W, self.device = W, device

    def matrix(self, name, N, K, E=1):
        a = np.stack([self.W[name.replace("*", str(e))] for e in range(E)]) if "*" in name else self.W[name][None]
        assert a.shape == (E, N, K)
        return QuantWeight(WFormat.BF16, N, K, E, torch.from_numpy(a).to(torch.bfloat16).to(self.device).contiguous())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
@pytest.mark.parametrize("experts,top,ff,width", [(6, 2, 40, 64), (11, 3, 72, 90), (3, 3, 32, 32), (5, 1, 100, 72), (64, 6, 96, 128)])
def test_experts(device, dtype, experts, top, ff, width):
    layer = oracle.latent_layer(1, 8, 8, 8, 8, 8, (experts, top, ff))
    W = oracle.random_weights(oracle.random_config([layer], width=width), seed=experts)
    row = (width + 31) // 32 * 32
    moe = UnaryMoEFFN(_Given(W, device), "l0.mlp", width, row, experts, top, ff, ops.ACT_RELU2)
    for T in (1, 3, 8, 9, 50, 300):
        h = torch.zeros(T, row, dtype=DT[dtype], device=device)
        h[:, :width] = rnd((T, width), T, device, dtype)
        x = f64(h)[:, :width]
        # a token whose choice of experts is within rounding of another says nothing: leave such tokens out
        z = np.sort(x @ np.float64(W["l0.mlp.router"]).T, axis=-1)[:, ::-1]
        clear = z[:, top - 1] - z[:, top] > 1e-4 if top < experts else np.ones(T, bool)
        got = moe(h, ParallelCtx())
        got = got if isinstance(got, torch.Tensor) else got.materialize()
        want = oracle.moe_mlp({n: np.float64(a) for n, a in W.items()}, "l0.mlp", layer["mlp"], x)
        assert clear.mean() > 0.9 and rel(got[:, :width][torch.from_numpy(clear)], want[clear]) < (1e-2 if dtype == "bf16" else 3e-6), T
        assert bool((got[:, width:] == 0).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("precise", [False, True])
def test_routing_weights(device, precise):
    z = rnd((40, 70), 3, device, std=4.0)
    idx, w = ops.moe_route(z, None, 5, True, precise=precise)
    want_idx, want_w = oracle.route(f64(z), 5)
    assert np.array_equal(f64(idx).astype(int), want_idx) and rel(w, want_w) < (3e-7 if precise else 3e-6)
