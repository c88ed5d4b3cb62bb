"""Plain PyTorch fp32 twins of every kernel in ``csrc/cuda`` (same signatures as ``ops.cuda``).

They are the numerical oracle of the GPU tests and the execution path on machines without a
GPU (CPU plumbing runs, gloo multi-process tests).  Shapes, layouts (paged KV, 16-row gate/up
interleave, packed MoE rows) and rounding points (bf16 activations) mirror the kernels.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from .weights import QuantWeight

ACT_NONE, ACT_SWIGLU, ACT_SWIGLU_OAI, ACT_GEGLU, ACT_XIELU, ACT_GELU_TANH, ACT_RELU2, ACT_TANH = 0, 1, 2, 3, 4, 5, 6, 7


def act_gated(act: int) -> bool:
    """Gated activations combine 16-row interleaved gate / up columns (N columns become N / 2); the others are element-wise."""
    return act in (ACT_SWIGLU, ACT_SWIGLU_OAI, ACT_GEGLU)


MOE_TILE = 128


# Matmul dtype of this module.  fp32 = the numerical oracle of the tests.  The library-baseline arm of the benchmarks (plain PyTorch
# = cuBLAS GEMMs + NCCL on the same model, no kernel of this engine) switches it to bf16 so that its GEMMs run on the tensor cores.
_MM_DTYPE = torch.float32
_DENSE_BUDGET = [None]          # bytes of decoded weights that may stay resident (None = unlimited); what does not fit is decoded per call


def set_matmul_dtype(dtype, dense_budget_bytes=None) -> None:
    global _MM_DTYPE
    _MM_DTYPE = dtype
    _DENSE_BUDGET[0] = dense_budget_bytes


def _mm(a: torch.Tensor, b_t: torch.Tensor) -> torch.Tensor:
    """a [M,K] @ b_t [N,K]^T in the module's matmul dtype, fp32 result."""
    if _MM_DTYPE == torch.float32:
        return a.to(torch.float32) @ b_t.to(torch.float32).t()
    return (a.to(_MM_DTYPE) @ b_t.to(_MM_DTYPE).t()).to(torch.float32)


class _LazyBank:
    """Expert bank decoded one expert at a time (and kept while the residency budget lasts)."""

    def __init__(self, w: QuantWeight):
        self.w, self.cache = w, {}

    def __getitem__(self, e):
        if isinstance(e, torch.Tensor):
            return torch.stack([self[int(i)] for i in e.tolist()])
        d = self.cache.get(e)
        if d is None:
            d = self.w.slice_experts(e, e + 1).dequantize(_MM_DTYPE)[0]
            nbytes = d.numel() * d.element_size()
            if _DENSE_BUDGET[0] is None or _DENSE_BUDGET[0] >= nbytes:
                self.cache[e] = d
                if _DENSE_BUDGET[0] is not None:
                    _DENSE_BUDGET[0] -= nbytes
        return d


def _dense(w: QuantWeight):
    if w._dense_cache is None:
        if _DENSE_BUDGET[0] is not None and w.E > 1:
            w._dense_cache = _LazyBank(w)
        else:
            w._dense_cache = w.dequantize(_MM_DTYPE)
            if _DENSE_BUDGET[0] is not None:
                _DENSE_BUDGET[0] -= w._dense_cache.numel() * w._dense_cache.element_size()
    return w._dense_cache


def embed(w: QuantWeight, ids: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    tbl = _dense(w)[0]
    return tbl[ids.long().clamp(0, w.N - 1)].to(torch.float32) * scale


def rmsnorm(x, w, eps, delta=None, dbias=None, one_plus_w=False, delta_scale=1.0, write_x=True, want_out=True):
    if delta is not None:
        d = delta.to(torch.float32)
        if dbias is not None:
            d = d + dbias
        xs = x + d * delta_scale
        if write_x:
            x.copy_(xs)
    else:
        xs = x
    if not want_out:
        return None
    g = (1.0 + w) if one_plus_w else w
    inv = torch.rsqrt(xs.pow(2).mean(dim=-1, keepdim=True) + eps)
    return (xs * inv * g).to(torch.bfloat16)


def act_unary(act, z, a, b):
    """xIELU: a z^2 + z / 2 above zero, b (e^z - 1 - z) + z / 2 below (a = softplus(p), b = 1/2 + softplus(q)); GELU in its tanh form; the
    square of ReLU; tanh."""
    if act == ACT_TANH:
        return torch.tanh(z)
    if act == ACT_GELU_TANH:
        return torch.nn.functional.gelu(z, approximate="tanh")
    if act == ACT_RELU2:
        return z.clamp(min=0.0).square()
    if act != ACT_XIELU:
        return z
    neg = z.clamp(max=0.0)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(neg) - neg)) + 0.5 * z


def _act(act, g, u, alpha, limit):
    if act == ACT_SWIGLU:
        return torch.nn.functional.silu(g) * u
    if act == ACT_SWIGLU_OAI:
        g = g.clamp(max=limit)
        u = u.clamp(-limit, limit)
        return g * torch.sigmoid(alpha * g) * (u + 1.0)
    return torch.nn.functional.gelu(g, approximate="tanh") * u


def _epilogue_act(y, act, alpha, limit):
    """A projection's activation: gate and up columns combined, or element by element."""
    if act_gated(act):
        g, u = _deinterleave16(y)
        return _act(act, g, u, alpha, limit)
    return y if act == ACT_NONE else act_unary(act, y, alpha, limit)


def _deinterleave16(y: torch.Tensor):
    """[..., 2F] with 16-wide interleaved gate|up groups -> (gate [...,F], up [...,F])."""
    F2 = y.shape[-1]
    v = y.reshape(*y.shape[:-1], F2 // 32, 2, 16)
    return v[..., 0, :].reshape(*y.shape[:-1], F2 // 2), v[..., 1, :].reshape(*y.shape[:-1], F2 // 2)


def glu(x, act, alpha=1.702, limit=7.0):
    g, u = _deinterleave16(x.to(torch.float32))
    return _act(act, g, u, alpha, limit).to(torch.float32 if x.dtype == torch.float32 else torch.bfloat16)


def linear(x, w: QuantWeight, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, out_f32=False, row_scale=None, out=None):
    if out is not None:
        return out.copy_(linear(x, w, bias, act, act_alpha, act_limit, out_f32, row_scale))
    y = _mm(x, _dense(w)[0])
    if bias is not None:
        y = y + bias
    y = _epilogue_act(y, act, act_alpha, act_limit)
    if row_scale is not None:
        y = y * row_scale.unsqueeze(-1)
    return y if (out_f32 or x.dtype == torch.float32) else y.to(torch.bfloat16)      # fp32 activations: the layer runs in fp32 throughout


def hadamard128(x, pre=None, post=None, bias=None, out_f32=False, out=None):
    """``had128(x * pre) * post + bias`` over every aligned run of 128 elements of the rows (EXL3 layers; src/ops/hadamard.cpp:36)."""
    from ..formats.exl3 import hadamard128 as _had
    v = x.to(torch.float32)
    if pre is not None:
        v = v * pre
    v = _had(v)
    if post is not None:
        v = v * post
    if bias is not None:
        v = v + bias
    v = v if out_f32 else v.to(torch.bfloat16)
    return v if out is None else out.copy_(v)


def grouped_linear(xp, w: QuantWeight, tile_expert, num_tiles, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, out_f32=False, bn=128,
                   out_dtype=None):
    """xp: packed rows [P,K]; tile t (rows 128t..128t+127) uses expert tile_expert[t] for t < num_tiles[0]."""
    W = _dense(w)
    P = xp.shape[0]
    n_out = w.N // 2 if act_gated(act) else w.N
    out = torch.zeros(P, n_out, dtype=torch.float32, device=xp.device)
    nt = int(num_tiles[0])
    te = tile_expert[:nt].tolist()
    for t, e in enumerate(te):
        rows = slice(t * MOE_TILE, min((t + 1) * MOE_TILE, P))
        y = _mm(xp[rows], W[e])
        if bias is not None:
            y = y + bias[e]
        y = _epilogue_act(y, act, act_alpha, act_limit)
        out[rows] = y
    return out.to(out_dtype) if out_dtype is not None else (out if (out_f32 or xp.dtype == torch.float32) else out.to(torch.bfloat16))


def expert_gemv(x, w: QuantWeight, slot_expert, x_div=1, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, slot_scale=None, out_f32=False,
                e_lo=0):
    """y[s] = W[slot_expert[s] - e_lo] @ x[s // x_div]; slots whose expert lies outside [e_lo, e_lo + E) give zero rows."""
    W = _dense(w)
    S = slot_expert.numel()
    rows = torch.arange(S, device=x.device) // x_div
    xe = x.to(torch.float32)[rows]
    se = slot_expert.long() - e_lo
    owned = (se >= 0) & (se < w.E)
    se = se.clamp(0, w.E - 1)
    y = torch.einsum("sk,snk->sn", xe.to(_MM_DTYPE), W[se]).to(torch.float32)
    if bias is not None:
        y = y + bias[se]
    y = _epilogue_act(y, act, act_alpha, act_limit)
    y = y * owned.unsqueeze(-1)
    if slot_scale is not None:
        y = y * slot_scale.unsqueeze(-1)
    return y if (out_f32 or x.dtype == torch.float32) else y.to(torch.bfloat16)


def qkv_post(qkv, bias, q_norm_w, k_norm_w, positions, rope_cos, rope_sin, slot_map, k_cache, v_cache, n_q, n_kv, hd, n_rot,
             q_gate=False, norm_one_plus_w=False, eps=1e-6, kv_scales=None, v_norm=False):
    """Returns (q [T,n_q,hd] bf16, gate or None); writes K/V into the paged cache (int8 rows + scales when kv_scales is given)."""
    T = qkv.shape[0]
    x = qkv.to(torch.float32)
    if bias is not None:
        x = x + bias
    q_stride = 2 * hd if q_gate else hd
    qc = n_q * q_stride
    qpart = x[:, :qc].reshape(T, n_q, q_stride)
    gate = None
    if q_gate:
        gate = qpart[..., hd:].to(torch.bfloat16).contiguous()
        qpart = qpart[..., :hd]
    k = x[:, qc:qc + n_kv * hd].reshape(T, n_kv, hd)
    v = x[:, qc + n_kv * hd:].reshape(T, n_kv, hd)

    def norm(t, w):
        if w is None:
            return t
        g = (1.0 + w) if norm_one_plus_w else w
        return t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * g

    qpart, k = norm(qpart, q_norm_w), norm(k, k_norm_w)
    if v_norm:
        v = v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)
    if n_rot > 0:
        half = n_rot // 2
        pos = positions.long().clamp(0, rope_cos.shape[0] - 1)
        c, s = rope_cos[pos].unsqueeze(1), rope_sin[pos].unsqueeze(1)

        def rope(t):
            a, b = t[..., :half], t[..., half:n_rot]
            return torch.cat([a * c - b * s, a * s + b * c, t[..., n_rot:]], dim=-1)

        qpart, k = rope(qpart), rope(k)
    if n_kv == 0:                   # queries only (a draft head that reads another model's cache)
        return qpart.to(torch.bfloat16).contiguous(), gate
    bs = k_cache.shape[2]
    ok = slot_map >= 0
    blk, off = (slot_map[ok] // bs).long(), (slot_map[ok] % bs).long()
    if kv_scales is not None:
        for cache, sc, t in ((k_cache, kv_scales[0], k[ok]), (v_cache, kv_scales[1], v[ok])):
            amax = t.abs().amax(-1)
            scale = torch.where(amax > 0, amax / 127.0, torch.ones_like(amax))
            cache[blk, :, off] = torch.round(t * (1.0 / scale).unsqueeze(-1)).clamp(-127, 127).to(torch.int8)
            sc[blk, :, off] = scale
        return qpart.to(torch.bfloat16).contiguous(), gate
    k_cache[blk, :, off] = k[ok].to(k_cache.dtype)
    v_cache[blk, :, off] = v[ok].to(v_cache.dtype)
    return qpart.to(torch.bfloat16).contiguous(), gate


def group_norm(x, w, eps, groups=1, delta=None, delta_w=None, fresh=False, width=None, out_dtype=torch.bfloat16, want_out=True):
    """RMSNorm over ``groups`` equal parts of a row.  With ``delta``: x <- (0 if fresh else x) + norm(delta) * delta_w, in place; returns
    norm(x) * w.  Rows are padded to x.shape[1] columns; the first ``width`` (default: all) are the row, the padding stays zero."""
    H = x.shape[1] if width is None else width

    def norm(t, g):
        p = t[:, :H].to(torch.float32).reshape(t.shape[0], groups, H // groups)
        return (p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)).reshape(-1, H) * g

    if delta is not None:
        d = norm(delta, delta_w)
        if fresh:
            x.zero_()
        x[:, :H] += d
    if not want_out:
        return None
    out = torch.zeros(x.shape, dtype=out_dtype, device=x.device)
    out[:, :H] = norm(x, w).to(out_dtype)
    return out


def dyt_norm(x, alpha, w, b, delta=None, step=None, out_dtype=torch.bfloat16, want_out=True):
    """x <- x + delta + step (fp32, in place; step is one vector for all rows); returns tanh(alpha x) w + b."""
    if delta is not None:
        x += delta.to(torch.float32)
    if step is not None:
        x += step
    return (torch.tanh(alpha * x) * w + b).to(out_dtype) if want_out else None


def kv_store(k, v, slot_map, k_cache, v_cache):
    """k [T, n_kv * dk], v [T, n_kv * dv] (any row stride) -> rows of the paged caches [blocks, n_kv, bs, dk / dv]; slots < 0 are skipped."""
    T, n_kv, bs = k.shape[0], k_cache.shape[1], k_cache.shape[2]
    ok = slot_map >= 0
    blk, off = (slot_map[ok] // bs).long(), (slot_map[ok] % bs).long()
    k_cache[blk, :, off] = k.reshape(T, n_kv, -1)[ok].to(k_cache.dtype)
    v_cache[blk, :, off] = v.reshape(T, n_kv, -1)[ok].to(v_cache.dtype)


def mingru_scan(z, u, g, zb, ub, state, state_slots, cu_q, seq_lens, max_q_len):
    """Element-wise gated recurrence over packed sequences: S_t = (1 - s(z)) S_(t-1) + s(z) c(u), y = S_t * silu(g) with s the sigmoid and
    c(u) = u + 1/2 above zero, s(u) below; z and u get their biases here.  z, u, g [T, W] (any row stride); state fp32 [slots, W] is
    advanced in place and starts from zeros for a sequence whose step begins at position 0."""
    T, W = z.shape
    y = torch.empty(T, W, dtype=z.dtype, device=z.device)
    zz = torch.sigmoid(z.to(torch.float32) + zb)
    uu = u.to(torch.float32) + ub
    c = torch.where(uu >= 0, uu + 0.5, torch.sigmoid(uu))
    gate = torch.nn.functional.silu(g.to(torch.float32))
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        S = torch.zeros(W, dtype=torch.float32, device=z.device) if int(seq_lens[b]) == t1 - t0 else state[slot].clone()
        for t in range(t0, t1):
            S = (1.0 - zz[t]) * S + zz[t] * c[t]
            y[t] = (S * gate[t]).to(y.dtype)
        state[slot] = S
    return y


def causal_conv(x, w, b, state, state_slots, cu_q, seq_lens, max_q_len):
    """Causal convolution per channel over packed sequences, no activation: y_t = sum_j w[:, j] x_(t - taps + 1 + j) + b, zeros before a sequence's start.
    x [T, C] (any row stride), w fp32 [C, taps], b fp32 [C]; state [slots, taps - 1, C] of x's dtype holds the inputs before the next token and is
    advanced in place."""
    T, C = x.shape
    taps = w.shape[1]
    y = torch.empty(T, C, dtype=x.dtype, device=x.device)
    cu = cu_q.tolist()
    for i in range(len(cu) - 1):
        t0, t1 = cu[i], cu[i + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[i])
        before = torch.zeros_like(state[slot]) if int(seq_lens[i]) == t1 - t0 else state[slot]
        full = torch.cat([before, x[t0:t1]]).to(torch.float32)
        y[t0:t1] = ((full.unfold(0, taps, 1) * w).sum(-1) + b).to(x.dtype)
        state[slot] = full[full.shape[0] - (taps - 1):].to(state.dtype)
    return y


def _rglru(r, i, u, y, coef, S):
    """One token: S <- a S + sqrt(1 - a^2) sigmoid(i) u with log a = coef sigmoid(r); (S, S gelu(y))."""
    la = coef * torch.sigmoid(r)
    S = torch.exp(la) * S + torch.sqrt(-torch.expm1(2.0 * la)) * torch.sigmoid(i) * u
    return S, S * torch.nn.functional.gelu(y, approximate="tanh")


def rglru_scan(gates, u, y, bias, coef, state, state_slots, cu_q, seq_lens, max_q_len):
    """Real-gated linear recurrence over packed sequences (see _rglru).  gates fp32 [T, blocks, 2 n] = the pre-activations of r and of i of a block's n
    channels, bias fp32 [blocks, 2 n] joins them; u, y [T, blocks * n] (any row stride); coef fp32 [blocks * n]; state fp32 [slots, blocks * n], advanced
    in place, from zeros for a sequence whose step begins at position 0."""
    T, W = u.shape
    n = gates.shape[2] // 2
    g = gates + bias
    r, i = g[..., :n].reshape(T, W), g[..., n:].reshape(T, W)
    out = torch.empty(T, W, dtype=u.dtype, device=u.device)
    uf, yf = u.to(torch.float32), y.to(torch.float32)
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        S = torch.zeros(W, dtype=torch.float32, device=u.device) if int(seq_lens[b]) == t1 - t0 else state[slot].clone()
        for t in range(t0, t1):
            S, o = _rglru(r[t], i[t], uf[t], yf[t], coef, S)
            out[t] = o.to(out.dtype)
        state[slot] = S
    return out


def rglru_step(x, y, conv_w, conv_b, w: QuantWeight, bias, coef, conv_state, state, state_slots, cu_q, seq_lens):
    """One token per sequence: convolution, gates and recurrence together.  x, y [T, W] (any row stride); w stacks per block the 2 n rows of the two gates."""
    u = causal_conv(x, conv_w, conv_b, conv_state, state_slots, cu_q, seq_lens, 1)
    gates = head_linear(u.view(u.shape[0], w.E, w.K), w, out_f32=True)
    return rglru_scan(gates, u, y, bias, coef, state, state_slots, cu_q, seq_lens, 1)


def attention(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks=None, window=0, scale=None, softcap=0.0, n_splits=1,
              kv_scales=None, max_kv_len=0, q_scale=None, gate=None, keep_first=0, pools=None, pool_dense=None, out_rope=None):
    """q [Tq,n_q,hd]; caches [blocks,n_kv,bs,hd] (bf16 / fp32, or int8 with kv_scales = (k_scale, v_scale) [blocks,n_kv,bs]); values may be
    wider or narrower than keys; returns [Tq,n_q,value width] (bf16; fp32 for fp32 queries).  ``q_scale`` [positions]: factor on the scores
    of a query at that position; ``gate`` [Tq, n_q * value width] or [Tq, n_q] (one number per head): the result is multiplied by its sigmoid.
    With a window the first ``keep_first`` keys of a sequence stay visible.  ``pools`` (:class:`PoolPages`): pooled blocks before the window are seen
    beside its keys (``pool_dense`` is what :func:`pool_blocks` returned).  ``out_rope`` = (cos, sin): the result at position p is turned by -p in
    interleaved pairs, before the gate."""
    Tq, n_q, hd = q.shape
    dv = v_cache.shape[3]
    n_kv, bs = k_cache.shape[1], k_cache.shape[2]
    gqa = n_q // n_kv
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    out = torch.zeros(Tq, n_q, dv, dtype=torch.float32, device=q.device)
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        q0, q1 = cu[b], cu[b + 1]
        if q1 <= q0:
            continue
        L = int(seq_lens[b])
        nblk = (L + bs - 1) // bs
        blocks = block_table[b, :nblk].long()
        Kp, Vp = k_cache[blocks].to(torch.float32), v_cache[blocks].to(torch.float32)
        if kv_scales is not None:
            Kp, Vp = Kp * kv_scales[0][blocks].unsqueeze(-1), Vp * kv_scales[1][blocks].unsqueeze(-1)
        K = Kp.permute(1, 0, 2, 3).reshape(n_kv, nblk * bs, hd)[:, :L]
        V = Vp.permute(1, 0, 2, 3).reshape(n_kv, nblk * bs, dv)[:, :L]
        qq = q[q0:q1].to(torch.float32) * scale                                 # [t, n_q, hd]
        if q_scale is not None:
            qq = qq * q_scale[L - (q1 - q0):L].reshape(-1, 1, 1)
        n_pool = 0
        if pools is not None:
            n_pool = max(L - pools.window, 0) // pools.pool
            if n_pool:
                page, row = pools.place(torch.arange(n_pool, device=q.device), bs)
                at = block_table[b].long()[page]
                K = torch.cat([K, pools.k[at, :, row].to(torch.float32).transpose(0, 1)], dim=1)
                V = torch.cat([V, pools.v[at, :, row].to(torch.float32).transpose(0, 1)], dim=1)
        Kh = K.repeat_interleave(gqa, dim=0)
        Vh = V.repeat_interleave(gqa, dim=0)
        s = torch.einsum("thd,hkd->htk", qq.to(_MM_DTYPE), Kh.to(_MM_DTYPE)).to(torch.float32)
        if softcap and softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        qpos = torch.arange(L - (q1 - q0), L, device=q.device).unsqueeze(-1)
        kpos = torch.arange(L, device=q.device).unsqueeze(0)
        ok = kpos <= qpos
        if window and window > 0:
            ok = ok & ((kpos > qpos - window) | (kpos < keep_first))
        if n_pool:
            ok = torch.cat([ok, torch.arange(1, n_pool + 1, device=q.device).unsqueeze(0) * pools.pool - 1 <= qpos - pools.window], dim=1)
        s = s.masked_fill(~ok.unsqueeze(0), float("-inf"))
        if sinks is not None:
            sk = sinks.to(torch.float32).reshape(n_q, 1, 1).expand(n_q, q1 - q0, 1)
            p = torch.softmax(torch.cat([s, sk], dim=-1), dim=-1)[..., :-1]
        else:
            p = torch.softmax(s, dim=-1)
        out[q0:q1] = torch.einsum("htk,hkd->thd", p.to(_MM_DTYPE), Vh.to(_MM_DTYPE)).to(torch.float32)
        if out_rope is not None:
            at = qpos.squeeze(-1).clamp(max=out_rope[0].shape[0] - 1)
            out[q0:q1] = _rotate_pairs(out[q0:q1], out_rope[0][at].unsqueeze(1), -out_rope[1][at].unsqueeze(1))
    if gate is not None:
        out = out * torch.sigmoid(gate.to(torch.float32)).reshape(Tq, n_q, -1)
    return out if q.dtype == torch.float32 else out.to(torch.bfloat16)


@dataclass
class PoolPages:
    """Pooled rows of one layer's cache: block b is the mean of the keys / values at positions b * pool .. b * pool + pool - 1.  ``k``, ``v`` [pages,
    n_kv, rows, width]: a page of bs tokens holds, from row 0 on, the blocks whose last token lies in it.  A query sees the blocks whose last token lies
    ``window`` or more positions before it, so a step forms the blocks that its own queries are the first to see."""
    k: torch.Tensor
    v: torch.Tensor
    pool: int
    window: int

    @staticmethod
    def rows_per_page(bs: int, pool: int) -> int:
        return (bs + pool - 1) // pool

    def place(self, block, bs: int):
        """(page of the sequence, row in it) of a block."""
        page = (block * self.pool + self.pool - 1) // bs
        return page, block - page * bs // self.pool


def _form_pools(k_cache, v_cache, pools: PoolPages, table, start: int, end: int) -> None:
    """The blocks that a step over positions start .. end - 1 of one sequence sees first."""
    bs, P = k_cache.shape[2], pools.pool
    for b in range(max(start - pools.window, 0) // P, max(end - pools.window, 0) // P):
        at = torch.arange(b * P, b * P + P, device=k_cache.device)
        page, row = pools.place(b, bs)
        for cache, out in ((k_cache, pools.k), (v_cache, pools.v)):
            out[table[page], :, row] = cache[table[at // bs], :, at % bs].to(torch.float32).mean(0).to(out.dtype)


def pool_blocks(k_cache, v_cache, pools: PoolPages, block_table, seq_lens, cu_q, max_q_len, max_kv_len=0):
    """Forms the pooled blocks that the queries of this step are the first to see (their tokens lie in the cache).  Returns what the attention of the step
    wants as ``pool_dense`` (here: nothing)."""
    cu = cu_q.tolist()
    for i in range(len(cu) - 1):
        L = int(seq_lens[i])
        if cu[i + 1] > cu[i]:
            _form_pools(k_cache, v_cache, pools, block_table[i].long(), L - (cu[i + 1] - cu[i]), L)
    return None


def qk_post(q, k, positions, rope_cos, rope_sin, slot_map, k_cache, v_cache, dim, rot_dim, interleaved=False, q_norm=None, k_norm=None, norm_after=False,
            eps=1e-6, v=None, v_rope=None, q_scale=None, pools=None, block_table=None):
    """Head epilogue of attention whose values are its projected keys.  q [T, n_q, dp], k [T, n_kv, dp] (column ranges of one projection; the first
    ``dim`` elements are the head, the rest zero padding): RMS norm with the weights q_norm / k_norm [dp], rotation of the first ``rot_dim``
    elements in interleaved pairs or half splits, and with ``norm_after`` an RMS norm without a weight behind it.  Returns the queries (the kernel works
    in place); the keys go into k_cache, and as they came into v_cache (slots < 0 are skipped).
    ``v`` [T, n_kv, dv]: values of their own, turned like keys, in interleaved pairs by the tables ``v_rope`` = (cos, sin) over their first 2 * columns
    elements.  ``q_scale`` [n_q]: factor on the finished queries of a head.  ``pools``: every sequence has one token, and the pooled block that it sees
    first, if there is one, is formed (from tokens of earlier steps)."""
    pos = positions.long().clamp(0, rope_cos.shape[0] - 1)
    c, s = rope_cos[pos].unsqueeze(1), rope_sin[pos].unsqueeze(1)
    half = rot_dim // 2
    rms = lambda t: t * torch.rsqrt(t[..., :dim].pow(2).mean(-1, keepdim=True) + eps)

    def turn(t, w):
        t = t.to(torch.float32)
        if w is not None:
            t = rms(t) * w
        if interleaved:
            t = _rotate_pairs(t, c, s)
        else:
            a, b = t[..., :half], t[..., half:rot_dim]
            t = torch.cat([a * c - b * s, b * c + a * s, t[..., rot_dim:]], dim=-1)
        return rms(t) if norm_after else t

    ok = slot_map >= 0
    bs = k_cache.shape[2]
    blk, off = (slot_map[ok] // bs).long(), (slot_map[ok] % bs).long()
    k_cache[blk, :, off] = turn(k, k_norm)[ok].to(k_cache.dtype)
    if v is None:
        v_cache[blk, :, off] = k[ok].to(v_cache.dtype)
    else:
        at = positions.long().clamp(0, v_rope[0].shape[0] - 1)
        v_cache[blk, :, off] = _rotate_pairs(v.to(torch.float32), v_rope[0][at].unsqueeze(1), v_rope[1][at].unsqueeze(1))[ok].to(v_cache.dtype)
    if pools is not None:
        for t in range(q.shape[0]):
            if bool(ok[t]):
                p = int(positions[t])
                _form_pools(k_cache, v_cache, pools, block_table[t].long(), p, p + 1)
    q = turn(q, q_norm)
    return (q if q_scale is None else q * q_scale.reshape(1, -1, 1)).to(k.dtype)


# ------------------------------------------------------------------ matrix-valued recurrences without a delta rule
def token_shift(x, mu, state, state_slots, cu_q, seq_lens, out_dtype=torch.bfloat16):
    """out[n] = x + (x' - x) mu[n], x' the row of the sequence's previous token (zeros before its first).  x fp32 [T, W], mu [n, W]; state fp32
    [slots, W] holds the last row of what came before and gets the last row of this step.  Returns [n, T, W]."""
    prev = torch.zeros_like(x)
    prev[1:] = x[:-1]
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        if cu[b + 1] <= cu[b]:
            continue
        slot = int(state_slots[b])
        prev[cu[b]] = 0.0 if int(seq_lens[b]) == cu[b + 1] - cu[b] else state[slot]
        state[slot] = x[cu[b + 1] - 1]
    return (x.unsqueeze(0) + (prev - x).unsqueeze(0) * mu.unsqueeze(1)).to(out_dtype)


def decay_scan(q, k, v, state, state_slots, cu_q, seq_lens, max_q_len, decay=None, z=None, u=None, silu=False, chunked=None):
    """Linear attention with a decaying state S [dk, dv] per head.  q, k [T, H, dk], v [T, H, dv] (any row stride); state fp32 [slots, H, dk, dv], advanced
    in place, from zeros for a sequence whose step begins at position 0.  Returns o fp32 [T, H * dv].
      decay [H]                        S <- decay S + k v^T, o = S^T q           (``silu``: q, k and v pass through it first)
      z fp32 [T, H * dk], u [H, dk]    o = (S + (u k) v^T)^T q, then S <- diag(exp(-exp(z))) S + k v^T"""
    T, H, dk = q.shape
    q, k, v = (t.to(torch.float32) for t in (q, k, v))
    if silu:
        q, k, v = (torch.nn.functional.silu(t) for t in (q, k, v))
    w = torch.exp(-torch.exp(z)).reshape(T, H, dk) if z is not None else None
    out = torch.empty(T, H, v.shape[2], dtype=torch.float32, device=q.device)
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        S = torch.zeros_like(state[slot]) if int(seq_lens[b]) == t1 - t0 else state[slot].clone()
        for t in range(t0, t1):
            kv = k[t].unsqueeze(-1) * v[t].unsqueeze(1)
            if w is None:
                S = decay.reshape(H, 1, 1) * S + kv
                out[t] = torch.einsum("hk,hkv->hv", q[t], S)
            else:
                out[t] = torch.einsum("hk,hkv->hv", q[t], S + u.unsqueeze(-1) * kv)
                S = w[t].unsqueeze(-1) * S + kv
        state[slot] = S
    return out.reshape(T, -1)


def gated_group_norm(o, gate, w, eps, groups=1, width=None, silu=False, out_dtype=torch.bfloat16):
    """norm(o) * w * act(gate): RMS norm over each of ``groups`` equal runs of a row whose first ``width`` elements (default: all) are live, the rest
    zero; act is SiLU or the sigmoid.  o fp32 [T, W], gate [T, W] (any row stride), w [W]."""
    T, W = o.shape
    x = o.reshape(T, groups, W // groups)
    n = x.shape[2] if width is None else width
    x = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps)).reshape(T, W)
    g = gate.to(torch.float32)
    return (x * w * (torch.nn.functional.silu(g) if silu else torch.sigmoid(g))).to(out_dtype)


# ------------------------------------------------------------------ norms on a sublayer's output
@dataclass
class ExpertSum:
    """A branch that has not been formed: the sum of the rows of a token's experts (``y`` [rows, H], row pair_to_packed[t * k + j] for its j-th), each
    times its weight when there are weights ``w`` [T, k], and, when there is one, of ``shared`` [T, H], times the sigmoid of ``shared_gate`` [T] (a
    column of a wider matrix: any stride) when there is one."""
    y: torch.Tensor
    pair_to_packed: torch.Tensor
    k: int
    shared: Optional[torch.Tensor] = None
    w: Optional[torch.Tensor] = None
    shared_gate: Optional[torch.Tensor] = None

    def rows(self, idx):
        pick = lambda t: None if t is None else t.index_select(0, idx)
        return ExpertSum(self.y, self.pair_to_packed.view(-1, self.k).index_select(0, idx).reshape(-1), self.k, pick(self.shared), pick(self.w),
                         pick(self.shared_gate))

    def materialize(self, eps=0.0, width=None):
        d = self.y.to(torch.float32)[self.pair_to_packed.long()].view(-1, self.k, self.y.shape[1])
        d = (d if self.w is None else d * self.w.unsqueeze(-1)).sum(1)
        if self.shared is None:
            return d
        s = self.shared.to(torch.float32)
        return d + (s if self.shared_gate is None else s * torch.sigmoid(self.shared_gate).unsqueeze(-1))


@dataclass
class BranchMean:
    """A branch that has not been formed: the mean of two branches [T, H], each RMS-normed with its own weight first."""
    a: torch.Tensor
    a_w: torch.Tensor
    b: torch.Tensor
    b_w: torch.Tensor

    def rows(self, idx):
        return BranchMean(self.a.index_select(0, idx), self.a_w, self.b.index_select(0, idx), self.b_w)

    def materialize(self, eps=0.0, width=None):
        n = width or self.a.shape[1]
        rms = lambda t: t.to(torch.float32) * torch.rsqrt(t.to(torch.float32).pow(2).sum(-1, keepdim=True) / n + eps)
        return 0.5 * (rms(self.a) * self.a_w + rms(self.b) * self.b_w)


def sublayer_norm(x, delta, delta_w, eps, w=None, width=None, out_dtype=torch.bfloat16, want_out=True, out=None):
    """x <- x + norm(delta) * delta_w, without ``delta_w`` x <- x + delta (fp32, in place; delta: a tensor, an :class:`ExpertSum`, a :class:`BranchMean`,
    or None); returns norm(x) * w, or without ``w`` x itself, as ``out_dtype``.  Rows are padded to x.shape[1] columns (weights too, with zeros); the mean
    runs over ``width``.  ``out``: where the result goes (unit column stride, any row stride)."""
    n = width or x.shape[1]
    rms = lambda t: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / n + eps)
    if delta is not None:
        d = delta.to(torch.float32) if isinstance(delta, torch.Tensor) else delta.materialize(eps, n)
        x += d if delta_w is None else rms(d) * delta_w
    if not want_out:
        return None
    y = (x if w is None else rms(x) * w).to(out_dtype)
    return y if out is None else out.copy_(y)


# ------------------------------------------------------------------ latent attention
def _rotate_pairs(t, cos, sin):
    """Interleaved pairs (2i, 2i + 1) of the first 2 * cos.shape[-1] elements."""
    n = 2 * cos.shape[-1]
    u, v = t[..., 0:n:2], t[..., 1:n:2]
    return torch.cat([torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2), t[..., n:]], dim=-1)


def latent_post(q_rot, ckv, norm_w, rank, eps, positions, rope_cos, rope_sin, slot_map, cache, q_out):
    """Head epilogue of latent attention.  q_rot [T, H, r]: the rotated part of the queries -> rotated into q_out [T, H, r] (may be the same
    memory).  ckv [T, R + r]: columns [0, rank) are RMS-normed (weight norm_w [R], zero past rank), columns R.. are the shared key part, rotated;
    the row goes into the paged cache [blocks, 1, bs, R + r] (slots < 0 are skipped)."""
    R, bs = norm_w.numel(), cache.shape[2]
    pos = positions.long().clamp(0, rope_cos.shape[0] - 1)
    c, s = rope_cos[pos], rope_sin[pos]
    q_out.copy_(_rotate_pairs(q_rot.to(torch.float32), c.unsqueeze(1), s.unsqueeze(1)).to(q_out.dtype))
    x = ckv.to(torch.float32)
    lat = x[:, :R] * torch.rsqrt(x[:, :rank].pow(2).mean(-1, keepdim=True) + eps) * norm_w
    row = torch.cat([lat, _rotate_pairs(x[:, R:], c, s)], dim=-1).to(cache.dtype)
    ok = slot_map >= 0
    cache[(slot_map[ok] // bs).long(), 0, (slot_map[ok] % bs).long()] = row[ok]


def head_linear(x, w: QuantWeight, gate=None, out=None, out_f32=False):
    """Every head its own matrix: out[t, h] = W[h] x[t, h] (* sigmoid(gate[t, h])).  x [T, H, K] (any row / head stride), w stacks H matrices
    [N, K]; gate [T, H * N]; out [T, H, N], in fp32 with ``out_f32``."""
    y = torch.einsum("thk,hnk->thn", x.to(_MM_DTYPE), _dense(w)).to(torch.float32)
    if gate is not None:
        y = y * torch.sigmoid(gate.to(torch.float32)).reshape(y.shape)
    y = y if out_f32 else y.to(x.dtype)
    return y if out is None else out.copy_(y)


def stacked_linear(x, w: QuantWeight):
    """Every matrix of a stack with its own input: out[n] = x[n] W[n]^T.  x [n, T, K] (contiguous), w n matrices [N, K] -> [n, T, N]."""
    return torch.einsum("ntk,nmk->ntm", x.to(_MM_DTYPE), _dense(w)).to(torch.float32).to(x.dtype)


def latent_attention(q, cache, block_table, seq_lens, cu_q, max_q_len, rank, window=0, scale=1.0):
    """Attention in the latent space: all heads share one cached row per token, whose first ``rank`` elements are also the value.
    q [Tq, H, width of a cache row] -> [Tq, H, rank]."""
    return attention(q, cache, cache[..., :rank], block_table, seq_lens, cu_q, max_q_len, window=window, scale=scale)


def latent_attention_expanded(q, w_kv: QuantWeight, cache, block_table, seq_lens, cu_q, max_q_len, dim, vdim, rank, window=0, scale=1.0, gate=None,
                              out=None, plans=None):
    """Attention with per-head keys and values formed from the cached latents.  q [Tq, H, dim + r] (rotated), w_kv [H * dim + H * vdim, rank] (key
    rows of all heads, then value rows) -> [Tq, H, vdim] (* sigmoid(gate)).  Only the rows that cu_q names are written."""
    H, bs = q.shape[1], cache.shape[2]
    out = torch.zeros(q.shape[0], H, vdim, dtype=q.dtype, device=q.device) if out is None else out
    cu, W = cu_q.tolist(), _dense(w_kv)[0]
    for b in range(len(cu) - 1):
        q0, q1 = cu[b], cu[b + 1]
        if q1 <= q0:
            continue
        L = int(seq_lens[b])
        rows = cache[block_table[b, :(L + bs - 1) // bs].long(), 0].reshape(-1, cache.shape[3])[:L]
        kv = _mm(rows[:, :rank], W).to(q.dtype).to(torch.float32)
        K = torch.cat([kv[:, :H * dim].reshape(L, H, dim), rows[:, rank:].to(torch.float32).unsqueeze(1).expand(L, H, -1)], dim=-1)
        s = torch.einsum("thd,khd->htk", q[q0:q1].to(torch.float32) * scale, K)
        gap = torch.arange(L - (q1 - q0), L, device=q.device).unsqueeze(1) - torch.arange(L, device=q.device)
        s = s.masked_fill((gap < 0) | ((gap >= window) if window > 0 else False), float("-inf"))
        o = torch.einsum("htk,khd->thd", torch.softmax(s, dim=-1), kv[:, H * dim:].reshape(L, H, vdim))
        if gate is not None:
            o = o * torch.sigmoid(gate[q0:q1].to(torch.float32)).reshape(o.shape)
        out[q0:q1] = o.to(q.dtype)
    return out


def sigmoid_mul(x, g):
    return (x.to(torch.float32) * torch.sigmoid(g.to(torch.float32))).to(torch.bfloat16)


def scaled_add(out, src, gate_logit=None):
    s = src.to(torch.float32)
    if gate_logit is not None:
        s = s * torch.sigmoid(gate_logit).unsqueeze(-1)
    out.add_(s)
    return out


def gated_rmsnorm(x, z, w, eps):
    """x fp32 [rows,hd], z bf16 [rows,hd]."""
    zz = z.to(torch.float32)
    return (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w * torch.nn.functional.silu(zz)).to(torch.bfloat16)


def gated_rmsnorm_heads(x, z, w, eps, hd):
    """x fp32 [T, n_h*hd]; z bf16 [T, n_h*hd] (any row stride); per-head y = w * x/rms(x) * silu(z) -> bf16 [T, n_h*hd]."""
    T = x.shape[0]
    xx = x.reshape(T, -1, hd)
    zz = z.to(torch.float32).reshape(T, -1, hd)
    y = xx * torch.rsqrt(xx.pow(2).mean(-1, keepdim=True) + eps) * w * torch.nn.functional.silu(zz)
    return y.reshape(T, -1).to(torch.bfloat16)


# ------------------------------------------------------------------ gated DeltaNet
def conv1d_silu(x, w, state, state_slots, cu_q, max_q_len, ckpt=None):
    """Depthwise causal conv + SiLU over packed variable-length sequences.

    x bf16 [T, C] (any row stride); w fp32 [C, Kc], tap j multiplies input t-(Kc-1)+j; state bf16 [slots, Kc-1, C]
    holds the Kc-1 inputs before each sequence's next token and is advanced in place; ckpt (optional, bf16
    [T, Kc-1, C]) receives the state as it stands after every position."""
    T, C = x.shape
    Kc = w.shape[1]
    y = torch.empty(T, C, dtype=torch.bfloat16, device=x.device)
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        full = torch.cat([state[slot].to(torch.float32), x[t0:t1].to(torch.float32)], dim=0)      # [Kc-1+n, C]
        win = full.unfold(0, Kc, 1)                                                               # [n, C, Kc]
        acc = (win * w.unsqueeze(0)).sum(-1)
        y[t0:t1] = torch.nn.functional.silu(acc).to(torch.bfloat16)
        if ckpt is not None:
            for i in range(t1 - t0):
                ckpt[t0 + i] = full[i + 1:i + Kc].to(torch.bfloat16)
        state[slot] = full[-(Kc - 1):].to(torch.bfloat16)
    return y


def deltanet_scan(qkv, n_k, ab, a_idx, b_idx, k_of_v, ssm_a, dt_bias, state, state_slots, cu_q, n_v, eps=1e-6, ckpt=None):
    """Gated delta rule over packed sequences.

    qkv bf16 [T, (2 n_k + n_v) * 128] = conv output (q heads | k heads | v heads); ab bf16 [T, *] holds the alpha / beta
    logits of v-head h in columns a_idx[h] / b_idx[h]; k_of_v[h] = k-head feeding v-head h.  Per token:
    q, k L2-normalised (q also scaled by 1/sqrt(128)); g = ssm_a * softplus(alpha + dt_bias); beta = sigmoid(.);
    S <- e^g S;  d = (v - S^T k) beta;  S <- S + k d^T;  out = S^T q.   state fp32 [slots, n_v, 128 (v), 128 (k)]
    is advanced in place; ckpt (optional fp32 [T, n_v, 128, 128]) receives S after every position.  Returns fp32 [T, n_v*128]."""
    T, D = qkv.shape[0], 128
    x = qkv.to(torch.float32)
    q = x[:, :n_k * D].reshape(T, n_k, D)
    k = x[:, n_k * D:2 * n_k * D].reshape(T, n_k, D)
    v = x[:, 2 * n_k * D:].reshape(T, n_v, D)
    q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + eps) / math.sqrt(D)
    k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + eps)
    kv = k_of_v.long()
    q, k = q[:, kv], k[:, kv]
    abf = ab.to(torch.float32)
    g = ssm_a * torch.nn.functional.softplus(abf[:, a_idx.long()] + dt_bias)
    beta = torch.sigmoid(abf[:, b_idx.long()])
    out = torch.empty(T, n_v, D, dtype=torch.float32, device=qkv.device)
    cu = cu_q.tolist()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        S = state[slot].clone()
        for t in range(t0, t1):
            S = S * torch.exp(g[t]).reshape(n_v, 1, 1)
            d = (v[t] - torch.einsum("hvk,hk->hv", S, k[t])) * beta[t].unsqueeze(-1)
            S = S + d.unsqueeze(-1) * k[t].unsqueeze(1)
            out[t] = torch.einsum("hvk,hk->hv", S, q[t])
            if ckpt is not None:
                ckpt[t] = S
        state[slot] = S
    return out.reshape(T, n_v * D)


# ------------------------------------------------------------------ MoE
DELTANET_CHUNK = 64


def deltanet_scan_chunked(qkv, n_k, ab, a_idx, b_idx, k_of_v, ssm_a, dt_bias, state, state_slots, cu_q, n_v, eps=1e-6, chunk=DELTANET_CHUNK):
    """The same recurrence as :func:`deltanet_scan` in its chunked (WY) form: the arithmetic of the tensor-core scan kernel, stated
    in fp32.  Within a chunk of C tokens with cumulative log-decay G_i, the per-token corrections U (rows u_i = d_i) solve
        (I + A) U = beta * V - diag(beta e^G) K S0^T,      A_ij = beta_i e^{G_i - G_j} (k_i . k_j) for j < i,
    so with T = (I + A)^-1:  U = T (beta V) - T (beta e^G K) S0^T;  the outputs are O = diag(e^G) Q S0^T + (M * Q K^T) U with
    M_ij = e^{G_i - G_j} for j <= i, and the state leaves the chunk as S = e^{G_last} S0 + U^T diag(e^{G_last - G}) K.
    Sequences are padded to whole chunks with beta = 0, g = 0, k = 0 rows (identity steps).  No per-position checkpoints."""
    T, D = qkv.shape[0], 128
    x = qkv.to(torch.float32)
    q = x[:, :n_k * D].reshape(T, n_k, D)
    k = x[:, n_k * D:2 * n_k * D].reshape(T, n_k, D)
    v = x[:, 2 * n_k * D:].reshape(T, n_v, D)
    q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + eps) / math.sqrt(D)
    k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + eps)
    kv = k_of_v.long()
    q, k = q[:, kv], k[:, kv]                                        # [T, n_v, D]
    abf = ab.to(torch.float32)
    g = ssm_a * torch.nn.functional.softplus(abf[:, a_idx.long()] + dt_bias)      # [T, n_v]
    beta = torch.sigmoid(abf[:, b_idx.long()])
    out = torch.empty(T, n_v, D, dtype=torch.float32, device=qkv.device)
    cu = cu_q.tolist()
    C = chunk
    tril = torch.tril(torch.ones(C, C, device=qkv.device), diagonal=-1).bool()
    for b in range(len(cu) - 1):
        t0, t1 = cu[b], cu[b + 1]
        if t1 <= t0:
            continue
        slot = int(state_slots[b])
        S = state[slot].clone()                                      # [n_v, D(v), D(k)]
        for c0 in range(t0, t1, C):
            n = min(C, t1 - c0)
            pad = lambda t: torch.cat([t[c0:c0 + n], t.new_zeros((C - n,) + t.shape[1:])]) if n < C else t[c0:c0 + n]
            qc, kc, vc, gc, bc = (pad(t).transpose(0, 1) for t in (q, k, v, g, beta))      # [n_v, C, ...]
            G = gc.cumsum(-1)                                        # [n_v, C]
            dec = torch.exp(G.unsqueeze(-1) - G.unsqueeze(-2))       # e^{G_i - G_j}
            A = (bc.unsqueeze(-1) * dec * (kc @ kc.transpose(-1, -2))).masked_fill(~tril, 0.0)
            Tm = torch.linalg.solve_triangular(torch.eye(C, device=A.device) + A, torch.eye(C, device=A.device).expand_as(A), upper=False)
            Wv = Tm @ (bc.unsqueeze(-1) * vc)                        # [n_v, C, D(v)]
            Wk = Tm @ ((bc * torch.exp(G)).unsqueeze(-1) * kc)       # [n_v, C, D(k)]
            U = Wv - Wk @ S.transpose(-1, -2)
            Mqk = (dec * (qc @ kc.transpose(-1, -2))).masked_fill(torch.triu(torch.ones(C, C, device=A.device), diagonal=1).bool(), 0.0)
            O = torch.exp(G).unsqueeze(-1) * (qc @ S.transpose(-1, -2)) + Mqk @ U
            Gl = G[:, -1]
            S = torch.exp(Gl).reshape(n_v, 1, 1) * S + U.transpose(-1, -2) @ (torch.exp(Gl.unsqueeze(-1) - G).unsqueeze(-1) * kc)
            out[c0:c0 + n] = O.transpose(0, 1)[:n]
        state[slot] = S
    return out.reshape(T, n_v * D)


def moe_route(logits, bias, k, renorm=True, precise=False, sigmoid=False, experts=None):
    """``sigmoid``: the weights are the sigmoids of the chosen logits, as they are.  ``experts``: only the first so many columns are experts."""
    x = logits[:, :experts].to(torch.float32)
    if bias is not None:
        x = x + bias
    # descending value, ties -> lowest index (stable sort on -x)
    order = torch.sort(-x, dim=-1, stable=True).indices[:, :k]
    sel = torch.gather(x, 1, order)
    if sigmoid:
        w = torch.sigmoid(sel)
    elif renorm:
        w = torch.softmax(sel, dim=-1)
    else:
        w = torch.exp(sel - torch.logsumexp(x, dim=-1, keepdim=True))
    return order.to(torch.int32), w


@dataclass
class MoePacking:
    counts: torch.Tensor          # [E]
    seg_start: torch.Tensor       # [E+1] padded segment starts
    packed_token: torch.Tensor    # [max_rows] token of each packed row (-1 = pad)
    pair_to_packed: torch.Tensor  # [T*K] packed row of each (token, slot) pair, -1 if not owned
    tile_expert: torch.Tensor     # [max_tiles]
    num_tiles: torch.Tensor       # [2]: live tiles, packed rows
    max_rows: int
    K: int
    tile_valid: Optional[torch.Tensor] = None   # [max_tiles] live rows of each tile (block-scaled MXFP4 kernel)


def moe_max_rows(n_pairs: int, n_local_experts: int) -> int:
    return (n_pairs + n_local_experts * (MOE_TILE - 1) + MOE_TILE - 1) // MOE_TILE * MOE_TILE


def moe_pack(topk_idx, E, e_lo=0, e_hi=None, tile=MOE_TILE):
    """``tile`` = 128: segments padded to GEMM tiles; ``tile`` = 1: compact segments (batched-decode GEMV path)."""
    e_hi = E if e_hi is None else e_hi
    T, K = topk_idx.shape
    dev = topk_idx.device
    flat = topk_idx.reshape(-1).long()
    n = flat.numel()
    max_rows = moe_max_rows(n, e_hi - e_lo) if tile > 1 else max(n, 1)
    owned = (flat >= e_lo) & (flat < e_hi)
    counts = torch.bincount(flat[owned], minlength=E)[:E]
    padded = (counts + tile - 1) // tile * tile
    seg = torch.zeros(E + 1, dtype=torch.long, device=dev)
    seg[1:] = torch.cumsum(padded, 0)
    packed_token = torch.full((max_rows,), -1, dtype=torch.int32, device=dev)
    pair_to_packed = torch.full((n,), -1, dtype=torch.int32, device=dev)
    order = torch.sort(torch.where(owned, flat, torch.full_like(flat, E)), stable=True).indices
    n_owned = int(owned.sum())
    order = order[:n_owned]
    e_sorted = flat[order]
    rank_in_e = torch.arange(n_owned, device=dev) - torch.cumsum(counts, 0)[e_sorted] + counts[e_sorted]
    dst = seg[e_sorted] + rank_in_e
    packed_token[dst] = (order // K).to(torch.int32)
    pair_to_packed[order] = dst.to(torch.int32)
    tiles = (padded // MOE_TILE) if tile > 1 else torch.zeros_like(padded)
    tile_expert = torch.repeat_interleave(torch.arange(E, device=dev), tiles).to(torch.int32)
    max_tiles = max(max_rows // MOE_TILE, 1)
    te = torch.zeros(max_tiles, dtype=torch.int32, device=dev)
    te[: tile_expert.numel()] = tile_expert
    num_tiles = torch.tensor([int(tiles.sum()), int(seg[E])], dtype=torch.int32, device=dev)
    tv = torch.zeros(max_tiles, dtype=torch.int32, device=dev)
    if tile > 1 and tile_expert.numel():
        first = torch.repeat_interleave(torch.cumsum(tiles, 0) - tiles, tiles)           # first tile of each tile's expert
        within = torch.arange(tile_expert.numel(), device=dev) - first
        tv[: tile_expert.numel()] = torch.clamp(counts[tile_expert.long()] - within * tile, max=tile).to(torch.int32)
    return MoePacking(counts.to(torch.int32), seg.to(torch.int32), packed_token, pair_to_packed, te, num_tiles, max_rows, K, tv)


def moe_gather(x, pk: MoePacking, f16=False):
    xp = torch.zeros(pk.max_rows, x.shape[1], dtype=torch.float16 if f16 else x.dtype, device=x.device)
    ok = pk.packed_token >= 0
    xp[ok] = x[pk.packed_token[ok].long()].to(xp.dtype)
    return xp


def moe_scale_rows(x, w, pk: Optional[MoePacking] = None):
    """Rows for experts whose weight scales their input: row of pair (t, k) = w[t, k] x[t], at its packed place or, without a packing, at t * K + k."""
    T, K = w.shape
    rows = (x.to(torch.float32).unsqueeze(1) * w.unsqueeze(-1)).reshape(T * K, -1).to(x.dtype)
    if pk is None:
        return rows
    xp = torch.zeros(pk.max_rows, x.shape[1], dtype=x.dtype, device=x.device)
    xp[pk.pair_to_packed.long()] = rows
    return xp


def mxfp8_roundtrip(x: torch.Tensor) -> torch.Tensor:
    """``x`` [..., K] (K a multiple of 32) rounded the way the activation quantiser of the block-scaled MXFP4 kernel rounds it:
    per 32 elements a power-of-two scale, the smallest that keeps the block inside e4m3's range (448), then round-to-nearest
    e4m3.  Returns the decoded fp32 values."""
    xs = x.to(torch.float32).reshape(*x.shape[:-1], x.shape[-1] // 32, 32)
    amax = xs.abs().amax(dim=-1, keepdim=True)
    ex = torch.floor(torch.log2(amax.clamp_min(1e-38))) - 8.0
    ex = torch.where(amax * torch.exp2(-ex) > 448.0, ex + 1.0, ex).clamp_(-126.0, 126.0)
    q = (xs * torch.exp2(-ex)).to(torch.float8_e4m3fn).to(torch.float32)
    return torch.where(amax > 0, q * torch.exp2(ex), torch.zeros_like(q)).reshape(x.shape)


def expert_group_gemv(x, w: QuantWeight, pk: MoePacking, x_index=None, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, e_lo=0):
    """y[r] = W[expert of packed row r] @ x[x_index[r] or r] over a compact packing; bf16 [max_rows, N_out]."""
    W = _dense(w)
    P = pk.max_rows
    n_out = w.N // 2 if act_gated(act) else w.N
    out = torch.zeros(P, n_out, dtype=torch.float32, device=x.device)
    xf = x.to(torch.float32)
    for el in range(w.E):
        e = e_lo + el
        c, s0 = int(pk.counts[e]), int(pk.seg_start[e])
        if c == 0:
            continue
        rows = torch.arange(s0, s0 + c, device=x.device)
        xin = xf[x_index[rows].long()] if x_index is not None else xf[rows]
        y = _mm(xin, W[el])
        if bias is not None:
            y = y + bias[el]
        y = _epilogue_act(y, act, act_alpha, act_limit)
        out[rows] = y
    return out.to(torch.bfloat16)


def moe_combine(yp, pk: MoePacking, w, out=None, accumulate=False):
    """sum_k w[t,k] * yp[pos(t,k)] -> fp32 [T,H] (into ``out`` when given)."""
    T, K = w.shape
    pos = pk.pair_to_packed.reshape(T, K).long()
    rows = yp.to(torch.float32)[pos.clamp_min(0)]                  # [T,K,H]
    rows = rows * (pos >= 0).unsqueeze(-1) * w.unsqueeze(-1)
    y = rows.sum(dim=1)
    if out is None:
        return y
    if accumulate:
        out.add_(y.to(out.dtype))
    else:
        out.copy_(y.to(out.dtype))
    return out


# ------------------------------------------------------------------ sampling
def argmax(logits):
    return torch.argmax(logits, dim=-1).to(torch.int32)   # first maximal index


def rep_penalty(logits, ids, penalty):
    for r in range(logits.shape[0]):
        sel = ids[r][ids[r] >= 0].long()
        if sel.numel() and float(penalty[r]) != 1.0:
            v = logits[r, sel]
            logits[r, sel] = torch.where(v > 0, v / penalty[r], v * penalty[r])
    return logits


def _xorshift(s: int) -> tuple[int, float]:
    m = (1 << 64) - 1
    s ^= s >> 12
    s ^= (s << 25) & m
    s ^= s >> 27
    z = (s * 2685821657736338717) & m
    return s, (z >> 40) / 16777216.0


def sample(logits, temperature, top_k, top_p, min_p, rng):
    """rng: int64/uint64-like tensor of xorshift states (updated in place).  Mirrors the kernel's order of cuts."""
    CAP = 256
    rows, V = logits.shape
    out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    for r in range(rows):
        t = float(temperature[r])
        k = int(top_k[r])
        if k <= 0 or k > CAP:
            k = CAP
        k = min(k, V)
        if t <= 0:
            out[r] = int(torch.argmax(logits[r]))
            continue
        order = torch.sort(-logits[r].to(torch.float32), stable=True).indices[:k]
        vals = logits[r, order].to(torch.float32)
        p = torch.exp((vals - vals[0]) / t)
        keep = k
        tp, mp = float(top_p[r]), float(min_p[r])
        if 0 < tp < 1:
            c = torch.cumsum(p / p.sum(), 0)
            hit = torch.nonzero(c >= tp)
            if hit.numel():
                keep = int(hit[0]) + 1
        if mp > 0:
            n = 1
            while n < keep and float(p[n]) >= mp * float(p[0]):
                n += 1
            keep = n
        state = int(rng[r]) & ((1 << 64) - 1)
        state, u = _xorshift(state)
        rng[r] = state if state < (1 << 63) else state - (1 << 64)
        u = u * float(p[:keep].sum())
        c = torch.cumsum(p[:keep], 0)
        hit = torch.nonzero(u < c)
        out[r] = int(order[int(hit[0])]) if hit.numel() else int(order[keep - 1])
    return out
