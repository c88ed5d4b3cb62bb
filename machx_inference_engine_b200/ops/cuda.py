"""Launchers for the sm_100a kernels (``csrc/cuda``): torch tensors in, raw pointers out via ctypes.

Every function has a twin with the same signature in :mod:`ops.ref`.  Nothing here falls back
to PyTorch math: a missing or failing kernel raises.
"""
from __future__ import annotations

import ctypes as C
import math
from typing import Optional

import torch

from .. import _lib
from .ref import ACT_GEGLU, ACT_NONE, ACT_SWIGLU, ACT_SWIGLU_OAI, MOE_TILE, BranchMean, ExpertSum, MoePacking, PoolPages, act_gated, moe_max_rows
from .weights import QuantWeight, WFormat

_vp = C.c_void_p


class KernelError(RuntimeError):
    pass


def _p(t: Optional[torch.Tensor]):
    return _vp(0) if t is None else _vp(t.data_ptr())


def _stream():
    return _vp(torch.cuda.current_stream().cuda_stream)


def _check(rc: int, what: str):
    if rc != 0:
        raise KernelError(f"{what} failed with code {rc}")


def _planes(w: QuantWeight):
    return int(w.fmt), _p(w.p0), _p(w.p1), _p(w.p2), _p(w.p3)


_launch_count = 0


def launches() -> int:
    """Number of kernel-launching calls made through this module (bench bookkeeping)."""
    return _launch_count


def _count(n=1):
    global _launch_count
    _launch_count += n


def check_status():
    """Synchronise and raise if any kernel recorded a bounded-wait timeout or bad argument."""
    v = _lib.cuda().mx_status_read_and_clear()
    if v:
        names = {1: "TMA producer wait", 2: "MMA wait", 3: "epilogue wait", 4: "dequant producer wait", 5: "peer flag wait",
                 6: "bad argument", 7: "softmax wait"}
        raise KernelError(f"kernel status {v}: {names.get(v, 'unknown')} ran out of its time limit")


def set_gemv_path(path) -> None:
    """Which decode GEMV kernel runs: "auto" (per case, the default), "register" (register-streamed kernels only) or
    "stream" (the bulk-copy streaming kernel wherever it applies); booleans mean register / auto."""
    code = {"auto": 0, "register": 1, "stream": 2, True: 1, False: 0}[path]
    _lib.cuda().mx_gemv_set_path(code)


def set_gemv_bf16_wide(on: Optional[bool]) -> None:
    """Streaming GEMV over bf16 weights with eight consumer warps per CTA instead of four; None: for short rows only, the default
    (MX_GEMV_BF16_WIDE=0/1 sets it at import)."""
    _lib.cuda().mx_gemv_stream_set_bf16_wide(2 if on is None else int(bool(on)))


def set_gemv_tma(on: bool) -> None:
    """Streaming GEMV with chunked rows (K above one chunk): one tiled TMA load per plane and stage (default) or one bulk copy per row."""
    _lib.cuda().mx_gemv_stream_set_tma(int(bool(on)))


def set_pdl(on: bool) -> None:
    """Programmatic dependent launch for the decode-chain kernels (default on): the next kernel's CTAs are scheduled while
    the previous kernel drains and the streaming GEMV prefetches its weights before its inputs exist."""
    _lib.cuda().mx_set_pdl(1 if on else 0)


_sm_count = 0


def sm_count() -> int:
    """Streaming multiprocessors of the current device (148 on a B200), asked once."""
    global _sm_count
    if not _sm_count:
        _sm_count = int(_lib.cuda().mx_sm_count())
    return _sm_count


def _profiled(name):
    """The ops that only exist on the GPU report to the per-op profiler themselves (the CPU/GPU dispatcher wraps the others)."""
    def deco(fn):
        import functools
        from ..utils.profiler import profiler as _prof

        @functools.wraps(fn)
        def wrapped(*args, **kwargs):
            if _prof.enabled:
                return _prof.record(name, fn, args, kwargs)
            return fn(*args, **kwargs)
        return wrapped
    return deco


# ------------------------------------------------------------------ elementwise
def embed(w: QuantWeight, ids, scale: float = 1.0):
    T = ids.numel()
    out = torch.empty(T, w.K, dtype=torch.float32, device=ids.device)
    fmt, p0, p1, p2, p3 = _planes(w)
    _check(_lib.cuda().mx_embed(fmt, p0, p1, p2, p3, _p(ids), _p(out), T, w.K, w.N, C.c_float(scale), _stream()), "embed")
    _count()
    return out


def rmsnorm(x, w, eps, delta=None, dbias=None, one_plus_w=False, delta_scale=1.0, write_x=True, want_out=True):
    T, H = x.shape
    out = torch.empty(T, H, dtype=torch.bfloat16, device=x.device) if want_out else None
    is_f32 = 1 if (delta is not None and delta.dtype == torch.float32) else 0
    if delta is not None:
        assert delta.is_contiguous() and delta.shape == x.shape
    _check(_lib.cuda().mx_rmsnorm(_p(x), _p(delta), is_f32, _p(dbias), _p(w), _p(out), C.c_float(eps), T, H, int(one_plus_w),
                                  C.c_float(delta_scale), int(write_x), _stream()), "rmsnorm")
    _count()
    return out


def group_norm(x, w, eps, groups=1, delta=None, delta_w=None, fresh=False, width=None, out_dtype=torch.bfloat16, want_out=True):
    T, ld = x.shape
    H = ld if width is None else width
    assert x.dtype == torch.float32 and x.is_contiguous() and (delta is None or (delta.is_contiguous() and delta.shape == x.shape))
    out = torch.empty(T, ld, dtype=out_dtype, device=x.device) if want_out else None
    _check(_lib.cuda().mx_group_norm(_p(x), _p(delta), int(delta is not None and delta.dtype == torch.float32), _p(delta_w), _p(w), _p(out),
                                     int(out_dtype == torch.float32), C.c_float(eps), T, H, ld, int(groups), int(fresh), _stream()), "group_norm")
    _count()
    return out


def dyt_norm(x, alpha, w, b, delta=None, step=None, out_dtype=torch.bfloat16, want_out=True):
    T, ld = x.shape
    comb = delta if isinstance(delta, CombineDelta) else None
    rows = comb.y if comb is not None else delta
    assert x.dtype == torch.float32 and x.is_contiguous() and w.numel() == b.numel() == ld and (step is None or step.numel() == ld)
    assert rows is None or (rows.is_contiguous() and rows.shape[1] == ld and (comb is not None or rows.shape[0] == T))
    out = torch.empty(T, ld, dtype=out_dtype, device=x.device) if want_out else None
    _check(_lib.cuda().mx_dyt_norm(_p(x), _p(rows), int(rows is not None and rows.dtype == torch.float32), _p(comb.pair_to_packed if comb else None),
                                   _p(comb.w if comb else None), comb.w.shape[1] if comb else 0, _p(step), C.c_float(alpha), _p(w), _p(b), _p(out),
                                   int(out_dtype == torch.float32), T, ld, _stream()), "dyt_norm")
    _count()
    return out


def sublayer_norm(x, delta, delta_w, eps, w=None, width=None, out_dtype=torch.bfloat16, want_out=True, out=None):
    T, ld = x.shape
    kind, a, b, pos, k, aw, bw, pw, bg = 0, None, None, None, 0, None, None, None, None
    if isinstance(delta, ExpertSum):
        kind, a, b, pos, k, pw, bg = 2, delta.y, delta.shared, delta.pair_to_packed, delta.k, delta.w, delta.shared_gate
        assert pos.numel() == T * k and pos.dtype == torch.int32 and (pw is None or (pw.is_contiguous() and pw.numel() == T * k and pw.dtype == torch.float32))
        assert bg is None or (bg.dtype == torch.float32 and bg.shape == (T,))
    elif isinstance(delta, BranchMean):
        kind, a, b, aw, bw = 3, delta.a, delta.b, delta.a_w, delta.b_w
    elif delta is not None:
        kind, a = 1, delta
    assert x.dtype == torch.float32 and x.is_contiguous()
    assert all(v is None or (v.dtype == torch.float32 and v.numel() == ld) for v in (delta_w, w, aw, bw))
    assert all(t is None or (t.is_contiguous() and t.dtype == out_dtype and t.shape[1] == ld and (kind == 2 or t.shape[0] == T)) for t in (a, b))
    if out is None and want_out:
        out = torch.empty(T, ld, dtype=out_dtype, device=x.device)
    assert out is None or (out.shape == (T, ld) and out.dtype == out_dtype and out.stride(1) == 1)
    _check(_lib.cuda().mx_sublayer_norm(kind, _p(x), _p(a), _p(b), _p(pos), int(k), _p(pw), _p(bg), 0 if bg is None else bg.stride(0), _p(aw), _p(bw), _p(delta_w),
                                        _p(w), _p(out), C.c_longlong(ld if out is None else out.stride(0)), int(out_dtype == torch.float32), C.c_float(eps), T,
                                        int(width or ld), ld, _stream()), "sublayer_norm")
    _count()
    return out


def qk_post(q, k, positions, rope_cos, rope_sin, slot_map, k_cache, v_cache, dim, rot_dim, interleaved=False, q_norm=None, k_norm=None, norm_after=False,
            eps=1e-6, v=None, v_rope=None, q_scale=None, pools=None, block_table=None):
    T, n_q, dp = q.shape
    n_kv = k.shape[1]
    dv = dp if v is None else v.shape[2]
    assert q.dtype == k.dtype == k_cache.dtype == v_cache.dtype and k_cache.shape[1] == n_kv and k_cache.shape[3] == dp
    assert v_cache.shape == (*k_cache.shape[:3], dv) and k_cache.is_contiguous() and v_cache.is_contiguous()
    for t in (q, k) if v is None else (q, k, v):
        assert t.dtype == q.dtype and t.stride(2) == 1 and (t.shape[1] == 1 or t.stride(1) == t.shape[2])
    assert v is None or v.shape[:2] == (T, n_kv)
    assert q_scale is None or (q_scale.dtype == torch.float32 and q_scale.numel() == n_q)
    assert pools is None or (block_table.shape[0] == T and block_table.is_contiguous())
    v_cos, v_sin = v_rope if v_rope is not None else (None, None)
    assert rope_cos.shape[1] == rot_dim // 2 and all(n is None or n.numel() == dp for n in (q_norm, k_norm))
    _check(_lib.cuda().mx_qk_post(_p(q), q.stride(0), _p(k), k.stride(0), _p(q_norm), _p(k_norm), _p(positions), _p(rope_cos), _p(rope_sin), rope_cos.shape[0],
                                  _p(slot_map), _p(k_cache), _p(v_cache), T, n_q, n_kv, dp, int(dim), int(rot_dim), int(interleaved), int(norm_after),
                                  k_cache.shape[2], C.c_float(eps), int(q.dtype == torch.float32), _p(q_scale), _p(v), 0 if v is None else v.stride(0), dv,
                                  _p(v_cos), _p(v_sin), 0 if v_cos is None else v_cos.shape[1], 1 if v_cos is None else v_cos.shape[0],
                                  *((_vp(0), _vp(0), _vp(0), 0, 0, 0, 0) if pools is None else
                                    (_p(pools.k), _p(pools.v), _p(block_table), block_table.shape[1], pools.pool, pools.k.shape[2], pools.window)), _stream()),
           "qk_post")
    _count()
    return q


def pool_blocks(k_cache, v_cache, pools: PoolPages, block_table, seq_lens, cu_q, max_q_len, max_kv_len=0):
    """For queries that take the tensor-core kernel: dense pages (K, V) [B * pages, n_kv, 128, width] of the blocks that every sequence's last query sees."""
    n_pages, n_kv, bs, dk = k_cache.shape
    dv, B, P = v_cache.shape[3], seq_lens.numel(), pools.pool
    assert pools.k.dtype == k_cache.dtype and pools.k.shape[:2] == (n_pages, n_kv) and block_table.is_contiguous()
    longest = max_kv_len if max_kv_len > 0 else block_table.shape[1] * bs
    seen = max(longest - pools.window, 0) // P
    if seen == 0:
        return None
    dense, pages, most = None, 0, min(seen, max_q_len // P + 1)
    if _takes_tc(max_q_len, bs, k_cache.dtype, dk, dv):
        pages, most = (seen + 127) // 128, seen
        dense = tuple(torch.empty(B * pages, n_kv, 128, w, dtype=k_cache.dtype, device=k_cache.device) for w in (dk, dv))
    _check(_lib.cuda().mx_pool_blocks(_p(k_cache), _p(v_cache), _p(pools.k), _p(pools.v), _p(dense[0] if dense else None), _p(dense[1] if dense else None),
                                      _p(block_table), _p(seq_lens), _p(cu_q), B, n_kv, bs, dk, dv, P, pools.k.shape[2], pools.window, block_table.shape[1],
                                      pages, most, int(k_cache.dtype == torch.float32), _stream()), "pool_blocks")
    _count()
    return dense


def causal_conv(x, w, b, state, state_slots, cu_q, seq_lens, max_q_len):
    T, W = x.shape
    assert x.stride(1) == 1 and state.dtype == x.dtype and state.shape[1:] == (w.shape[1] - 1, W) and w.is_contiguous() and w.dtype == b.dtype == torch.float32
    y = torch.empty(T, W, dtype=x.dtype, device=x.device)
    _check(_lib.cuda().mx_causal_conv(_p(x), x.stride(0), _p(w), _p(b), _p(state), _p(state_slots), _p(cu_q), _p(seq_lens), _p(y), cu_q.numel() - 1, T, W,
                                      w.shape[1], int(max_q_len), int(x.dtype == torch.float32), _stream()), "causal_conv")
    _count(2 if w.shape[1] > 1 and max_q_len > 1 else 1)
    return y


def rglru_scan(gates, u, y, bias, coef, state, state_slots, cu_q, seq_lens, max_q_len):
    T, W = u.shape
    n = gates.shape[2] // 2
    assert gates.dtype == state.dtype == torch.float32 and gates.is_contiguous() and gates.shape == (T, W // n, 2 * n) and bias.numel() == 2 * W
    assert u.dtype == y.dtype and u.stride(1) == y.stride(1) == 1 and state.shape[1] == W == coef.numel()
    out = torch.empty(T, W, dtype=u.dtype, device=u.device)
    _check(_lib.cuda().mx_rglru_scan(_p(gates), _p(bias), _p(coef), _p(u), u.stride(0), _p(y), y.stride(0), _p(state), _p(state_slots), _p(cu_q), _p(seq_lens),
                                     _p(out), cu_q.numel() - 1, W, n, int(max_q_len), int(u.dtype == torch.float32), _stream()), "rglru_scan")
    _count()
    return out


RGLRU_FUSED_MAX_B = 4        # up to this many sequences a step is one kernel; more have enough rows for the tensor cores


def rglru_step(x, y, conv_w, conv_b, w: QuantWeight, bias, coef, conv_state, state, state_slots, cu_q, seq_lens):
    T, W = x.shape
    n = w.K
    assert w.fmt == WFormat.BF16 and (w.N, w.E) == (2 * n, W // n) and x.dtype == y.dtype == conv_state.dtype and x.stride(1) == y.stride(1) == 1
    assert cu_q.numel() - 1 == T and state.dtype == torch.float32 and state.shape[1] == W and conv_state.shape[1:] == (conv_w.shape[1] - 1, W)
    if T > RGLRU_FUSED_MAX_B and x.dtype == torch.bfloat16:
        u = causal_conv(x, conv_w, conv_b, conv_state, state_slots, cu_q, seq_lens, 1)
        gates = head_linear(u.view(T, w.E, n), w, out_f32=True)
        return rglru_scan(gates, u, y, bias, coef, state, state_slots, cu_q, seq_lens, 1)
    out = torch.empty(T, W, dtype=x.dtype, device=x.device)
    _check(_lib.cuda().mx_rglru_step(_p(x), x.stride(0), _p(y), y.stride(0), _p(conv_w), _p(conv_b), _p(w.p0), _p(bias), _p(coef), _p(conv_state), _p(state),
                                     _p(state_slots), _p(cu_q), _p(seq_lens), _p(out), T, W, n, conv_w.shape[1], int(x.dtype == torch.float32), _stream()),
           "rglru_step")
    _count()
    return out


def token_shift(x, mu, state, state_slots, cu_q, seq_lens, out_dtype=torch.bfloat16):
    T, W = x.shape
    n = mu.shape[0]
    assert x.dtype == mu.dtype == state.dtype == torch.float32 and x.is_contiguous() and mu.is_contiguous() and mu.shape[1] == state.shape[1] == W
    out = torch.empty(n, T, W, dtype=out_dtype, device=x.device)
    _check(_lib.cuda().mx_token_shift(_p(x), _p(mu), _p(state), _p(state_slots), _p(cu_q), _p(seq_lens), _p(out), int(out_dtype == torch.float32), T, W, n,
                                      cu_q.numel() - 1, _stream()), "token_shift")
    _count()
    return out


DECAY_CHUNKED_MIN_Q = 64          # query segments at least this long take the chunked tensor-core form


def decay_scan(q, k, v, state, state_slots, cu_q, seq_lens, max_q_len, decay=None, z=None, u=None, silu=False, chunked=None):
    """``chunked``: None picks the chunked tensor-core kernels for prompts in bf16 and the sequential kernel otherwise; True / False force one."""
    T, H, dk = q.shape
    dv = v.shape[2]
    assert q.dtype == k.dtype == v.dtype and state.dtype == torch.float32 and state.shape[1:] == (H, dk, dv) and k.shape == q.shape
    for t in (q, k, v):
        assert t.stride(2) == 1 and (H == 1 or t.stride(1) == t.shape[2])
    assert z is None or (z.dtype == torch.float32 and z.is_contiguous() and z.shape == (T, H * dk) and u.shape == (H, dk))
    out = torch.empty(T, H * dv, dtype=torch.float32, device=q.device)
    if chunked is None:
        chunked = q.dtype == torch.bfloat16 and dk <= 128 and max_q_len >= DECAY_CHUNKED_MIN_Q
    if chunked:
        lib, B = _lib.cuda(), cu_q.numel() - 1
        for f in (lib.mx_decay_chunk_ws_bytes, lib.mx_decay_chunk_gl_floats):
            f.restype = C.c_longlong
        assert q.dtype == torch.bfloat16
        ws = torch.empty(int(lib.mx_decay_chunk_ws_bytes(T, B, H, dk, dv)), dtype=torch.uint8, device=q.device)
        gl = torch.empty(int(lib.mx_decay_chunk_gl_floats(T, B, H, dk)), dtype=torch.float32, device=q.device)
        _check(lib.mx_decay_scan_chunked(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(z), _p(u), _p(decay), _p(state), _p(state_slots),
                                         _p(cu_q), _p(seq_lens), _p(out), B, T, H, dk, dv, int(silu), _p(ws), _p(gl), _stream()), "decay_scan_chunked")
        _count(2)
        return out
    _check(_lib.cuda().mx_decay_scan(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(z), _p(u), _p(decay), _p(state), _p(state_slots), _p(cu_q),
                                     _p(seq_lens), _p(out), cu_q.numel() - 1, H, dk, dv, int(silu), int(q.dtype == torch.float32), _stream()), "decay_scan")
    _count()
    return out


def gated_group_norm(o, gate, w, eps, groups=1, width=None, silu=False, out_dtype=torch.bfloat16):
    T, W = o.shape
    assert o.dtype == torch.float32 and o.is_contiguous() and gate.shape == o.shape and gate.stride(1) == 1 and gate.dtype == out_dtype and w.numel() == W
    out = torch.empty(T, W, dtype=out_dtype, device=o.device)
    _check(_lib.cuda().mx_gated_group_norm(_p(o), _p(gate), gate.stride(0), _p(w), _p(out), int(out_dtype == torch.float32), C.c_float(eps), T, int(groups),
                                           W // groups, int(width or W // groups), int(silu), _stream()), "gated_group_norm")
    _count()
    return out


def kv_store(k, v, slot_map, k_cache, v_cache):
    T, n_kv, bs, dk = k.shape[0], k_cache.shape[1], k_cache.shape[2], k_cache.shape[3]
    dv = v_cache.shape[3]
    assert k.dtype == v.dtype == k_cache.dtype == v_cache.dtype and k.stride(1) == 1 and v.stride(1) == 1
    assert k.shape[1] == n_kv * dk and v.shape[1] == n_kv * dv
    _check(_lib.cuda().mx_kv_store(_p(k), _p(v), k.stride(0), v.stride(0), _p(slot_map), _p(k_cache), _p(v_cache), T, n_kv, dk, dv, bs,
                                   k.element_size(), _stream()), "kv_store")
    _count()


def mingru_scan(z, u, g, zb, ub, state, state_slots, cu_q, seq_lens, max_q_len):
    T, W = z.shape
    assert z.dtype == u.dtype == g.dtype and z.stride() == u.stride() == g.stride() and z.stride(1) == 1 and state.dtype == torch.float32
    y = torch.empty(T, W, dtype=z.dtype, device=z.device)
    _check(_lib.cuda().mx_mingru_scan(_p(z), _p(u), _p(g), z.stride(0), _p(zb), _p(ub), _p(state), _p(state_slots), _p(cu_q), _p(seq_lens), _p(y),
                                      cu_q.numel() - 1, W, int(max_q_len), int(z.dtype == torch.float32), _stream()), "mingru_scan")
    _count()
    return y


class CombineDelta:
    """The weighted sum of expert outputs that has not been formed: ``y`` [rows, H] bf16, the packed position of every (token, slot)
    pair (negative = not on this rank) and the routing weights [T, K].  ``rmsnorm_combine`` folds it into the residual inside the
    next norm; ``materialize`` forms it."""

    def __init__(self, y, pair_to_packed, w):
        self.y, self.pair_to_packed, self.w = y, pair_to_packed, w
        self.shape = (w.shape[0], y.shape[1])

    def materialize(self):
        return moe_combine(self.y, MoePacking(None, None, None, self.pair_to_packed, None, None, self.y.shape[0], self.w.shape[1]), self.w)

    def index_select(self, dim, rows):
        assert dim == 0
        return self.materialize().index_select(0, rows)

    def rows(self, rows):
        """The combine of some tokens only, still not formed."""
        K = self.w.shape[1]
        return CombineDelta(self.y, self.pair_to_packed.view(-1, K).index_select(0, rows).reshape(-1), self.w.index_select(0, rows))


@_profiled("rmsnorm_combine")
def rmsnorm_combine(x, w, eps, d: "CombineDelta", one_plus_w=False, delta_scale=1.0, want_out=True):
    T, H = x.shape
    out = torch.empty(T, H, dtype=torch.bfloat16, device=x.device) if want_out else None
    _check(_lib.cuda().mx_rmsnorm_combine(_p(x), _p(d.y), _p(d.pair_to_packed), _p(d.w), d.w.shape[1], _p(w), _p(out), C.c_float(eps), T, H,
                                          int(one_plus_w), C.c_float(delta_scale), _stream()), "rmsnorm_combine")
    _count()
    return out


def glu(x, act, alpha=1.702, limit=7.0):
    T, F2 = x.shape
    if x.dtype == torch.float32:
        out = torch.empty(T, F2 // 2, dtype=torch.float32, device=x.device)
        _check(_lib.cuda().mx_glu_f32(_p(x), _p(out), C.c_longlong(T), F2 // 2, act, C.c_float(alpha), C.c_float(limit), _stream()), "glu")
        _count()
        return out
    out = torch.empty(T, F2 // 2, dtype=torch.bfloat16, device=x.device)
    _check(_lib.cuda().mx_glu(_p(x), _p(out), C.c_longlong(T), F2 // 2, act, C.c_float(alpha), C.c_float(limit), _stream()), "glu")
    _count()
    return out


def sigmoid_mul(x, g):
    y = torch.empty_like(x)
    _check(_lib.cuda().mx_sigmoid_mul(_p(x), _p(g), _p(y), C.c_longlong(x.numel()), _stream()), "sigmoid_mul")
    _count()
    return y


def scaled_add(out, src, gate_logit=None):
    _check(_lib.cuda().mx_scaled_add(_p(out), _p(src), _p(gate_logit), out.shape[-1], C.c_longlong(out.numel()), _stream()), "scaled_add")
    _count()
    return out


def gated_rmsnorm(x, z, w, eps):
    rows, hd = x.shape
    y = torch.empty(rows, hd, dtype=torch.bfloat16, device=x.device)
    _check(_lib.cuda().mx_gated_rmsnorm(_p(x), _p(z), _p(w), _p(y), rows, hd, C.c_float(eps), _stream()), "gated_rmsnorm")
    _count()
    return y


def gated_rmsnorm_heads(x, z, w, eps, hd):
    T = x.shape[0]
    n_h = x.shape[1] // hd
    assert x.dtype == torch.float32 and x.is_contiguous() and z.dtype == torch.bfloat16 and z.stride(1) == 1
    y = torch.empty(T, n_h * hd, dtype=torch.bfloat16, device=x.device)
    _check(_lib.cuda().mx_gated_rmsnorm_ld(_p(x), _p(z), z.stride(0), _p(w), _p(y), T, n_h, hd, C.c_float(eps), _stream()), "gated_rmsnorm")
    _count()
    return y


def conv1d_silu(x, w, state, state_slots, cu_q, max_q_len, ckpt=None):
    T, Cc = x.shape
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1 and w.dtype == torch.float32 and w.is_contiguous() and state.dtype == torch.bfloat16
    y = torch.empty(T, Cc, dtype=torch.bfloat16, device=x.device)
    _check(_lib.cuda().mx_conv1d_silu(_p(x), x.stride(0), Cc, w.shape[1], _p(w), _p(state), _p(state_slots), _p(cu_q), cu_q.numel() - 1, T,
                                      int(max_q_len), _p(y), _p(ckpt), _stream()), "conv1d_silu")
    _count(1 if max_q_len == 1 else 2)
    return y


DELTANET_CHUNKED_MIN_T = 128      # batches of at least this many tokens take the chunked tensor-core scan (no checkpoints there)


def deltanet_scan(qkv, n_k, ab, a_idx, b_idx, k_of_v, ssm_a, dt_bias, state, state_slots, cu_q, n_v, eps=1e-6, ckpt=None, chunked=None):
    """``chunked``: None picks the chunked (WY) tensor-core kernel for prefill-sized batches without checkpoints and the sequential
    kernel otherwise; True / False force one (tests, benches)."""
    T = qkv.shape[0]
    D = 128
    assert qkv.dtype == torch.bfloat16 and qkv.stride(1) == 1 and ab.dtype == torch.bfloat16 and ab.stride(1) == 1 and state.dtype == torch.float32
    out = torch.empty(T, n_v * D, dtype=torch.float32, device=qkv.device)
    if chunked is None:
        chunked = ckpt is None and T >= DELTANET_CHUNKED_MIN_T
    if chunked:
        assert ckpt is None, "the chunked scan keeps no per-position checkpoints"
        B = cu_q.numel() - 1
        lib = _lib.cuda()
        lib.mx_deltanet_chunk_ws_bytes.restype = C.c_longlong
        ws = torch.empty(int(lib.mx_deltanet_chunk_ws_bytes(T, B, n_v)), dtype=torch.uint8, device=qkv.device)
        egl = torch.empty((T // 64 + B) * n_v, dtype=torch.float32, device=qkv.device)
        _check(lib.mx_deltanet_scan_chunked(_p(qkv), qkv.stride(0), 0, n_k * D, 2 * n_k * D, _p(ab), ab.stride(0), _p(a_idx), _p(b_idx), _p(k_of_v),
                                            _p(ssm_a), _p(dt_bias), _p(state), _p(state_slots), _p(cu_q), B, T, n_v, D,
                                            C.c_float(1.0 / math.sqrt(D)), C.c_float(eps), _p(out), _p(ws), _p(egl), _stream()), "deltanet_scan_chunked")
        _count(2)
        return out
    _check(_lib.cuda().mx_deltanet_scan(_p(qkv), qkv.stride(0), 0, n_k * D, 2 * n_k * D, _p(ab), ab.stride(0), _p(a_idx), _p(b_idx), _p(k_of_v),
                                        _p(ssm_a), _p(dt_bias), _p(state), _p(state_slots), _p(cu_q), cu_q.numel() - 1, n_v, D,
                                        C.c_float(1.0 / math.sqrt(D)), C.c_float(eps), _p(out), _p(ckpt), _stream()), "deltanet_scan")
    _count()
    return out


def qkv_post(qkv, bias, q_norm_w, k_norm_w, positions, rope_cos, rope_sin, slot_map, k_cache, v_cache, n_q, n_kv, hd, n_rot,
             q_gate=False, norm_one_plus_w=False, eps=1e-6, kv_scales=None, v_norm=False):
    T = qkv.shape[0]
    q = torch.empty(T, n_q, hd, dtype=torch.bfloat16, device=qkv.device)
    gate = torch.empty(T, n_q, hd, dtype=torch.bfloat16, device=qkv.device) if q_gate else None
    bs = k_cache.shape[2]
    max_pos = rope_cos.shape[0] if rope_cos is not None else 1
    if kv_scales is not None:
        assert k_cache.dtype == torch.int8 and kv_scales[0].dtype == torch.float32
    else:
        assert k_cache.dtype == torch.bfloat16
    ks, vs = kv_scales if kv_scales is not None else (None, None)
    _check(_lib.cuda().mx_qkv_post_kv8(_p(qkv), _p(bias), _p(q_norm_w), _p(k_norm_w), _p(positions), _p(rope_cos), _p(rope_sin),
                                       _p(slot_map), _p(q), _p(gate), _p(k_cache), _p(v_cache), _p(ks), _p(vs), T, n_q, n_kv, hd, n_rot, bs,
                                       int(q_gate) | (2 if v_norm else 0), int(norm_one_plus_w), C.c_float(eps), max_pos, _stream()), "qkv_post")
    _count()
    return q, gate


# ------------------------------------------------------------------ linear layers
GEMV_MAX_M = 8


def _pick_bn(M: int, N: int, wide: bool = False) -> int:
    """Columns per GEMM tile.  ``wide`` (bf16 weights): 256-column tiles may be taken."""
    # small-M problems are weight-read bound: use narrow tiles so every SM streams weights
    sms = sm_count()
    if M <= 128:
        for bn in (128, 64, 32):
            if (N + bn - 1) // bn >= sms:
                return bn
        return 32
    tiles = lambda bn: ((M + 127) // 128) * ((N + bn - 1) // bn)
    if tiles(128) < sms:
        return 64
    # whole waves of tiles, a 256-column tile at 1.71 times the time of a 128-column one (8192^3: 1005 against 1172 us)
    waves = lambda bn: (tiles(bn) + sms - 1) // sms
    return 256 if wide and 1.71 * waves(256) < waves(128) else 128


def _gemm_a(x, w: QuantWeight):
    """Activations in the dtype the tensor-core path of this weight format multiplies in."""
    want = torch.bfloat16
    return x if x.dtype == want else x.to(want)


import os as _os

# dense quantised GEMMs with at least this many rows decode the weight once to bf16 first (MX_DEQUANT_ONCE_MIN_M overrides).  Measured on
# Llama-3-8B Q4_K_M, ms per prefill step without -> with: 64 rows 12.3 -> 11.6, 256 rows 16.5 -> 12.8, 512 rows 27.5 -> 17.2,
# 2048 rows 89.6 -> 46.2; batches of 9..63 rows were not measured and keep the in-kernel decode
DEQUANT_ONCE_MIN_M = int(_os.environ.get("MX_DEQUANT_ONCE_MIN_M", "64"))
if _os.environ.get("MX_GEMV_BF16_WIDE") is not None:
    set_gemv_bf16_wide(_os.environ["MX_GEMV_BF16_WIDE"] not in ("", "0"))


def _out_kind(dtype) -> int:
    return {torch.bfloat16: 0, torch.float32: 1, torch.float16: 2}[dtype]


def _few_rows_take_gemm(M: int, w: QuantWeight, act: int) -> bool:
    """A few rows against a bf16 matrix that the streaming GEMV serves badly: rows too long to sit in its shared memory beside two stages
    (the register GEMV would run: 8 x 21504 against 4096 rows 392 us, the tensor-core kernel 74), or so much weight that five and more rows
    are bound by its arithmetic (8 x 4096 against 21504 rows: 121 us against 55)."""
    if w.fmt != WFormat.BF16 or act_gated(act) or w.K % 8:
        return False
    return (M >= 3 and 2 * M * w.K + 16 * min(w.K, 4096) > 190 * 1024) or (M >= 5 and w.N * w.K >= 48 << 20)


def linear(x, w: QuantWeight, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, out_f32=False, row_scale=None, out=None):
    """``out``: write into this [M, n_out] view (unit column stride; a column slice of a wider matrix is fine), so that projections
    whose weights differ in format can share one output without a concatenation."""
    if x.dtype == torch.float32:
        return _linear_f32(x, w, bias, act, act_alpha, act_limit, row_scale, out)
    assert x.dtype == torch.bfloat16 and x.is_contiguous() and x.shape[-1] == w.K and w.E == 1
    M = x.shape[0]
    if w.fmt == WFormat.EXL3:
        assert act == ACT_NONE and row_scale is None, "EXL3 layers have no fused activation or row scale"
        return _exl3_linear(x, w, bias, out_f32, out)
    n_out = w.N // 2 if act_gated(act) else w.N
    odt = torch.float32 if out_f32 else torch.bfloat16
    if out is None:
        out = torch.empty(M, n_out, dtype=odt, device=x.device)
    assert out.shape == (M, n_out) and out.dtype == odt and (M == 0 or out.stride(1) == 1)
    if M == 0:
        return out
    fmt, p0, p1, p2, p3 = _planes(w)
    lib = _lib.cuda()
    if M <= GEMV_MAX_M and row_scale is None and not _few_rows_take_gemm(M, w, act):
        # the GEMV kernels write dense rows: a strided view of more than one row goes through a dense buffer
        dst = out if (M == 1 or out.stride(0) == n_out) else torch.empty(M, n_out, dtype=odt, device=x.device)
        _check(lib.mx_gemv(fmt, p0, p1, p2, p3, _p(x), _p(dst), _p(bias), M, w.N, w.K, int(out_f32), act, C.c_float(act_alpha),
                           C.c_float(act_limit), _vp(0), _vp(0), M, 1, _stream()), "gemv")
        if dst is not out:
            out.copy_(dst)
    else:
        xa = _gemm_a(x, w)
        if M >= DEQUANT_ONCE_MIN_M and fmt != int(WFormat.BF16):
            # long chunk, quantised dense weight: decode it once to bf16 and multiply with the TMA-fed kernel (the in-kernel decode
            # repeats per 128-row activation tile).  The scratch matrix is an ordinary allocation: stream-ordered, graph-safe.
            wb = torch.empty(w.N, w.K, dtype=torch.bfloat16, device=x.device)
            _check(lib.mx_dequant_bf16(fmt, p0, p1, p2, p3, C.c_longlong(w.N), w.K, _p(wb), _stream()), "dequant_bf16")
            _count()
            fmt, p0, p1, p2, p3 = int(WFormat.BF16), _p(wb), _vp(0), _vp(0), _vp(0)
        _check(lib.mx_gemm(_p(xa), fmt, p0, p1, p2, p3, 1, _p(out), out.stride(0), int(out_f32), _p(bias), _p(row_scale), act,
                           C.c_float(act_alpha), C.c_float(act_limit), M, w.N, w.K, _vp(0), _vp(0), _pick_bn(M, w.N, wide=fmt == int(WFormat.BF16)), _stream()), "gemm")
    _count()
    return out


def _linear_f32(x, w: QuantWeight, bias, act, act_alpha, act_limit, row_scale, out):
    """fp32 activations: the layer runs in full 32-bit on the CUDA cores (``csrc/cuda/linear_f32.cu``); dense bf16 weights only."""
    if w.fmt != WFormat.BF16 or w.E != 1 or row_scale is not None:
        raise KernelError("32-bit linear layers take dense bf16 weights")
    if act_gated(act):
        y = glu(_linear_f32(x, w, bias, ACT_NONE, 0.0, 0.0, None, None), act, act_alpha, act_limit)
        return y if out is None else out.copy_(y)
    assert x.is_contiguous() and x.shape[-1] == w.K
    M = x.shape[0]
    if out is None:
        out = torch.empty(M, w.N, dtype=torch.float32, device=x.device)
    assert out.shape == (M, w.N) and out.dtype == torch.float32 and (M == 0 or out.stride(1) == 1)
    if M:
        _check(_lib.cuda().mx_linear_f32(_p(x), _p(w.p0), _p(bias), _p(out), M, w.N, w.K, out.stride(0), act, C.c_float(act_alpha), C.c_float(act_limit),
                                         _stream()), "linear_f32")
        _count()
    return out


EXL3_GEMV_MAX_M = 8


def hadamard128(x, pre=None, post=None, bias=None, out_f32=False, out=None):
    """Normalised 128-point Sylvester Hadamard transform of every aligned run of 128 elements of the rows of ``x`` (bf16 or fp32, unit
    column stride): ``had128(x * pre) * post + bias`` with optional fp32 vectors.  ``out``: a [rows, n] view with unit column stride.
    A 3-D fp32 ``x`` [parts, rows, n] (contiguous) stands for the sum of its parts (the partial sums of a K-split product)."""
    nsum, sum_stride = 1, 0
    if x.dim() == 3:
        assert x.dtype == torch.float32 and x.is_contiguous()
        nsum, sum_stride = x.shape[0], x.shape[1] * x.shape[2]
        x = x[0]
    assert x.dim() == 2 and x.stride(1) == 1 and x.dtype in (torch.bfloat16, torch.float32) and x.shape[1] % 128 == 0
    rows, n = x.shape
    odt = torch.float32 if out_f32 else torch.bfloat16
    if out is None:
        out = torch.empty(rows, n, dtype=odt, device=x.device)
    assert out.shape == (rows, n) and out.dtype == odt and (rows == 0 or out.stride(1) == 1)
    for v in (pre, post, bias):
        assert v is None or (v.dtype == torch.float32 and v.numel() == n and v.is_contiguous())
    if rows:
        _check(_lib.cuda().mx_hadamard128_cuda(_p(x), int(x.dtype == torch.float32), _p(pre), _p(post), _p(bias), _p(out), int(out_f32),
                                               C.c_longlong(rows), n, x.stride(0), out.stride(0), nsum, C.c_longlong(sum_stride), _stream()), "hadamard128")
        _count()
    return out


def exl3_dequant(w: QuantWeight) -> torch.Tensor:
    """The rotated weight W_rot of an EXL3 layer as bf16 [N, K] (without the Hadamard transforms and the sign / scale vectors)."""
    assert w.fmt == WFormat.EXL3
    wb = torch.empty(w.N, w.K, dtype=torch.bfloat16, device=w.device)
    _check(_lib.cuda().mx_exl3_dequant_bf16(_p(w.p0), w.K // 16, w.N // 16, w.bits, _p(wb), _stream()), "exl3 dequant")
    _count()
    return wb


def _exl3_linear(x, w: QuantWeight, bias, out_f32, out):
    """y = had128(had128(x * suh) W_rot) * svh + bias: the trellis is decoded in registers for decode-sized batches and once to a bf16
    scratch matrix for the tensor-core GEMM otherwise (src/ops/gemv_exl3.cpp:162 runs the same three steps)."""
    M = x.shape[0]
    lib = _lib.cuda()
    xh = hadamard128(x, pre=w.p1[0])
    if M == 0:
        return hadamard128(torch.empty(0, w.N, dtype=torch.float32, device=x.device), out_f32=out_f32, out=out)
    if M <= EXL3_GEMV_MAX_M:
        # the K tiles are cut into ranges (more CTAs for narrow matrices); the partial sums meet in the Hadamard kernel below
        ranges = lib.mx_exl3_gemv_ranges(w.K // 16, w.N // 16)
        acc = torch.empty(ranges, M, w.N, dtype=torch.float32, device=x.device)
        _check(lib.mx_exl3_gemv(_p(w.p0), w.K // 16, w.N // 16, w.bits, _p(xh), _p(acc), M, ranges, _stream()), "exl3 gemv")
        _count()
    else:
        wb = exl3_dequant(w)
        acc = torch.empty(M, w.N, dtype=torch.float32, device=x.device)
        _check(lib.mx_gemm(_p(xh), int(WFormat.BF16), _p(wb), _vp(0), _vp(0), _vp(0), 1, _p(acc), w.N, 1, _vp(0), _vp(0), ACT_NONE, C.c_float(0.0),
                           C.c_float(0.0), M, w.N, w.K, _vp(0), _vp(0), _pick_bn(M, w.N), _stream()), "gemm")
        _count()
    return hadamard128(acc, post=w.p2[0], bias=bias, out_f32=out_f32, out=out)


def gemm(x, w: QuantWeight, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, out_f32=False, row_scale=None, bn=None):
    """Always the tcgen05 path (tests and benches)."""
    M = x.shape[0]
    n_out = w.N // 2 if act_gated(act) else w.N
    out = torch.empty(M, n_out, dtype=torch.float32 if out_f32 else torch.bfloat16, device=x.device)
    fmt, p0, p1, p2, p3 = _planes(w)
    xa = _gemm_a(x, w)
    _check(_lib.cuda().mx_gemm(_p(xa), fmt, p0, p1, p2, p3, 1, _p(out), n_out, int(out_f32), _p(bias), _p(row_scale), act,
                               C.c_float(act_alpha), C.c_float(act_limit), M, w.N, w.K, _vp(0), _vp(0), bn or _pick_bn(M, w.N), _stream()), "gemm")
    _count()
    return out


def grouped_linear(xp, w: QuantWeight, tile_expert, num_tiles, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, out_f32=False, bn=128,
                   out_dtype=None):
    """``out_dtype`` (bf16 / fp16 / fp32) overrides ``out_f32``; fp16 feeds a following MXFP4 GEMM without a cast."""
    P = xp.shape[0]
    if xp.dtype == torch.float32:            # 32-bit models: every row in fp32 on the CUDA cores
        if w.fmt != WFormat.BF16 or bias is not None or out_dtype not in (None, torch.float32):
            raise KernelError("32-bit grouped layers take bf16 weights without biases")
        if act_gated(act):                   # (rows past the live tiles pass through unread)
            return glu(grouped_linear(xp, w, tile_expert, num_tiles), act, act_alpha, act_limit)
        out = torch.empty(P, w.N, dtype=torch.float32, device=xp.device)
        _check(_lib.cuda().mx_grouped_linear_f32(_p(xp), _p(w.p0), _p(out), P, w.N, w.K, _p(tile_expert), _p(num_tiles), act, C.c_float(act_alpha),
                                                 C.c_float(act_limit), _stream()), "grouped linear_f32")
        _count()
        return out
    n_out = w.N // 2 if act_gated(act) else w.N
    odt = out_dtype or (torch.float32 if out_f32 else torch.bfloat16)
    out = torch.empty(P, n_out, dtype=odt, device=xp.device)
    fmt, p0, p1, p2, p3 = _planes(w)
    xp = _gemm_a(xp, w)
    _check(_lib.cuda().mx_gemm(_p(xp), fmt, p0, p1, p2, p3, w.E, _p(out), n_out, _out_kind(odt), _p(bias), _vp(0), act, C.c_float(act_alpha),
                               C.c_float(act_limit), P, w.N, w.K, _p(tile_expert), _p(num_tiles), bn, _stream()), "grouped gemm")
    _count()
    return out


def expert_gemv(x, w: QuantWeight, slot_expert, x_div=1, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, slot_scale=None, out_f32=False,
                e_lo=0):
    """``w`` holds experts [e_lo, e_lo + w.E); slots routed to other experts produce zero rows (expert parallelism)."""
    S = slot_expert.numel()
    n_out = w.N // 2 if act_gated(act) else w.N
    out = torch.empty(S, n_out, dtype=torch.float32 if out_f32 else torch.bfloat16, device=x.device)
    fmt, p0, p1, p2, p3 = _planes(w)
    _check(_lib.cuda().mx_gemv_experts(fmt, p0, p1, p2, p3, _p(x), _p(out), _p(bias), w.N, w.K, int(out_f32), act, C.c_float(act_alpha),
                                       C.c_float(act_limit), _p(slot_expert), _p(slot_scale), S, x_div, int(e_lo), int(e_lo) + w.E, _stream()),
           "expert gemv")
    _count()
    return out


# ------------------------------------------------------------------ attention
_attn_scratch: dict = {}


TC_PREFILL_MIN_Q = 64      # query segments at least this long take the tensor-core kernel


def _q_rows(q):
    """Elements between query rows: q is [Tq, n_q, dk] with dense heads, possibly a column range of a wider projection."""
    assert q.stride(2) == 1 and (q.shape[1] == 1 or q.stride(1) == q.shape[2])
    return q.stride(0)


def attention_prefill_tc(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks=None, window=0, scale=None, softcap=0.0, q_scale=None,
                         gate=None, keep_first=0):
    """tcgen05 FlashAttention (key / value widths that are multiples of 8 up to 256, page size 128, optional logit soft-cap)."""
    Tq, n_q, hd = q.shape
    n_kv, bs, dv = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    out = torch.empty(Tq, n_q, dv, dtype=torch.bfloat16, device=q.device)
    _check(_lib.cuda().mx_attention_prefill_tc_ext(_p(q), _q_rows(q), _p(k_cache), _p(v_cache), _p(block_table), _p(seq_lens), _p(cu_q), _p(sinks),
                                                   _p(gate), 0 if gate is None else gate.stride(0), _p(q_scale), 0 if q_scale is None else q_scale.numel(),
                                                   _p(out), seq_lens.numel(), Tq, int(max_q_len), n_q, n_kv, hd, dv, block_table.shape[1],
                                                   k_cache.shape[0], bs, int(window), int(keep_first), int(gate is not None and gate.shape[1] == n_q), C.c_float(scale),
                                                   C.c_float(softcap or 0.0), _stream()),
           "attention_prefill_tc")
    _count()
    return out


_kv8_scratch: dict = {}


def _dequant_pages(k_cache, v_cache, kv_scales, block_table, seq_lens, max_kv_len):
    """The pages of this batch of an int8 cache as a bf16 scratch cache [B * nb, n_kv, bs, hd] with its own block table."""
    _, n_kv, bs, hd = k_cache.shape
    B = seq_lens.numel()
    nb = block_table.shape[1] if max_kv_len <= 0 else min(block_table.shape[1], (max_kv_len + bs - 1) // bs)
    need = 2 * B * nb * n_kv * bs * hd
    buf = _kv8_scratch.get(k_cache.device)
    if buf is None or buf.numel() < need:
        buf = torch.zeros(need, dtype=torch.bfloat16, device=k_cache.device)      # zeros: pages that are never filled stay finite
        _kv8_scratch[k_cache.device] = buf
    dk = buf[: need // 2].view(B * nb, n_kv, bs, hd)
    dv = buf[need // 2: need].view(B * nb, n_kv, bs, hd)
    key = (k_cache.device, "table", B, nb)
    table = _kv8_scratch.get(key)
    if table is None:
        table = torch.arange(B * nb, dtype=torch.int32, device=k_cache.device).view(B, nb)
        _kv8_scratch[key] = table
    _check(_lib.cuda().mx_kv_dequant_pages(_p(k_cache), _p(v_cache), _p(kv_scales[0]), _p(kv_scales[1]), _p(block_table), _p(seq_lens),
                                           _p(dk), _p(dv), B, n_kv, bs, hd, block_table.shape[1], nb, _stream()), "kv_dequant_pages")
    _count()
    return dk, dv, table


ATTN_MAX_SPLITS = 32


def _tc_prefill_takes(q, dk, dv, softcap, kv_scales) -> bool:
    if q.dtype != torch.bfloat16:
        return False
    if dk == dv and dk in (64, 128, 256):
        return True
    return kv_scales is None and not softcap and 8 <= dk <= 256 and 8 <= dv <= 256 and dk % 8 == 0 and dv % 8 == 0


def _takes_tc(max_q_len: int, bs: int, dtype, dk: int, dv: int) -> bool:
    """Whether attention over pooled blocks runs on the tensor-core kernel."""
    return max_q_len >= TC_PREFILL_MIN_Q and bs == 128 and dtype == torch.bfloat16 and 8 <= dk <= 256 and 8 <= dv <= 256


def attention_prefill_pooled(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks, window, scale, softcap, gate, pools, dense, out_rope):
    """tcgen05 FlashAttention over a window and the dense pages of pooled blocks that :func:`pool_blocks` has written (None: no query sees one)."""
    Tq, n_q, dk = q.shape
    n_pages, n_kv, bs, dv = v_cache.shape
    cos, sin = out_rope if out_rope is not None else (None, None)
    pk, pv = dense if dense is not None else (None, None)
    out = torch.empty(Tq, n_q, dv, dtype=torch.bfloat16, device=q.device)
    _check(_lib.cuda().mx_attention_prefill_pooled(_p(q), _q_rows(q), _p(k_cache), _p(v_cache), _p(block_table), _p(seq_lens), _p(cu_q), _p(sinks), _p(gate),
                                                   0 if gate is None else gate.stride(0), _p(out), seq_lens.numel(), Tq, int(max_q_len), n_q, n_kv, dk, dv,
                                                   block_table.shape[1], n_pages, bs, int(window), C.c_float(scale), C.c_float(softcap or 0.0), _p(pk), _p(pv),
                                                   pools.pool if dense is not None else 0, 0 if pk is None else pk.shape[0] // seq_lens.numel(), _p(cos), _p(sin),
                                                   0 if cos is None else cos.shape[0], 0 if cos is None else cos.shape[1], _stream()), "attention_prefill_pooled")
    _count()
    return out


def attention(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks=None, window=0, scale=None, softcap=0.0, n_splits=None,
              kv_scales=None, max_kv_len=0, q_scale=None, gate=None, v_width=0, keep_first=0, pools=None, pool_dense=None, out_rope=None):
    """``v_cache`` None: a value is the first ``v_width`` elements of its key row (latent cache)."""
    Tq, n_q, hd = q.shape
    n_kv, bs, dv = k_cache.shape[1], k_cache.shape[2], v_width if v_cache is None else v_cache.shape[3]
    assert k_cache.dtype == torch.int8 or (k_cache.dtype == q.dtype and (v_cache is None or v_cache.dtype == q.dtype))
    assert gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1 and gate.shape in ((Tq, n_q * dv), (Tq, n_q)))
    B = seq_lens.numel()
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    assert (k_cache.dtype == torch.int8) == (kv_scales is not None)
    extended = pools is not None or out_rope is not None
    if extended:
        assert kv_scales is None and v_cache is not None and not keep_first and (gate is None or gate.shape[1] == n_q * dv)
        if n_splits is None and q_scale is None and _takes_tc(max_q_len, bs, q.dtype, hd, dv):
            return attention_prefill_pooled(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks, window, scale, softcap, gate, pools, pool_dense,
                                            out_rope)
    if not extended and max_q_len >= TC_PREFILL_MIN_Q and bs == 128 and n_splits is None and v_cache is not None and _tc_prefill_takes(q, hd, dv, softcap, kv_scales):
        if kv_scales is not None:       # the tensor-core kernel reads bf16 pages: expand this batch's pages first
            dk, dv, table = _dequant_pages(k_cache, v_cache, kv_scales, block_table, seq_lens, max_kv_len)
            return attention_prefill_tc(q, dk, dv, table, seq_lens, cu_q, max_q_len, sinks=sinks, window=window, scale=scale, softcap=softcap,
                                        q_scale=q_scale, gate=gate)
        return attention_prefill_tc(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, sinks=sinks, window=window, scale=scale,
                                    softcap=softcap, q_scale=q_scale, gate=gate, keep_first=keep_first)
    if n_splits is None:
        # decode-sized problems: split the KV range so that ~2 CTAs per SM exist
        ctas = B * n_kv * max(1, (max_q_len * (n_q // n_kv) + 31) // 32)
        max_kv_tiles = max(1, (block_table.shape[1] * bs) // 64)
        # (the cap: with two KV heads of 256 and one sequence, 128 ranges instead of 32 took a 16k context from 119 to 103 us but a 4k
        # context from 48 to 54 us -- the last CTA's merge grows with the ranges; the kernel itself takes any number)
        n_splits = max(1, min(max_kv_tiles, ATTN_MAX_SPLITS, (2 * sm_count()) // max(ctas, 1)))
    need = n_splits * Tq * n_q * (dv + 2)
    if torch.cuda.is_current_stream_capturing():
        # a captured kernel keeps the raw address: the scratch must live exactly as long as the graph, so it comes from the
        # graph's own pool.  (The shared buffer below is re-allocated when a larger request arrives; a graph that had
        # captured its old address would then write through a dangling pointer.)
        buf = torch.empty(need, dtype=torch.float32, device=q.device)
    else:
        buf = _attn_scratch.get(q.device)
        if buf is None or buf.numel() < need:
            buf = torch.empty(max(need, 1 << 20), dtype=torch.float32, device=q.device)
            _attn_scratch[q.device] = buf
    o_part = buf[: n_splits * Tq * n_q * dv]
    ml_part = buf[n_splits * Tq * n_q * dv: need]
    out = torch.empty(Tq, n_q, dv, dtype=q.dtype, device=q.device)
    if kv_scales is not None:
        assert q_scale is None and gate is None and not keep_first and q.is_contiguous(), "the int8 cache has no gated / position-scaled form"
        _check(_lib.cuda().mx_attention_kv8(_p(q), _p(k_cache), _p(v_cache), _p(kv_scales[0]), _p(kv_scales[1]), _p(block_table), _p(seq_lens),
                                            _p(cu_q), _p(sinks), _p(out), _p(o_part), _p(ml_part), B, Tq, int(max_q_len), n_q, n_kv, hd,
                                            block_table.shape[1], bs, int(window), C.c_float(scale), C.c_float(softcap), int(n_splits),
                                            _stream()), "attention_kv8")
    else:
        _check(_lib.cuda().mx_attention_ext(_p(q), _q_rows(q), _p(k_cache), _p(v_cache), _p(block_table), _p(seq_lens), _p(cu_q), _p(sinks), _p(gate),
                                            0 if gate is None else gate.stride(0), _p(q_scale), 0 if q_scale is None else q_scale.numel(), _p(out),
                                            _p(o_part), _p(ml_part), B, Tq, int(max_q_len), n_q, n_kv, hd, dv, block_table.shape[1], bs, int(window),
                                            int(keep_first), int(gate is not None and gate.shape[1] == n_q), C.c_float(scale), C.c_float(softcap), int(n_splits),
                                            int(q.dtype == torch.float32), *((_vp(0), _vp(0), 0, 0) if pools is None else
                                                                             (_p(pools.k), _p(pools.v), pools.pool, pools.k.shape[2])),
                                            *((_vp(0), _vp(0), 0, 0) if out_rope is None else (_p(out_rope[0]), _p(out_rope[1]), *out_rope[0].shape)),
                                            _stream()), "attention")
    _count(_lib.cuda().mx_attention_launches(B, int(max_q_len), n_q, n_kv))
    return out


# ------------------------------------------------------------------ latent attention
def latent_post(q_rot, ckv, norm_w, rank, eps, positions, rope_cos, rope_sin, slot_map, cache, q_out):
    T, H, r = q_rot.shape
    R = norm_w.numel()
    assert q_rot.dtype == ckv.dtype == cache.dtype == q_out.dtype and q_rot.stride(2) == ckv.stride(1) == q_out.stride(2) == 1
    assert cache.is_contiguous() and cache.shape[1] == 1 and cache.shape[3] == R + r == ckv.shape[1] and q_out.shape == q_rot.shape
    _check(_lib.cuda().mx_latent_post(_p(q_rot), q_rot.stride(0), q_rot.stride(1), _p(q_out), q_out.stride(0), q_out.stride(1), _p(ckv), ckv.stride(0),
                                      _p(norm_w), int(rank), C.c_float(eps), _p(positions), _p(rope_cos), _p(rope_sin), rope_cos.shape[1], rope_cos.shape[0],
                                      _p(slot_map), _p(cache), T, H, R, r, int(cache.dtype == torch.float32), _stream()), "latent_post")
    _count()


LATENT_MAX_SPLITS = 64
HEAD_GEMV_MAX_T = 4          # up to this many rows a head's matrix is streamed by the CUDA cores; more go to the tensor cores


def head_linear(x, w: QuantWeight, gate=None, out=None, out_f32=False):
    T, H, K = x.shape
    assert w.fmt == WFormat.BF16 and (w.E, w.K) == (H, K) and x.stride(2) == 1
    odt = torch.float32 if out_f32 else x.dtype
    if out is None:
        out = torch.empty(T, H, w.N, dtype=odt, device=x.device)
    assert out.shape == (T, H, w.N) and out.dtype == odt and out.stride(2) == 1 and (gate is None or (gate.dtype == x.dtype and gate.stride(1) == 1))
    g_ld = 0 if gate is None else gate.stride(0)
    if x.dtype == torch.float32 or T <= HEAD_GEMV_MAX_T:
        _check(_lib.cuda().mx_head_linear(_p(x), C.c_longlong(x.stride(0)), x.stride(1), _p(w.p0), _p(gate), g_ld, _p(out), C.c_longlong(out.stride(0)),
                                          out.stride(1), T, H, w.N, K, int(x.dtype == torch.float32), int(odt == torch.float32), _stream()), "head_linear")
    else:
        tiles = H * ((T + 127) // 128)
        bn = next((b for b in (128, 64, 32) if tiles * ((w.N + b - 1) // b) >= sm_count()), 32)
        _check(_lib.cuda().mx_gemm_heads(_p(x), x.stride(0), C.c_longlong(x.stride(1)), _p(w.p0), _p(out), out.stride(0), C.c_longlong(out.stride(1)), _p(gate),
                                         g_ld, T, H, w.N, K, bn, int(out_f32), _stream()), "gemm_heads")
    _count()
    return out


STACK_GEMV_MAX_ROWS = 8      # up to this many rows in all matrices together stream their matrix each; more take the tensor-core kernel
_stack_slots: dict = {}


def stacked_linear(x, w: QuantWeight):
    n, T, K = x.shape
    assert x.is_contiguous() and w.fmt == WFormat.BF16 and (w.E, w.K) == (n, K)
    if x.dtype == torch.float32:
        out = torch.empty(n, T, w.N, dtype=x.dtype, device=x.device)
        for i in range(n):
            _linear_f32(x[i], QuantWeight(WFormat.BF16, w.N, K, 1, w.p0[i:i + 1]), None, ACT_NONE, 0.0, 0.0, None, out[i])
        return out
    if n * T <= STACK_GEMV_MAX_ROWS:
        if (n, T, x.device) not in _stack_slots:
            _stack_slots[n, T, x.device] = torch.arange(n, dtype=torch.int32, device=x.device).repeat_interleave(T).contiguous()
        return expert_gemv(x.view(n * T, K), w, _stack_slots[n, T, x.device]).view(n, T, w.N)
    out = torch.empty(n, T, w.N, dtype=x.dtype, device=x.device)
    _check(_lib.cuda().mx_gemm_heads(_p(x), K, C.c_longlong(T * K), _p(w.p0), _p(out), w.N, C.c_longlong(T * w.N), _vp(0), 0, T, n, w.N, K,
                                     _stack_bn(n, T, w.N), 0, _stream()), "gemm_heads")
    _count()
    return out


def _stack_bn(n: int, T: int, N: int) -> int:
    rows = n * ((T + 127) // 128)
    if T > 128:
        return _pick_bn(rows * 128, N, wide=True)
    return next((b for b in (128, 64, 32) if rows * ((N + b - 1) // b) >= sm_count()), 32)


def latent_attention(q, cache, block_table, seq_lens, cu_q, max_q_len, rank, window=0, scale=1.0, n_splits=None):
    Tq, H, width = q.shape
    B, bs = seq_lens.numel(), cache.shape[2]
    if q.dtype == torch.float32:
        return attention(q, cache, None, block_table, seq_lens, cu_q, max_q_len, window=window, scale=scale, n_splits=n_splits, v_width=rank)
    assert q.is_contiguous() and cache.is_contiguous() and q.dtype == cache.dtype == torch.bfloat16 and cache.shape[1:] == (1, 128, width)
    out = torch.empty(Tq, H, rank, dtype=q.dtype, device=q.device)
    if n_splits is None:
        # ranges of whole pages, so that about one CTA per SM exists
        pages = block_table.shape[1] if window <= 0 else min(block_table.shape[1], (window + max_q_len + bs - 3) // bs + 1)
        rows = max_q_len * H
        ctas = B * ((rows + 63) // 64 if rows > 32 else 1)
        n_splits = max(1, min(pages, LATENT_MAX_SPLITS, sm_count() // ctas))
    part = torch.empty(n_splits * Tq * H * (rank + 2), dtype=torch.float32, device=q.device) if n_splits > 1 else None
    ml = part[n_splits * Tq * H * rank:] if part is not None else None
    _check(_lib.cuda().mx_latent_attention(_p(q), _p(cache), cache.shape[0], _p(block_table), block_table.shape[1], _p(seq_lens), _p(cu_q), _p(out), _p(part),
                                           _p(ml), B, Tq, int(max_q_len), H, int(rank), width - rank, int(window), C.c_float(scale), int(n_splits), _stream()),
           "latent_attention")
    _count()
    if n_splits > 1:
        _check(_lib.cuda().mx_attention_combine(_p(part), _p(ml), _p(out), Tq, H, int(rank), int(n_splits), _stream()), "attention_combine")
        _count()
    return out


def _latent_plan(plans, block_table, seq_lens, cu_q, Tq, window, bs):
    """(page list, number of live pages, table of the expanded pages) of the batch; one per window and forward."""
    key = (window, block_table.data_ptr())
    if plans is not None and key in plans:
        return plans[key]
    B, mb = block_table.shape
    # a segment of n queries reaches n + window - 1 keys: at most n / bs + (window - 2) / bs + 2 pages
    most = B * mb if window <= 0 else min(B * mb, Tq // bs + 1 + B * ((window + bs - 3) // bs + 2))
    buf = torch.empty(most + B * mb + 1, dtype=torch.int32, device=block_table.device)
    pages, table, num = buf[:most], buf[most:most + B * mb], buf[most + B * mb:]
    _check(_lib.cuda().mx_latent_plan(_p(block_table), _p(seq_lens), _p(cu_q), B, mb, bs, int(window), most, _p(pages), _p(table), _p(num), _stream()), "latent_plan")
    _count()
    if plans is not None:
        plans[key] = (pages, num, table)
    return pages, num, table


def latent_attention_expanded(q, w_kv: QuantWeight, cache, block_table, seq_lens, cu_q, max_q_len, dim, vdim, rank, window=0, scale=1.0, gate=None,
                              out=None, plans=None):
    Tq, H, dq = q.shape
    bs, width = cache.shape[2], cache.shape[3]
    assert q.dtype == cache.dtype == torch.bfloat16 and bs == 128 and cache.is_contiguous() and w_kv.fmt == WFormat.BF16 and block_table.is_contiguous()
    assert (w_kv.N, w_kv.K) == (H * (dim + vdim), rank) and dq - dim == width - rank
    if out is None:
        out = torch.empty(Tq, H, vdim, dtype=q.dtype, device=q.device)
    assert out.is_contiguous() and out.shape == (Tq, H, vdim)
    plan = _latent_plan(plans, block_table, seq_lens, cu_q, Tq, window, bs)
    kv = torch.empty(plan[0].numel() * bs, w_kv.N, dtype=torch.bfloat16, device=q.device)
    gemm_paged(cache, plan, w_kv, kv)
    return expanded_attention(q, kv, plan, cache, block_table, seq_lens, cu_q, max_q_len, dim, vdim, rank, window, scale, gate, out)


def gemm_paged(cache, plan, w: QuantWeight, out) -> None:
    """Rows of ``plan``'s pages of a latent cache (their first ``w.K`` elements) times ``w``, page after page into ``out``."""
    pages, num, _ = plan
    bs, width = cache.shape[2], cache.shape[3]
    _check(_lib.cuda().mx_gemm_paged(_p(cache), width, C.c_longlong(cache.shape[0] * bs), _p(pages), _p(num), _p(w.p0), _p(out), pages.numel(), w.N, w.K,
                                     _pick_bn(pages.numel() * bs, w.N, wide=True), _stream()), "gemm_paged")
    _count()


def expanded_attention(q, kv, plan, cache, block_table, seq_lens, cu_q, max_q_len, dim, vdim, rank, window, scale, gate, out):
    """The attention of :func:`latent_attention_expanded` over keys and values ``kv`` that :func:`gemm_paged` has formed."""
    pages, _, table = plan
    Tq, H, dq = q.shape
    _check(_lib.cuda().mx_attention_prefill_latent(_p(q), _q_rows(q), _p(kv), pages.numel(), _p(table), _p(cache), cache.shape[0], _p(block_table),
                                                   block_table.shape[1], _p(seq_lens), _p(cu_q), _p(gate), 0 if gate is None else gate.stride(0), _p(out),
                                                   seq_lens.numel(), Tq, int(max_q_len), H, dim, dq - dim, vdim, rank, int(window), C.c_float(scale), _stream()),
           "attention_prefill_latent")
    _count()
    return out


# ------------------------------------------------------------------ MoE
def moe_route(logits, bias, k, renorm=True, precise=False, sigmoid=False, experts=None):
    T, ld = logits.shape
    E = experts or ld
    assert logits.is_contiguous() and logits.dtype == torch.float32
    idx = torch.empty(T, k, dtype=torch.int32, device=logits.device)
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    _check(_lib.cuda().mx_moe_route(_p(logits), _p(bias), T, E, k, 2 if sigmoid else int(renorm), int(precise), ld, _p(idx), _p(w), _stream()), "moe_route")
    _count()
    return idx, w


def moe_pack(topk_idx, E, e_lo=0, e_hi=None, tile=MOE_TILE):
    e_hi = E if e_hi is None else e_hi
    T, K = topk_idx.shape
    dev = topk_idx.device
    n = T * K
    max_rows = moe_max_rows(n, e_hi - e_lo) if tile > 1 else max(n, 1)
    counts = torch.empty(E, dtype=torch.int32, device=dev)
    seg = torch.empty(E + 1, dtype=torch.int32, device=dev)
    packed_token = torch.empty(max_rows, dtype=torch.int32, device=dev)
    pair_to_packed = torch.empty(n, dtype=torch.int32, device=dev)
    tile_expert = torch.zeros(max(max_rows // MOE_TILE, 1), dtype=torch.int32, device=dev)
    tile_valid = torch.zeros(max(max_rows // MOE_TILE, 1), dtype=torch.int32, device=dev) if tile > 1 else None
    num_tiles = torch.empty(2, dtype=torch.int32, device=dev)
    _check(_lib.cuda().mx_moe_pack(_p(topk_idx), n, K, E, e_lo, e_hi, _p(counts), _p(seg), _p(packed_token), _p(pair_to_packed),
                                   _p(tile_expert), _p(num_tiles), max_rows, int(tile), _p(tile_valid), _stream()), "moe_pack")
    _count()
    return MoePacking(counts, seg, packed_token, pair_to_packed, tile_expert, num_tiles, max_rows, K, tile_valid)


@_profiled("moe_quant")
def moe_quant(x, rows, max_tiles, rows_per_tile, src_index=None, x_div=1, row_limit=None):
    """bf16 rows -> MXFP8 rows + scale atoms for :func:`mxf4_gemm` (see ``mx_moe_quant``).  Returns (xq [rows, KB*128] uint8,
    sfx [KB, max_tiles, 512] uint8).  Rows that are skipped (negative index, beyond ``row_limit``) are left unwritten."""
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1
    K = x.shape[1]
    KB = (K + 127) // 128
    xq = torch.empty(rows, KB * 128, dtype=torch.uint8, device=x.device)
    sfx = torch.empty(KB, max_tiles, 512, dtype=torch.uint8, device=x.device)
    _check(_lib.cuda().mx_moe_quant(_p(x), x.stride(0), _p(src_index), int(x_div), _p(row_limit), int(rows), K, int(max_tiles),
                                    int(rows_per_tile), _p(xq), _p(sfx), _stream()), "moe_quant")
    _count()
    return xq, sfx


@_profiled("moe_route_quant")
def moe_route_quant(logits, bias, k, x, renorm=True, w_copies=1):
    """Decode: router top-k and pair-mode MXFP8 quantisation of the T rows of ``x`` in one launch.  Returns (idx, w, xq, sfx); ``w`` is
    [T, w_copies * k], the k weights repeated (one per partial row when the down projection splits K)."""
    T, E = logits.shape
    Kd = x.shape[1]
    KB = (Kd + 127) // 128
    n = T * k
    idx = torch.empty(T, k, dtype=torch.int32, device=logits.device)
    w = torch.empty(T, w_copies * k, dtype=torch.float32, device=logits.device)
    xq = torch.empty(n, KB * 128, dtype=torch.uint8, device=x.device)
    sfx = torch.empty(KB, n, 512, dtype=torch.uint8, device=x.device)
    _check(_lib.cuda().mx_moe_route_quant(_p(logits), _p(bias), T, E, k, int(renorm), _p(idx), _p(w), int(w_copies), _p(x), x.stride(0), Kd, n, _p(xq), _p(sfx),
                                          _stream()), "moe_route_quant")
    _count()
    return idx, w, xq, sfx


GEMV_NORM_MAX_M = 2      # the fused prologue normalises its rows one after the other; more rows take the separate kernel


@_profiled("gemv_norm")
def gemv_norm(x, norm_w, eps, w: QuantWeight, bias=None, delta=None, one_plus_w=False, delta_scale=1.0, out_f32=False, want_h=False, route=None):
    """Decode (at most GEMV_NORM_MAX_M rows of at most 4096 elements): residual add + RMSNorm + dense GEMV in one launch (``csrc/cuda/gemv_stream.cu``).  ``x`` fp32 [T, H] is
    not modified; ``delta`` is None, a bf16 [T, H] tensor or a :class:`CombineDelta`.  Returns None when the shape or the weight format
    is not taken, else ``(y, x_new, h)``: the product, the updated residual (``x`` itself without a delta) and, with ``want_h``, the
    normalised rows.  ``route = (router_bias, k, renorm, w_copies)`` makes ``w`` the router: the last CTA also picks the top-k experts
    and writes the rows as MXFP8 pair tiles, and the result is ``(logits, x_new, h, idx, topk_w, xq, sfx)`` with ``topk_w`` of shape
    [T, w_copies * k] (the k weights repeated: one per partial row when the down projection splits K)."""
    T, H = x.shape
    if T > GEMV_NORM_MAX_M or H > 4096 or w.E != 1 or w.fmt not in (WFormat.BF16, WFormat.Q8) or x.dtype != torch.float32 or not x.is_contiguous():
        return None
    comb = delta if isinstance(delta, CombineDelta) else None
    if delta is not None and comb is None and not (isinstance(delta, torch.Tensor) and delta.dtype == torch.bfloat16 and delta.is_contiguous()):
        return None
    if comb is not None and comb.w.shape[1] > 8:
        return None
    dev = x.device
    fmt, p0, p1, _, _ = _planes(w)
    y = torch.empty(T, w.N, dtype=torch.float32 if (out_f32 or route is not None) else torch.bfloat16, device=dev)
    x_new = torch.empty_like(x) if delta is not None else x
    h = torch.empty(T, H, dtype=torch.bfloat16, device=dev) if want_h else None
    idx = tw = xq = sfx = None
    rb, k, renorm, n, copies = None, 0, 1, 0, 1
    if route is not None:
        rb, k, renorm, copies = route
        KB = (H + 127) // 128
        n = T * k
        idx = torch.empty(T, k, dtype=torch.int32, device=dev)
        tw = torch.empty(T, copies * k, dtype=torch.float32, device=dev)
        xq = torch.empty(n, KB * 128, dtype=torch.uint8, device=dev)
        sfx = torch.empty(KB, n, 512, dtype=torch.uint8, device=dev)
    rc = _lib.cuda().mx_gemv_norm(fmt, p0, p1, _p(x), _p(x_new) if delta is not None else _vp(0), _p(delta) if (delta is not None and comb is None) else _vp(0),
                                  _p(comb.y) if comb is not None else _vp(0), _p(comb.pair_to_packed) if comb is not None else _vp(0),
                                  _p(comb.w) if comb is not None else _vp(0), comb.w.shape[1] if comb is not None else 0, _p(norm_w), C.c_float(eps),
                                  int(one_plus_w), C.c_float(delta_scale), _p(h), _p(y), _p(bias), T, w.N, w.K, int(y.dtype == torch.float32),
                                  int(route is not None), _p(rb), k, int(bool(renorm)), _p(idx), _p(tw), copies, _p(xq), _p(sfx), n, _stream())
    if rc == 1:
        return None
    _check(rc, "gemv_norm")
    _count()
    if route is not None:
        return y, x_new, h, idx, tw, xq, sfx
    return y, x_new, h


def mxf4_ksplit(K: int, want: int) -> int:
    """K ranges ``mxf4_gemm(..., ksplit=want)`` really uses for a reduction length K: every range owns at least one 128-element block."""
    kb = (K + 127) // 128
    per = (kb + max(want, 1) - 1) // max(want, 1)
    return (kb + per - 1) // per


@_profiled("mxf4_gemm")
def mxf4_gemm(w: QuantWeight, xq, sfx, tile_expert, max_tiles, row_stride, tile_valid=None, default_valid=128, num_tiles=None, e_lo=0,
              bias0=None, bias1=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, zero_out=False, ksplit=1):
    """Block-scaled MXFP4 x MXFP8 grouped GEMM on the tensor cores (``csrc/cuda/gemm_mxf4.cu``).  ``w`` is an MXF4T bank and
    ``xq``/``sfx`` come from :func:`moe_quant` or from a gated call of this function.  A plain bank returns bf16 [rows, N]; a gated
    pair (``w.dual``, with ``act``) returns the activation already quantised for the next projection: (oq [rows, N rounded up to
    128] uint8, osf scale atoms).  Rows that belong to no live tile are left unwritten unless ``zero_out``.  ``ksplit`` > 1 (plain banks):
    K is cut into that many ranges and the result has ``ksplit`` x rows rows, range s in rows [s * rows, (s + 1) * rows): partial sums
    that the consumer adds (decode, where a handful of pairs would otherwise leave most SMs idle)."""
    assert w.fmt == WFormat.MXF4T
    rows = xq.shape[0]
    dev = xq.device
    out = oq = osf = None
    oq_ld = 0
    if w.dual:
        oq_ld = (w.N + 127) // 128 * 128
        oq = torch.empty(rows, oq_ld, dtype=torch.uint8, device=dev)
        osf = torch.empty(oq_ld // 128, max_tiles, 512, dtype=torch.uint8, device=dev)
    else:
        ksplit = mxf4_ksplit(w.K, ksplit)
        out = (torch.zeros if zero_out else torch.empty)(ksplit * rows, w.N, dtype=torch.bfloat16, device=dev)
    _check(_lib.cuda().mx_mxf4_gemm(_p(w.p0), _p(w.p1), int(w.dual), w.E, _p(xq), _p(sfx), rows, w.N, w.K, _p(tile_expert), _p(tile_valid),
                                    int(default_valid), _p(num_tiles), int(max_tiles), int(row_stride), int(e_lo), _p(bias0), _p(bias1),
                                    _p(out), w.N, _p(oq), _p(osf), oq_ld, int(act), C.c_float(act_alpha), C.c_float(act_limit), int(ksplit), _stream()),
           "mxf4 gemm")
    _count()
    return (oq, osf) if w.dual else out


def expert_group_gemv(x, w: QuantWeight, pk: MoePacking, x_index=None, bias=None, act=ACT_NONE, act_alpha=1.702, act_limit=7.0, e_lo=0):
    """Batched-decode MoE GEMV over a compact packing (``moe_pack(..., tile=1)``): every local expert streams its weights once
    and multiplies them with all rows routed to it (8 rows per pass).  Row r of the output belongs to packed position r;
    its input is ``x[x_index[r]]`` (gate|up reads the token rows in place) or ``x[r]`` (down)."""
    P = pk.max_rows
    n_out = w.N // 2 if act_gated(act) else w.N
    out = torch.empty(P, n_out, dtype=torch.bfloat16, device=x.device)
    fmt, p0, p1, p2, p3 = _planes(w)
    _check(_lib.cuda().mx_gemv_group(fmt, p0, p1, p2, p3, _p(x), _p(x_index), _p(out), _p(bias), w.N, w.K, act, C.c_float(act_alpha),
                                     C.c_float(act_limit), _p(pk.counts), _p(pk.seg_start), int(e_lo), w.E, _stream()), "gemv_group")
    _count()
    return out


def moe_gather(x, pk: MoePacking, f16=False, zero_pad=False):
    """Rows of ``x`` in packed order.  Padding rows of the expert tiles are left unwritten unless ``zero_pad`` (no consumer reads them:
    a grouped GEMM row depends on its own input row only)."""
    H = x.shape[1]
    assert x.is_contiguous() and (x.dtype == torch.bfloat16 or (x.dtype == torch.float32 and not f16))
    xp = torch.empty(pk.max_rows, H, dtype=torch.float16 if f16 else x.dtype, device=x.device)
    _check(_lib.cuda().mx_moe_gather(_p(x), _p(pk.packed_token), _p(pk.num_tiles), _p(xp), H * (x.element_size() // 2), pk.max_rows, int(f16), int(zero_pad), _stream()), "moe_gather")
    _count()
    return xp


def moe_scale_rows(x, w, pk: Optional[MoePacking] = None):
    T, K = w.shape
    H = x.shape[1]
    assert x.is_contiguous() and x.shape[0] == T and w.dtype == torch.float32 and w.is_contiguous()
    xp = torch.empty(T * K if pk is None else pk.max_rows, H, dtype=x.dtype, device=x.device)
    _check(_lib.cuda().mx_moe_scale_rows(_p(x), _p(w), _p(None if pk is None else pk.pair_to_packed), _p(xp), T * K, H, K, int(x.dtype == torch.float32),
                                         _stream()), "moe_scale_rows")
    _count()
    return xp


def moe_combine(yp, pk: MoePacking, w, out=None, accumulate=False):
    T, K = w.shape
    H = yp.shape[1]
    if out is None:
        out = torch.empty(T, H, dtype=torch.float32, device=yp.device)
        accumulate = False
    _check(_lib.cuda().mx_moe_combine(_p(yp), int(yp.dtype == torch.float32), _p(pk.pair_to_packed), _p(w), _p(out), int(out.dtype == torch.float32), T, H, K,
                                      int(accumulate), _stream()), "moe_combine")
    _count()
    return out


# ------------------------------------------------------------------ sampling
def argmax(logits):
    rows, V = logits.shape
    out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    _check(_lib.cuda().mx_argmax(_p(logits), rows, V, logits.stride(0), _p(out), _stream()), "argmax")
    _count()
    return out


def rep_penalty(logits, ids, penalty):
    rows, V = logits.shape
    _check(_lib.cuda().mx_rep_penalty(_p(logits), rows, V, logits.stride(0), _p(ids), ids.shape[1], _p(penalty), _stream()), "rep_penalty")
    _count()
    return logits


def sample(logits, temperature, top_k, top_p, min_p, rng):
    rows, V = logits.shape
    out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    _check(_lib.cuda().mx_sample(_p(logits), rows, V, logits.stride(0), _p(temperature), _p(top_k), _p(top_p), _p(min_p), _p(rng), _p(out),
                                 _stream()), "sample")
    _count()
    return out
