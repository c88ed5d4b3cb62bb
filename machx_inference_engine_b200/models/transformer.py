"""One decoder-only graph for the attention-based families: dense Llama / Qwen2 / Qwen3 / Mistral /
Phi-3 / Granite, Qwen3-MoE and gpt-oss (attention sinks, alternating sliding window, biased
projections, clamped SwiGLU, MXFP4 experts).  Hybrid (gated-DeltaNet) layers plug in through
``models/hybrid.py``.

The graph is config-driven instead of one class per family: the reference copies its dense
forward for every architecture (src/model/dense_transformer.cpp:381-744, gptoss.cpp:312-523,
qwen3moe.cpp) and again for every parallel form (dense_tp.cpp, gptoss_tp.cpp, qwen3moe_tp.cpp);
here parallelism is a property of the linear layers (:class:`ParallelCtx`).

Per layer the launch sequence is
  rmsnorm(+residual) -> qkv GEMM -> qkv_post (bias, QK-norm, RoPE, paged KV write) -> attention
  -> o GEMM [-> all-reduce] -> rmsnorm(+residual) -> FFN (gate|up GEMM with fused activation,
  down GEMM) or MoE (router GEMM, top-k, pack, gather, grouped GEMMs, combine) [-> all-reduce].
The residual stream is fp32, activations bf16; nothing goes back to the host inside forward.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..formats.model_config import ModelConfig
from ..ops import ACT_GEGLU, ACT_NONE, ACT_SWIGLU, ACT_SWIGLU_OAI, QuantWeight
from ..ops.weights import WFormat
from ..parallel.comm import ParallelCtx
from ..utils.rope import rope_tables

KV_BLOCK = 128


@dataclass
class ForwardBatch:
    """Device-side description of one step (prefill chunk(s), decode tokens, or a mix)."""
    ids: torch.Tensor            # int32 [T]
    positions: torch.Tensor      # int32 [T]
    slot_map: torch.Tensor       # int64 [T]  block*KV_BLOCK + offset, <0 = do not cache
    block_table: torch.Tensor    # int32 [B, max_blocks]
    seq_lens: torch.Tensor       # int32 [B]  kv length after this step
    cu_q: torch.Tensor           # int32 [B+1]
    max_q_len: int
    logit_rows: Optional[torch.Tensor] = None   # int64 rows of the T tokens that need logits (None: last of each sequence)
    state_slots: Optional[torch.Tensor] = None  # int32 [B] recurrent-state slot per sequence (hybrid models)
    state_slots_host: Optional[list] = None     # host copy of state_slots
    q_lens_host: Optional[list] = None          # host copy of per-sequence query lengths (hybrid scan scheduling)
    start_host: Optional[list] = None           # host copy of per-sequence start positions (0 = fresh state)
    want_hidden: bool = False                   # also return the pre-final-norm hidden rows (MTP)
    max_kv_len: int = 0                         # host copy of max(seq_lens); 0 = unknown (the block table's capacity is assumed)
    short: Optional[tuple] = None               # (sequences, rows, longest query) of the leading short ones, when short and long queries meet in a batch

    @property
    def T(self) -> int:
        return self.ids.numel()

    @property
    def B(self) -> int:
        return self.seq_lens.numel()

    def query_parts(self, apart: bool = True) -> list:
        """[(first row, end row, block table, sequence lengths, cu_q, longest query)]: the batch, or (``apart``) its short and its long queries
        (cu_q keeps the rows of the whole batch)."""
        if self.short is None or not apart:
            return [(0, self.T, self.block_table, self.seq_lens, self.cu_q, self.max_q_len)]
        n, rows, longest = self.short
        return [(0, rows, self.block_table[:n], self.seq_lens[:n], self.cu_q[:n + 1], longest),
                (rows, self.T, self.block_table[n:], self.seq_lens[n:], self.cu_q[n:], self.max_q_len)]


class KVCache:
    """Paged KV: per attention layer ``k, v [num_blocks, n_kv_local, KV_BLOCK, head_dim]`` bf16 or fp32, or int8 with one fp32 scale
    per (block, kv head, token) row in ``ks, vs [num_blocks, n_kv_local, KV_BLOCK]`` (value = q * scale, scale = max|x| / 127).
    ``geometry`` gives layers their own (n_kv, head_dim) or (n_kv, key width, value width); a value width of 0 is a latent cache, whose
    values are formed from the key rows.  A layer that runs several times has one entry per run.  ``pools`` {layer: (tokens per block, window)} gives
    layers rows for pooled blocks in every page (``pools[layer]``, :class:`ops.PoolPages`): they live and die with the page, so sharing and reuse of
    pages cover them.

    The reference cache is contiguous per sequence (include/ie/kv_cache.hpp:27-114) and keeps int8 rows beside it when
    ``--int8-kv`` is given (src/core/kv_cache.cpp:182-240, src/ops/attention.cpp:145-229); pages make continuous batching
    and block-level prefix sharing possible, and here the int8 rows replace the bf16 ones instead of shadowing them.
    """

    BLOCK = KV_BLOCK

    def __init__(self, n_layers: int, num_blocks: int, n_kv: int, head_dim: int, device, attn_layers: Optional[list[int]] = None,
                 dtype: str = "bf16", geometry: Optional[dict] = None, pools: Optional[dict] = None):
        if dtype not in ("bf16", "fp32", "int8"):
            raise ValueError(f"unknown KV cache dtype {dtype!r}")
        self.num_blocks = num_blocks
        self.block_size = KV_BLOCK
        self.dtype = dtype
        layers = attn_layers if attn_layers is not None else list(range(n_layers))
        td = {"bf16": torch.bfloat16, "fp32": torch.float32, "int8": torch.int8}[dtype]
        geo = {l: ((geometry or {}).get(l) or (n_kv, head_dim)) for l in layers}       # per layer: Gemma-4 mixes two, Tikarax lists them
        self.k = {l: torch.zeros(num_blocks, geo[l][0], KV_BLOCK, geo[l][1], dtype=td, device=device) for l in layers}
        self.v = {l: torch.zeros(num_blocks, geo[l][0], KV_BLOCK, geo[l][-1], dtype=td, device=device) for l in layers}
        rows = lambda l, width: torch.zeros(num_blocks, geo[l][0], ops.PoolPages.rows_per_page(KV_BLOCK, pools[l][0]), width, dtype=td, device=device)
        self.pools = {l: ops.PoolPages(rows(l, geo[l][1]), rows(l, geo[l][-1]), *pools[l]) for l in (pools or {})}
        self.ks = {l: torch.ones(num_blocks, geo[l][0], KV_BLOCK, dtype=torch.float32, device=device) for l in layers} if dtype == "int8" else None
        self.vs = {l: torch.ones(num_blocks, geo[l][0], KV_BLOCK, dtype=torch.float32, device=device) for l in layers} if dtype == "int8" else None

    def scales(self, layer: int):
        return (self.ks[layer], self.vs[layer]) if self.ks is not None else None

    @staticmethod
    def bytes_per_block(n_attn_layers: int, n_kv: int, head_dim: int, dtype: str = "bf16") -> int:
        per_row = head_dim * 2 if dtype == "bf16" else head_dim + 4
        return 2 * n_attn_layers * n_kv * KV_BLOCK * per_row

    def copy_blocks(self, src: list[int], dst: list[int]) -> None:
        if not src:
            return
        s = torch.tensor(src, dtype=torch.long, device=next(iter(self.k.values())).device)
        d = torch.tensor(dst, dtype=torch.long, device=s.device)
        for l in self.k:
            self.k[l][d] = self.k[l][s]
            self.v[l][d] = self.v[l][s]
            for t in (self.pools[l].k, self.pools[l].v) if l in self.pools else ():
                t[d] = t[s]
            if self.ks is not None:
                self.ks[l][d] = self.ks[l][s]
                self.vs[l][d] = self.vs[l][s]


# ---------------------------------------------------------------------------------------------
class Linear:
    """y = x W^T (+b).  ``reduce`` marks a row-parallel layer whose output is a partial sum."""

    def __init__(self, w: QuantWeight, bias: Optional[torch.Tensor] = None, act: int = ACT_NONE, act_alpha: float = 1.702,
                 act_limit: float = 7.0, reduce: bool = False):
        self.w, self.bias, self.act, self.act_alpha, self.act_limit, self.reduce = w, bias, act, act_alpha, act_limit, reduce

    def __call__(self, x: torch.Tensor, par: Optional[ParallelCtx] = None, out_f32: bool = False, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        if out is not None:        # (column-parallel projections only: a caller-provided slice of a shared output)
            return ops.linear(x, self.w, bias=self.bias, act=self.act, act_alpha=self.act_alpha, act_limit=self.act_limit, out_f32=out_f32, out=out)
        if self.reduce and par is not None and par.enabled:
            # the bias of a row-parallel layer is added once, after the reduction
            if par.fused is not None and x.is_cuda:
                return par.fused.linear_all_reduce(x, self.w, self.bias)
            y = par.all_reduce(ops.linear(x, self.w, out_f32=True))
            return y if self.bias is None else y + self.bias
        return ops.linear(x, self.w, bias=self.bias, act=self.act, act_alpha=self.act_alpha, act_limit=self.act_limit, out_f32=out_f32)


class MultiLinear:
    """Column-concatenation of linears whose weights have different storage formats (e.g. Q4_K q/k with Q6_K v)."""

    def __init__(self, parts: list[Linear]):
        self.parts = parts
        self.widths = [p.w.N // 2 if ops.act_gated(p.act) else p.w.N for p in parts]

    def __call__(self, x, par=None, out_f32=False):
        # every part writes its own column slice of one output (no concatenation pass)
        out = torch.empty(x.shape[0], sum(self.widths), dtype=torch.float32 if out_f32 else torch.bfloat16, device=x.device)
        lo = 0
        for p, n in zip(self.parts, self.widths):
            p(x, par, out_f32, out=out[:, lo:lo + n])
            lo += n
        return out


def _fuse_rows(ws: list[QuantWeight], biases: list[Optional[torch.Tensor]]):
    if all(w.fmt == ws[0].fmt for w in ws) and ws[0].fmt != WFormat.EXL3:
        b = None
        if any(bb is not None for bb in biases):
            b = torch.cat([bb if bb is not None else torch.zeros(w.N, device=w.device) for w, bb in zip(ws, biases)])
        return Linear(QuantWeight.cat_rows(ws), b)
    return MultiLinear([Linear(w, b) for w, b in zip(ws, biases)])


def unpermute_llama_qk(w: QuantWeight, n_heads: int, head_dim: int) -> QuantWeight:
    """GGUF ``llama`` files store Q/K rows interleaved for pairwise RoPE; the kernels rotate NEOX
    half-splits, so rows are regrouped: dest h*hd + b*hd/2 + k  <-  src h*hd + 2k + b
    (src/model/dense_transformer.cpp:24-32,130-137)."""
    hd = head_dim
    k = torch.arange(hd // 2)
    src = torch.cat([2 * k, 2 * k + 1])                       # b = 0 block then b = 1 block
    idx = (torch.arange(n_heads).unsqueeze(1) * hd + src.unsqueeze(0)).reshape(-1)
    return w.select_rows(idx)


class AttentionBlock:
    def __init__(self, cfg: ModelConfig, layer: int, src, par: ParallelCtx, prefix: Optional[str] = None, q_gate: bool = False):
        c = cfg
        p = prefix or f"blk.{layer}"
        if c.arch == "gemma4":           # per-layer head geometry: the rest of this constructor sees a config of this layer's shape
            from dataclasses import replace
            hd_l, n_kv_l, n_rot_l, _ = c.layer_geometry(layer)
            c = replace(c, head_dim=hd_l, n_kv_heads=n_kv_l, n_rot=n_rot_l)
        hd, H = c.head_dim, c.hidden
        tp = par.world if par.mode == "tp" else 1
        self.layer = layer
        self.q_gate = q_gate
        self.n_q = c.n_heads // tp
        if c.n_heads % tp:
            raise ValueError(f"{c.n_heads} attention heads do not split over {tp} ranks")
        # KV heads: shard when they divide, otherwise each rank keeps the one head its query heads use
        if c.n_kv_heads >= tp:
            if c.n_kv_heads % tp:
                raise ValueError(f"{c.n_kv_heads} KV heads do not split over {tp} ranks")
            self.n_kv = c.n_kv_heads // tp
            kv_lo = par.rank * self.n_kv if tp > 1 else 0
        else:
            self.n_kv = 1
            kv_lo = (par.rank * c.n_kv_heads) // tp
        q_lo = (par.rank * self.n_q) if tp > 1 else 0
        q_rows_per_head = hd * (2 if q_gate else 1)

        if c.arch == "phi3" and not src.has(f"{p}.attn_q.weight"):
            # Phi-3 files keep one fused attn_qkv matrix: q rows, then k rows, then v rows
            nq_rows, nkv_rows = c.n_heads * hd, c.n_kv_heads * hd
            fused = src.matrix(f"{p}.attn_qkv.weight", nq_rows + 2 * nkv_rows, H)
            wq, wk, wv = fused.slice_rows(0, nq_rows), fused.slice_rows(nq_rows, nq_rows + nkv_rows), fused.slice_rows(nq_rows + nkv_rows, nq_rows + 2 * nkv_rows)
        else:
            wq = src.matrix(f"{p}.attn_q.weight", c.n_heads * q_rows_per_head, H)
            wk = src.matrix(f"{p}.attn_k.weight", c.n_kv_heads * hd, H)
            has_v = True
            if c.arch == "gemma4":       # files simply lack attn_v on the global layers; random-init graphs decide by the pattern
                has_v = src.has(f"{p}.attn_v.weight") if getattr(src, "r", None) is not None else bool(c.layer_swa[layer])
            if not has_v:
                wv = wk                  # V is the raw K projection (src/model/gemma4.cpp:178-183,660)
            else:
                wv = src.matrix(f"{p}.attn_v.weight", c.n_kv_heads * hd, H)
        if c.arch == "llama" and getattr(src, "r", None) is not None and wq.fmt != WFormat.EXL3:
            # (imported EXL3 layers keep the Hugging Face row order, which is the half-split one: src/model/dense_transformer.cpp:165-212)
            wq, wk = unpermute_llama_qk(wq, c.n_heads, hd), unpermute_llama_qk(wk, c.n_kv_heads, hd)
        has_bias = c.arch in ("qwen2", "gpt-oss") and src.has(f"{p}.attn_q.bias")
        bq = src.vector(f"{p}.attn_q.bias", c.n_heads * q_rows_per_head) if has_bias else None
        bk = src.vector(f"{p}.attn_k.bias", c.n_kv_heads * hd) if has_bias else None
        bv = src.vector(f"{p}.attn_v.bias", c.n_kv_heads * hd) if has_bias else None
        sl = lambda w, lo, n: w if (lo == 0 and n == w.N) else w.slice_rows(lo, lo + n)
        sb = lambda b, lo, n: None if b is None else b[lo:lo + n].contiguous()
        ws = [sl(wq, q_lo * q_rows_per_head, self.n_q * q_rows_per_head), sl(wk, kv_lo * hd, self.n_kv * hd), sl(wv, kv_lo * hd, self.n_kv * hd)]
        bs = [sb(bq, q_lo * q_rows_per_head, self.n_q * q_rows_per_head), sb(bk, kv_lo * hd, self.n_kv * hd), sb(bv, kv_lo * hd, self.n_kv * hd)]
        self.qkv = _fuse_rows(ws, bs)
        wo = src.matrix(f"{p}.attn_output.weight", H, c.n_heads * hd)
        bo = src.vector(f"{p}.attn_output.bias", H) if (c.arch == "gpt-oss" and src.has(f"{p}.attn_output.bias")) else None
        if tp > 1:
            wo = wo.slice_k(q_lo * hd, (q_lo + self.n_q) * hd, requant=True)
        self.o = Linear(wo, bo, reduce=tp > 1)
        qk_norm = c.arch in ("qwen3", "qwen3moe", "qwen3next", "qwen35", "qwen35moe", "gemma4") and src.has(f"{p}.attn_q_norm.weight")
        self.v_norm = c.arch == "gemma4"       # weightless RMS norm on V (src/model/gemma4.cpp:663)
        self.q_norm = src.vector(f"{p}.attn_q_norm.weight", hd) if qk_norm else None
        self.k_norm = src.vector(f"{p}.attn_k_norm.weight", hd) if qk_norm else None
        self.sinks = None
        if c.arch == "gpt-oss":
            s = src.vector(f"{p}.attn_sinks.weight", c.n_heads)
            self.sinks = s[q_lo:q_lo + self.n_q].contiguous()
        self.window = c.layer_window(layer)
        self.scale = c.attention_scale if c.attention_scale > 0 else 1.0 / math.sqrt(hd)
        self.hd, self.n_rot, self.eps = hd, c.n_rot, c.rms_eps
        self.norm_one_plus_w = c.arch in ("qwen35", "qwen35moe")      # Qwen3-Next files store 1 + w already

    def __call__(self, h: torch.Tensor, fb: ForwardBatch, kv: KVCache, rope, par: ParallelCtx) -> torch.Tensor:
        return self.attend(self.qkv(h), fb, kv, rope, par)

    def attend(self, qkv: torch.Tensor, fb: ForwardBatch, kv: KVCache, rope, par: ParallelCtx) -> torch.Tensor:
        """Everything after the qkv projection: head epilogue + cache write, attention, output projection."""
        q, gate = ops.qkv_post(qkv, None, self.q_norm, self.k_norm, fb.positions, rope[0], rope[1], fb.slot_map, kv.k[self.layer],
                               kv.v[self.layer], self.n_q, self.n_kv, self.hd, self.n_rot, q_gate=self.q_gate,
                               norm_one_plus_w=self.norm_one_plus_w, eps=self.eps, kv_scales=kv.scales(self.layer),
                               **({"v_norm": True} if self.v_norm else {}))
        a = ops.attention(q, kv.k[self.layer], kv.v[self.layer], fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, sinks=self.sinks,
                          window=self.window, scale=self.scale, kv_scales=kv.scales(self.layer), max_kv_len=fb.max_kv_len)
        a = a.reshape(a.shape[0], self.n_q * self.hd)
        if gate is not None:
            a = ops.sigmoid_mul(a, gate.reshape(a.shape))
        return self.o(a, par)


def _attn_gathered(self, sc, T: int, gbuf: int, fb: ForwardBatch, kv: KVCache, rope, par: ParallelCtx):
    """Row-sharded prefill: qkv on the gathered rows (all-gather -> GEMM), attention over this rank's heads, and the output
    projection with the reduce-scatter epilogue (each row's partial goes to the rank that owns the row)."""
    qkv = sc.linear_gathered(self.qkv, T, gbuf)
    q, gate = ops.qkv_post(qkv, None, self.q_norm, self.k_norm, fb.positions, rope[0], rope[1], fb.slot_map, kv.k[self.layer],
                           kv.v[self.layer], self.n_q, self.n_kv, self.hd, self.n_rot, q_gate=self.q_gate,
                           norm_one_plus_w=self.norm_one_plus_w, eps=self.eps, kv_scales=kv.scales(self.layer),
                           **({"v_norm": True} if self.v_norm else {}))
    a = ops.attention(q, kv.k[self.layer], kv.v[self.layer], fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, sinks=self.sinks,
                      window=self.window, scale=self.scale, kv_scales=kv.scales(self.layer), max_kv_len=fb.max_kv_len)
    a = a.reshape(a.shape[0], self.n_q * self.hd)
    if gate is not None:
        a = ops.sigmoid_mul(a, gate.reshape(a.shape))
    return par.fused.linear_all_reduce(a, self.o.w, self.o.bias, rs_rows=T // par.world)


AttentionBlock.forward_gathered = _attn_gathered


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class NoRopeAttentionBlock:
    """Attention without rotation: separate key and value widths, biased q / k / v, a query temperature given as a table over positions
    (folded into the fp32 scores) and a sigmoid output gate that reads the block's own input.

    One projection produces the columns [q | k | v | gate]; the queries and the gate are read in place by the attention kernel (which
    applies the gate as it writes), only K and V are moved, into the cache pages.  Head widths are padded to multiples of 8 at load."""

    def __init__(self, src, prefix: str, layer: int, hidden: int, row: int, heads: int, kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 q_scale: Optional[torch.Tensor] = None):
        self.layer, self.n_q, self.n_kv, self.scale, self.q_scale = layer, heads, kv_heads, scale, q_scale
        self.dk, self.dv = round_up(key_dim, 8), round_up(value_dim, 8)
        H = hidden

        def rows(name, n, d, dp, biased=True):
            w = src.matrix(f"{prefix}.{name}", n * d, H).pad_groups(rows=(n, dp), cols=(1, row))
            b = torch.zeros(n, dp, dtype=torch.float32, device=w.device)
            if biased:
                b[:, :d] = src.vector(f"{prefix}.{name}.b", n * d).reshape(n, d)
            return w, b.reshape(-1)

        parts = [rows("q", heads, key_dim, self.dk), rows("k", kv_heads, key_dim, self.dk), rows("v", kv_heads, value_dim, self.dv),
                 rows("g", heads, value_dim, self.dv, biased=False)]
        self.proj = _fuse_rows([w for w, _ in parts], [b for _, b in parts])
        ends = [0]
        for w, _ in parts:
            ends.append(ends[-1] + w.N)
        self.cols = ends
        wo = src.matrix(f"{prefix}.o", H, heads * value_dim).pad_groups(rows=(1, row), cols=(heads, self.dv))
        self.o = Linear(wo)

    def __call__(self, h: torch.Tensor, fb: ForwardBatch, kv: KVCache) -> torch.Tensor:
        y = self.proj(h)
        T, c, l = y.shape[0], self.cols, self.layer
        ops.kv_store(y[:, c[1]:c[2]], y[:, c[2]:c[3]], fb.slot_map, kv.k[l], kv.v[l])
        a = ops.attention(y[:, :c[1]].view(T, self.n_q, self.dk), kv.k[l], kv.v[l], fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, scale=self.scale,
                          max_kv_len=fb.max_kv_len, q_scale=self.q_scale, gate=y[:, c[3]:])
        return self.o(a.reshape(T, self.n_q * self.dv))


class LatentAttentionBlock:
    """Attention over a cached latent: one row per token, [c | r], serves all heads.  A head's key is [W_uk c | r] with the rotated part r shared
    by the heads, its value W_uv c; sliding window; sigmoid output gate that reads the block's own input.

    One projection produces the columns [q: per head unrotated | rotated | c, r | gate].  Short queries (decoding, small portions) stay in the
    latent space: q is taken through W_uk^T once, the kernel reads each cached row once for all heads and as key and value, and W_uv follows.
    Long queries form the keys and values of the pages in reach once per step and run on the prefill kernel, which costs a head (dim + rot_dim +
    vdim) products per key and query where the latent space costs 2 rank + rot_dim.  Widths are padded to multiples of 8 at load."""

    EXPAND_MIN_Q = 64            # query segments at least this long take per-head keys and values ...
    EXPAND_MAX = (192, 64, 256)  # ... when the widths (unrotated, rotated, value) fit that kernel; otherwise all stay in the latent space
    MAX_RANK = 512               # what the latent kernel's accumulators hold

    def __init__(self, src, prefix: str, hidden: int, row: int, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float, window: int,
                 eps: float, rope: tuple):
        if rank > self.MAX_RANK:
            raise ValueError(f"{prefix}: a latent of {rank} elements is wider than the {self.MAX_RANK} the kernels take")
        H, K = heads, hidden
        self.n_q, self.n_kv, self.scale, self.window, self.eps, self.rank, self.rope = H, 1, scale, window, eps, rank, rope
        self.d, self.r, self.v, self.R = (round_up(n, 8) for n in (dim, rot_dim, vdim, rank))
        self.can_expand = all(n <= m for n, m in zip((self.d, self.r, self.v), self.EXPAND_MAX))

        def padded(w: QuantWeight, parts, sizes, row_to):
            """Rows of every group are ``parts`` runs; each run is padded to its size, the columns to ``row_to``."""
            t = (w if w.fmt == WFormat.BF16 else QuantWeight(**_as_bf16(w))).p0[0]
            t = t.reshape(-1, sum(parts), t.shape[-1])
            out = torch.zeros(t.shape[0], sum(sizes), row_to, dtype=t.dtype, device=t.device)
            lo = at = 0
            for n, m in zip(parts, sizes):
                out[:, at:at + n, :t.shape[2]] = t[:, lo:lo + n]
                lo, at = lo + n, at + m
            return out

        stack = lambda t: QuantWeight(WFormat.BF16, t.shape[1], t.shape[2], t.shape[0], t.contiguous())
        flat = lambda t: t.reshape(1, -1, t.shape[-1])
        q = padded(src.matrix(f"{prefix}.q", H * (dim + rot_dim), K), (dim, rot_dim), (self.d, self.r), row)
        ckv = padded(src.matrix(f"{prefix}.dkv", rank + rot_dim, K), (rank, rot_dim), (self.R, self.r), row)
        g = padded(src.matrix(f"{prefix}.g", H * vdim, K), (vdim,), (self.v,), row)
        self.proj = Linear(stack(torch.cat([flat(q), flat(ckv), flat(g)], dim=1)))
        self.cols = (H * (self.d + self.r), H * (self.d + self.r) + self.R + self.r)
        uk = padded(src.matrix(f"{prefix}.uk", H * dim, rank), (dim,), (self.d,), self.R)
        uv = padded(src.matrix(f"{prefix}.uv", H * vdim, rank), (vdim,), (self.v,), self.R)
        self.kv_up = stack(torch.cat([flat(uk), flat(uv)], dim=1))          # keys of all heads, then values
        self.absorb = stack(uk.transpose(1, 2))                               # per head [R, d]
        self.v_up = QuantWeight(WFormat.BF16, self.v, self.R, H, self.kv_up.p0[0, H * self.d:].view(H, self.v, self.R))
        self.norm = torch.zeros(self.R, dtype=torch.float32, device=uk.device)
        self.norm[:rank] = src.vector(f"{prefix}.dkv.norm", rank)
        self.o = Linear(src.matrix(f"{prefix}.o", K, H * vdim).pad_groups(rows=(1, row), cols=(H, self.v)))

    def __call__(self, h: torch.Tensor, fb: ForwardBatch, cache: torch.Tensor, plans: dict) -> torch.Tensor:
        y = self.proj(h)
        T, H, d, R = y.shape[0], self.n_q, self.d, self.R
        q, ckv, gate = y[:, :self.cols[0]].view(T, H, d + self.r), y[:, self.cols[0]:self.cols[1]], y[:, self.cols[1]:]
        a = torch.empty(T, H, self.v, dtype=y.dtype, device=y.device)
        expand = self.can_expand and not (y.is_cuda and y.dtype == torch.float32)          # (32-bit kernels: latent space only)
        for lo, hi, table, lens, cu, longest in fb.query_parts(apart=expand):
            latent = longest < self.EXPAND_MIN_Q or not expand
            rows = slice(lo, hi)
            qc = torch.empty(hi - lo, H, R + self.r, dtype=y.dtype, device=y.device) if latent else None
            ops.latent_post(q[rows, :, d:], ckv[rows], self.norm, self.rank, self.eps, fb.positions[rows], self.rope[0], self.rope[1], fb.slot_map[rows],
                            cache, qc[..., R:] if latent else q[rows, :, d:])
            if latent:               # (the latent part of a batch starts at its first row)
                ops.head_linear(q[rows, :, :d], self.absorb, out=qc[..., :R])
                o = ops.latent_attention(qc, cache, table, lens, cu, longest, R, window=self.window, scale=self.scale)
                ops.head_linear(o, self.v_up, gate=gate[rows], out=a[rows])
            else:
                ops.latent_attention_expanded(q, self.kv_up, cache, table, lens, cu, longest, d, self.v, R, window=self.window, scale=self.scale,
                                              gate=gate, out=a, plans=plans)
        return self.o(a.view(T, H * self.v))


class KeyValueAttentionBlock:
    """Attention whose values are its keys as projected (before norm and rotation): no value projection.  Rotation of part of a head in either pairing,
    per-head RMS norms of queries and keys with a weight before it or without one after it, sliding window that may keep the first tokens of the
    sequence, an optional score of 0 in the softmax denominator (``zero_sink``) and an optional output gate of one number per head.

    One projection gives the columns [q | k | gate]; the queries are rotated where they stand, keys and values go into the cache pages.  ``parts`` are the
    projection's row blocks, so that a mixer that reads the same input can share it.  Head widths are padded to multiples of 8 at load."""

    MAX_DIM = 512

    def __init__(self, src, prefix: str, layer: int, hidden: int, row: int, heads: int, kv_heads: int, dim: int, scale: float, window: int, keep_first: int,
                 rot_dim: int, rope: tuple, eps: float, interleaved: bool = False, biased: bool = False, qk_norm: bool = False, norm_after: bool = False,
                 head_gate: bool = False, zero_sink: bool = False):
        self.layer, self.n_q, self.n_kv, self.dim, self.scale, self.eps = layer, heads, kv_heads, dim, scale, eps
        self.window, self.keep_first = window, keep_first
        self.rot_dim, self.rope, self.interleaved, self.norm_after = rot_dim, rope, interleaved, norm_after
        dp = self.dp = round_up(dim, 8)
        if dp > self.MAX_DIM:
            raise ValueError(f"{prefix}: heads of {dim} elements are wider than the {self.MAX_DIM} the kernels take")

        def rows(name, n, d, to):
            w = src.matrix(f"{prefix}.{name}", n * d, hidden).pad_groups(rows=(n, to), cols=(1, row))
            if not biased:
                return w, None
            b = torch.zeros(n, to, dtype=torch.float32, device=w.device)
            b[:, :d] = src.vector(f"{prefix}.{name}.b", n * d).reshape(n, d)
            return w, b.reshape(-1)

        self.parts = [rows("q", heads, dim, dp), rows("k", kv_heads, dim, dp)]
        self.gate_at = (heads + kv_heads) * dp if head_gate else None
        if head_gate:
            self.parts.append((src.matrix(f"{prefix}.g", heads, hidden).pad_groups(rows=(1, round_up(heads, 8)), cols=(1, row)), None))
        self.columns = sum(w.N for w, _ in self.parts)
        norm = lambda n: torch.nn.functional.pad(src.vector(f"{prefix}.{n}.norm", dim), (0, dp - dim)).contiguous()
        self.q_norm, self.k_norm = (norm("q"), norm("k")) if qk_norm else (None, None)
        self.sinks = torch.zeros(heads, dtype=torch.float32, device=self.parts[0][0].device) if zero_sink else None
        self.o = Linear(src.matrix(f"{prefix}.o", hidden, heads * dim).pad_groups(rows=(1, row), cols=(heads, dp)))
        self.proj = None

    def own_projection(self) -> "KeyValueAttentionBlock":
        self.proj, self.parts = _fuse_rows(*map(list, zip(*self.parts))), None
        return self

    def __call__(self, h: torch.Tensor, fb: ForwardBatch, kv: KVCache) -> torch.Tensor:
        return self.attend(self.proj(h), fb, kv)

    def attend(self, y: torch.Tensor, fb: ForwardBatch, kv: KVCache) -> torch.Tensor:
        """y: this block's columns of the projection."""
        T, nq, dp, l = y.shape[0], self.n_q * self.dp, self.dp, self.layer
        q = ops.qk_post(y[:, :nq].unflatten(1, (self.n_q, dp)), y[:, nq:nq + self.n_kv * dp].unflatten(1, (self.n_kv, dp)), fb.positions, self.rope[0],
                        self.rope[1], fb.slot_map, kv.k[l], kv.v[l], self.dim, self.rot_dim, interleaved=self.interleaved, q_norm=self.q_norm,
                        k_norm=self.k_norm, norm_after=self.norm_after, eps=self.eps)
        gate = y[:, self.gate_at:self.gate_at + self.n_q] if self.gate_at is not None else None
        a = ops.attention(q, kv.k[l], kv.v[l], fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, sinks=self.sinks, window=self.window, scale=self.scale,
                          max_kv_len=fb.max_kv_len, gate=gate, keep_first=self.keep_first)
        return self.o(a.reshape(T, nq))


def pair_order(n: int, rot: int) -> torch.Tensor:
    """Order of a head's n elements in which the planes (i, i + rot / 2) of a half-split rotation stand side by side; elements past ``rot`` stay."""
    half = torch.arange(rot // 2)
    return torch.cat([torch.stack([half, half + rot // 2], dim=1).reshape(-1), torch.arange(rot, n)])


class PooledAttentionBlock:
    """Attention over a sliding window of tokens and, before it, over pooled blocks (one key and value for ``pool`` tokens), all in one softmax.  Keys of
    width ``dim`` rotated over ``rot_dim`` elements, values rotated over their whole width and cached so, each head's output turned back by its own position;
    a factor per head on the scores (folded into the queries behind the rotation), soft-capped scores, a learned sink per head, sigmoid output gate that
    reads the block's own input.

    One projection gives the columns [q | k | v | gate]; queries and gate are read in place by the attention kernel (which turns the output back and gates
    it as it writes).  Scores do not depend on the order of a head's elements, nor the output on that of its value elements when the output projection's
    columns follow: both are reordered at load so that the half-split planes become neighbouring pairs.  Head widths are padded to multiples of 8."""

    MAX_DIM = 512

    def __init__(self, src, prefix: str, hidden: int, row: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, softcap: float,
                 rot_dim: int, rope: tuple, v_rope: tuple):
        if max(dim, vdim) > self.MAX_DIM:
            raise ValueError(f"{prefix}: heads of {max(dim, vdim)} elements are wider than the {self.MAX_DIM} the kernels take")
        self.n_q, self.n_kv, self.dim, self.scale, self.window, self.softcap = heads, kv_heads, dim, scale, window, softcap
        self.rot_dim, self.rope, self.v_rope = rot_dim, rope, v_rope
        self.dk, self.dv = round_up(dim, 8), round_up(vdim, 8)
        index = lambda n, d, rot: (torch.arange(n).unsqueeze(1) * d + pair_order(d, rot)).reshape(-1)

        def rows(name, n, d, rot, to, biased=True):
            at = index(n, d, rot)
            w = src.matrix(f"{prefix}.{name}", n * d, hidden)
            w = w.select_rows(at.to(w.device)).pad_groups(rows=(n, to), cols=(1, row))
            b = torch.zeros(n, to, dtype=torch.float32, device=w.device)
            if biased:
                b[:, :d] = src.vector(f"{prefix}.{name}.b", n * d)[at.to(w.device)].reshape(n, d)
            return w, b.reshape(-1)

        parts = [rows("q", heads, dim, rot_dim, self.dk), rows("k", kv_heads, dim, rot_dim, self.dk), rows("v", kv_heads, vdim, vdim, self.dv),
                 rows("g", heads, vdim, vdim, self.dv, biased=False)]
        self.proj = _fuse_rows(*map(list, zip(*parts)))
        ends = [0]
        for w, _ in parts:
            ends.append(ends[-1] + w.N)
        self.cols = ends
        self.temp, self.sinks = src.vector(f"{prefix}.temp", heads), src.vector(f"{prefix}.sink", heads)
        wo = src.matrix(f"{prefix}.o", hidden, heads * vdim)
        if wo.fmt != WFormat.BF16:
            wo = QuantWeight(**_as_bf16(wo))
        wo = QuantWeight(WFormat.BF16, wo.N, wo.K, 1, wo.p0[..., index(heads, vdim, vdim).to(wo.device)].contiguous())
        self.o = Linear(wo.pad_groups(rows=(1, row), cols=(heads, self.dv)))

    def __call__(self, h: torch.Tensor, fb: ForwardBatch, kv: KVCache, run: int) -> torch.Tensor:
        """``run``: which of the cache's entries (a layer that runs several times has one per run)."""
        y = self.proj(h)
        T, c, k, v, pools, dense = y.shape[0], self.cols, kv.k[run], kv.v[run], kv.pools.get(run), None
        one_each = fb.max_q_len == 1             # a block that a single token sees first is formed beside its head epilogue
        q = ops.qk_post(y[:, :c[1]].unflatten(1, (self.n_q, self.dk)), y[:, c[1]:c[2]].unflatten(1, (self.n_kv, self.dk)), fb.positions, self.rope[0],
                        self.rope[1], fb.slot_map, k, v, self.dim, self.rot_dim, interleaved=True, v=y[:, c[2]:c[3]].unflatten(1, (self.n_kv, self.dv)),
                        v_rope=self.v_rope, q_scale=self.temp, pools=pools if one_each else None, block_table=fb.block_table)
        if pools is not None and not one_each:
            dense = ops.pool_blocks(k, v, pools, fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, max_kv_len=fb.max_kv_len)
        a = ops.attention(q, k, v, fb.block_table, fb.seq_lens, fb.cu_q, fb.max_q_len, sinks=self.sinks, window=self.window, scale=self.scale,
                          softcap=self.softcap, max_kv_len=fb.max_kv_len, gate=y[:, c[3]:], pools=pools, pool_dense=dense, out_rope=self.v_rope)
        return self.o(a.reshape(T, self.n_q * self.dv))


class GatedFFN:
    """down(act(gate h, up h)), the gate and up rows interleaved for the projection's epilogue."""

    def __init__(self, src, prefix: str, hidden: int, row: int, ffn: int, act: int = ACT_SWIGLU, act_alpha: float = 1.702, act_limit: float = 7.0):
        f = round_up(ffn, 32)
        g, u = (src.matrix(f"{prefix}.{n}", ffn, hidden).pad_groups(rows=(1, f), cols=(1, row)) for n in ("gate", "up"))
        self.gate_up = Linear(QuantWeight.interleave_gate_up(g, u), act=act, act_alpha=act_alpha, act_limit=act_limit)
        self.down = Linear(src.matrix(f"{prefix}.down", hidden, ffn).pad_groups(rows=(1, row), cols=(1, f)))

    def __call__(self, h):
        return self.down(self.gate_up(h))


class UnaryFFN:
    """down(act(up h)): a feed-forward without a gate branch; the activation runs in the up projection's epilogue."""

    def __init__(self, src, prefix: str, hidden: int, row: int, ffn: int, act: int, act_a: float = 0.0, act_b: float = 0.0):
        f = round_up(ffn, 32)
        self.up = Linear(src.matrix(f"{prefix}.up", ffn, hidden).pad_groups(rows=(1, f), cols=(1, row)), act=act, act_alpha=act_a, act_limit=act_b)
        self.down = Linear(src.matrix(f"{prefix}.down", hidden, ffn).pad_groups(rows=(1, row), cols=(1, f)))

    def __call__(self, h):
        return self.down(self.up(h))


class DenseFFN:
    def __init__(self, cfg: ModelConfig, layer: int, src, par: ParallelCtx, prefix: Optional[str] = None, act: int = ACT_SWIGLU,
                 ffn: Optional[int] = None, suffix: str = ""):
        p = prefix or f"blk.{layer}"
        H, F = cfg.hidden, ffn or cfg.ffn
        tp = par.world if par.mode == "tp" else 1
        if cfg.arch == "phi3" and not src.has(f"{p}.ffn_gate{suffix}.weight"):
            up2 = src.matrix(f"{p}.ffn_up{suffix}.weight", 2 * F, H)            # fused gate|up rows
            g, u = up2.slice_rows(0, F), up2.slice_rows(F, 2 * F)
        else:
            g = src.matrix(f"{p}.ffn_gate{suffix}.weight", F, H)
            u = src.matrix(f"{p}.ffn_up{suffix}.weight", F, H)
        d = src.matrix(f"{p}.ffn_down{suffix}.weight", H, F)
        if tp > 1:
            gran = max(d.k_granule(), 16)
            if F % gran or (F // gran) < tp:
                gran = 32 if F % 32 == 0 else 16          # finer than the weight's blocks: the shard is re-encoded
            lo, hi = _even_chunks(F, tp, gran)[par.rank]
            g, u, d = g.slice_rows(lo, hi), u.slice_rows(lo, hi), d.slice_k(lo, hi, requant=True)
        if g.fmt == u.fmt and g.fmt != WFormat.EXL3:
            self.gate_up = Linear(QuantWeight.interleave_gate_up(g, u), act=act)
            self.split = None
        else:
            self.gate_up = None
            self.split = (Linear(g), Linear(u))
            self.act = act
        self.down = Linear(d, reduce=tp > 1)

    def __call__(self, h, par):
        if self.gate_up is not None:
            a = self.gate_up(h)
        else:
            g, u = self.split[0](h), self.split[1](h)
            F = g.shape[1]
            il = torch.cat([g.reshape(-1, F // 16, 16), u.reshape(-1, F // 16, 16)], dim=2).reshape(-1, 2 * F)
            a = ops.glu(il.contiguous(), self.act)
        return self.down(a, par)


def _ffn_gathered(self, sc, T: int, gbuf: int, par: ParallelCtx):
    if self.gate_up is not None:
        a = sc.linear_gathered(self.gate_up, T, gbuf)
    else:
        g, u = sc.linear_gathered(self.split[0], T, gbuf), sc.linear_gathered(self.split[1], T, gbuf)
        F = g.shape[1]
        il = torch.cat([g.reshape(-1, F // 16, 16), u.reshape(-1, F // 16, 16)], dim=2).reshape(-1, 2 * F)
        a = ops.glu(il.contiguous(), self.act)
    return par.fused.linear_all_reduce(a, self.down.w, self.down.bias, rs_rows=T // par.world)


DenseFFN.forward_gathered = _ffn_gathered


def _even_chunks(n: int, parts: int, gran: int) -> list[tuple[int, int]]:
    """Split n (a multiple of gran) into `parts` contiguous ranges on gran boundaries, sizes differing by <= gran."""
    blocks = n // gran
    base, extra = divmod(blocks, parts)
    out, lo = [], 0
    for r in range(parts):
        sz = (base + (1 if r < extra else 0)) * gran
        out.append((lo, lo + sz))
        lo += sz
    return out


class MoEFFN:
    """Router -> top-k -> experts -> weighted combine, expert-parallel over the ranks of ``par``.

    Every rank sees every token (activations are replicated under tensor parallelism), packs only
    the pairs routed to its own experts and contributes a partial sum that the caller reduces.
    """

    MXF4_TENSOR_CORE = True      # class switch (tests compare against the bf16-activation path by turning it off)
    EXPERT_TP = False            # True: split every expert's FFN width over the ranks even when the expert count divides (tests)
    PAIR_GEMV_MAX_TOKENS = 8     # up to this many tokens every (token, expert) pair streams its expert in a GEMV slot; more are packed
    MXF4_PAIR_MAX_TOKENS = 8     # up to this many tokens every (token, expert) pair is its own tile: no packing pass
    DOWN_KSPLIT = 3              # one-token decode: K ranges of the down projection (their partial rows are summed by the combine)

    def __init__(self, cfg: ModelConfig, layer: int, src, par: ParallelCtx, act: int, with_bias: bool, prefix: Optional[str] = None):
        c = cfg
        p = prefix or f"blk.{layer}"
        H, F, E = c.hidden, c.expert_ffn, c.n_experts
        ep = par.world if par.mode == "tp" else 1
        # Experts are sharded whole (expert parallelism) when their count divides by the ranks.  Otherwise (or with EXPERT_TP) every
        # rank keeps all experts and a slice of each one's FFN width, cut on the 32-element blocks of the quantised formats and not
        # necessarily even (src/model/gptoss_tp.cpp:343-354 in the reference): gate / up rows [lo, hi), the matching input columns of
        # down, the down bias on rank 0 only; every rank then holds a partial sum for every pair, reduced like any row-parallel output.
        self.expert_tp = ep > 1 and (E % ep != 0 or self.EXPERT_TP)
        self.E, self.K = E, c.n_experts_used
        self.e_lo, self.e_hi = (par.rank * (E // ep), (par.rank + 1) * (E // ep)) if (ep > 1 and not self.expert_tp) else (0, E)
        rng = (self.e_lo, self.e_hi)
        f_lo, f_hi = 0, F
        if self.expert_tp:
            if F % 32 or F // 32 < ep:
                raise ValueError(f"expert FFN width {F} cannot be cut into {ep} slices of whole 32-element blocks")
            f_lo, f_hi = _even_chunks(F, ep, 32)[par.rank]
        rw = src.matrix(f"{p}.ffn_gate_inp.weight", E, H)
        self.router = Linear(rw if rw.fmt == ops.WFormat.BF16 else QuantWeight(**_as_bf16(rw)))
        self.router_bias = src.vector(f"{p}.ffn_gate_inp.bias", E) if with_bias else None
        if c.arch == "gemma4":           # one bank [E, gate rows | up rows, H] (src/model/gemma4.cpp:267-289)
            gu = src.matrix(f"{p}.ffn_gate_up_exps.weight", 2 * F, H, E, experts=rng)
            g, u = gu.slice_rows(0, F), gu.slice_rows(F, 2 * F)
            del gu
        else:
            g = src.matrix(f"{p}.ffn_gate_exps.weight", F, H, E, experts=rng)
            u = src.matrix(f"{p}.ffn_up_exps.weight", F, H, E, experts=rng)
        d = src.matrix(f"{p}.ffn_down_exps.weight", H, F, E, experts=rng)
        if self.expert_tp:
            g, u, d = g.slice_rows(f_lo, f_hi), u.slice_rows(f_lo, f_hi), d.slice_k(f_lo, f_hi, requant=True)
        # MXFP4 banks on a GPU run on the block-scaled tensor-core kernel: gate / up / down stay three banks in its tiled layout
        self.mx = None
        # all-MXFP4 expert banks multiply MXFP8 activations (e4m3 + a power-of-two scale per 32): the arithmetic of the block-scaled
        # tensor-core kernel, and the arithmetic the CPU path restates so that both produce the same numbers
        self.a8 = g.fmt == u.fmt == d.fmt == ops.WFormat.MXFP4 and act in (ACT_SWIGLU, ACT_SWIGLU_OAI) and self.MXF4_TENSOR_CORE
        if g.p0.is_cuda and self.a8:
            from ..ops.weights import to_mxf4_tiles
            self.mx = (to_mxf4_tiles(g, u), to_mxf4_tiles(d))
            self.gate_up = self.down = None
        else:
            self.gate_up = QuantWeight.interleave_gate_up(g, u)
            self.down = d
        del g, u, d
        # banks past the device's expert budget live in host memory and are staged per forward (models/spill.py)
        self._spill = None
        from . import spill as _spill_mod
        sp = _spill_mod.active()
        if sp is not None:
            banks = list(self.mx) if self.mx is not None else [self.gate_up, self.down]
            if not sp.admit(sum(b.nbytes for b in banks)):
                self._spill = (sp, [sp.to_host(i, b) for i, b in enumerate(banks)])
                self._stage_banks()
        self.expert_scale = None         # optional per-expert factor on the down projection's output, folded into the routing weight
        self.gu_bias = self.down_bias = self.g_bias = self.u_bias = None
        if with_bias:
            gb = src.table(f"{p}.ffn_gate_exps.bias", (E, F))[self.e_lo:self.e_hi, f_lo:f_hi]
            ub = src.table(f"{p}.ffn_up_exps.bias", (E, F))[self.e_lo:self.e_hi, f_lo:f_hi]
            F = f_hi - f_lo
            n = self.e_hi - self.e_lo
            if self.mx is not None:
                self.g_bias, self.u_bias = gb.contiguous(), ub.contiguous()
            else:
                self.gu_bias = torch.cat([gb.reshape(n, F // 16, 16), ub.reshape(n, F // 16, 16)], dim=2).reshape(n, 2 * F).contiguous()
            self.down_bias = src.table(f"{p}.ffn_down_exps.bias", (E, H))[self.e_lo:self.e_hi].contiguous()
            if self.expert_tp and par.rank != 0:
                self.down_bias = torch.zeros_like(self.down_bias)      # the bias joins the reduced sum once
        self.act = act
        self.reduce = ep > 1
        self.group_gemv_max_tokens = 0   # > 0: batches of up to that many tokens take the expert-major GEMV path
        self.shared = None          # optional always-on expert (hybrid families): its partial joins the sum before the reduction
        self._arange = {}

    LAZY_COMBINE = False         # the graph's norm takes an expert combine that has not been formed (ops.cuda.CombineDelta)

    def _lazy(self, h) -> bool:
        return self.LAZY_COMBINE and h.is_cuda and ops.backend() != "torch" and self.shared is None and not self.reduce and self.K <= 32

    def _stage_banks(self) -> None:
        """Spilled layer: copy the banks from host memory into the shared staging area and point the layer at them."""
        sp, host = self._spill
        banks = [sp.fetch(i, b) for i, b in enumerate(host)]
        if self.mx is not None:
            self.mx = (banks[0], banks[1])
        else:
            self.gate_up, self.down = banks

    def __call__(self, h: torch.Tensor, par: ParallelCtx, router_h: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Returns this rank's fp32 contribution [T, H] (already reduced when EP > 1).  ``router_h``: the router's own input
        when it differs from the experts' (Gemma-4)."""
        if self._spill is not None:
            self._stage_banks()
        T = h.shape[0]
        pre = None
        ksplit = 1
        if not isinstance(router_h, tuple):
            logits = self.router(h if router_h is None else router_h, out_f32=True)
        if isinstance(router_h, tuple):
            # decode: the router GEMV's launch has already routed and quantised the rows (ops.cuda.gemv_norm)
            idx, w, xq, sfx = router_h
            pre = (xq, sfx)
            ksplit = w.shape[1] // self.K
        elif self.mx is not None and T <= self.MXF4_PAIR_MAX_TOKENS:
            # decode: routing and the MXFP8 rounding of the token rows share one launch
            from ..ops.cuda import moe_route_quant
            # one token on one rank: the down projection has too few (pair, column block) items for the chip and splits K
            if T * self.K <= 4 and not self.reduce and self.shared is None and self.expert_scale is None:
                from ..ops.cuda import mxf4_ksplit
                ksplit = mxf4_ksplit(self.mx[1].K, self.DOWN_KSPLIT)
            idx, w, xq, sfx = moe_route_quant(logits, self.router_bias, self.K, h, w_copies=ksplit)
            pre = (xq, sfx)
        else:
            idx, w = ops.moe_route(logits, self.router_bias, self.K, True, precise=h.dtype == torch.float32)
        if self.expert_scale is not None:
            w = w * self.expert_scale[idx.long()]
        local = self.e_hi - self.e_lo
        # expert parallelism on the peer-memory path: the combine writes its partial into every rank's inbox itself
        fuse_push = self.reduce and par.fused is not None and h.is_cuda and self.shared is None
        if self.mx is not None:
            y, p2p = self._mx_experts(h, idx, pre, ksplit)
            if fuse_push:
                return par.fused.moe_combine_push(y, p2p, w)
            if self.shared is None and not self.reduce and self.K <= 32:
                # single rank: the weighted sum is formed inside the residual add + norm that consumes it
                from ..ops.cuda import CombineDelta
                return CombineDelta(y, p2p, w.contiguous())
            out = ops.moe_combine(y, ops.ref.MoePacking(None, None, None, p2p, None, None, y.shape[0], self.K), w)
        elif self.a8:
            # CPU restatement of the block-scaled path: same rounding points, fp32 math
            q8 = lambda t: ops.ref.mxfp8_roundtrip(t).to(torch.bfloat16)
            slot_e = idx.reshape(-1)
            a = ops.expert_gemv(q8(h), self.gate_up, slot_e, x_div=self.K, bias=self.gu_bias, act=self.act, e_lo=self.e_lo)
            y = ops.expert_gemv(q8(a), self.down, slot_e, x_div=1, bias=self.down_bias, e_lo=self.e_lo)
            pk = ops.ref.MoePacking(None, None, None, torch.arange(T * self.K, dtype=torch.int32, device=h.device), None, None, T * self.K, self.K)
            out = ops.moe_combine(y, pk, w)
        elif T <= self.PAIR_GEMV_MAX_TOKENS and h.dtype != torch.float32:
            # decode: one GEMV slot per (token, expert) pair, weights streamed once per pair; under expert
            # parallelism the slots of experts that live on other ranks contribute zero rows here
            slot_e = idx.reshape(-1)
            a = ops.expert_gemv(h, self.gate_up, slot_e, x_div=self.K, bias=self.gu_bias, act=self.act, e_lo=self.e_lo)
            y = ops.expert_gemv(a, self.down, slot_e, x_div=1, bias=self.down_bias, e_lo=self.e_lo)
            key = (T, h.device)
            if key not in self._arange:
                pk = ops.ref.MoePacking(None, None, torch.zeros(1, dtype=torch.int32, device=h.device),
                                        torch.arange(T * self.K, dtype=torch.int32, device=h.device), None, None, T * self.K, self.K)
                self._arange[key] = pk
            if fuse_push:
                return par.fused.moe_combine_push(y, self._arange[key].pair_to_packed, w)
            if self._lazy(h):
                from ..ops.cuda import CombineDelta
                return CombineDelta(y, self._arange[key].pair_to_packed, w)
            out = ops.moe_combine(y, self._arange[key], w)
        elif T <= self.group_gemv_max_tokens and T * self.K <= 8 * local:
            # expert-major GEMV over a compact packing: every local expert streams its weights once against all of its rows (token
            # rows are read in place through the packing's index: no gather, no tile padding).  Measured slower than the grouped
            # tensor-core GEMM for gpt-oss-120b at 64 concurrent sequences (75 vs 61 ms per step), so it is off by default.
            pk = ops.moe_pack(idx, self.E, self.e_lo, self.e_hi, tile=1)
            a = ops.expert_group_gemv(h, self.gate_up, pk, x_index=pk.packed_token, bias=self.gu_bias, act=self.act, e_lo=self.e_lo)
            y = ops.expert_group_gemv(a, self.down, pk, bias=self.down_bias, e_lo=self.e_lo)
            if fuse_push:
                return par.fused.moe_combine_push(y, pk.pair_to_packed, w)
            out = ops.moe_combine(y, pk, w)
        else:
            pk = ops.moe_pack(idx, self.E, self.e_lo, self.e_hi)
            xp = ops.moe_gather(h, pk)
            te = pk.tile_expert - self.e_lo if self.e_lo else pk.tile_expert
            a = ops.grouped_linear(xp, self.gate_up, te, pk.num_tiles, bias=self.gu_bias, act=self.act)
            y = ops.grouped_linear(a, self.down, te, pk.num_tiles, bias=self.down_bias)
            if fuse_push:
                return par.fused.moe_combine_push(y, pk.pair_to_packed, w)
            if self._lazy(h):
                from ..ops.cuda import CombineDelta
                return CombineDelta(y, pk.pair_to_packed, w)
            out = ops.moe_combine(y, pk, w)
        if self.shared is not None:
            out = self.shared.add_into(out, h)
        if self.reduce:
            out = par.fused.push(out) if (par.fused is not None and out.is_cuda) else par.all_reduce(out)
        return out


class UnaryMoEFFN(MoEFFN):
    """Experts down(act(up h)) without a gate branch and without biases, of which each token uses the best K by router score; the weights are
    the softmax scores of the chosen ones, renormalised.  Routing, packing and execution are :class:`MoEFFN`'s; one GPU."""

    LAZY_COMBINE = True
    PAIR_GEMV_MAX_TOKENS = 6     # 8 tokens, 6 of 64 experts of 2304 x 4096: slots 478 us, packed 301; 4 tokens: 174 against 198

    def __init__(self, src, prefix: str, hidden: int, row: int, experts: int, used: int, ffn: int, act: int):
        f = round_up(ffn, 32)
        self.E, self.K, self.e_lo, self.e_hi, self.expert_tp = experts, used, 0, experts, False
        rw = src.matrix(f"{prefix}.router", experts, hidden)
        self.router = Linear((rw if rw.fmt == WFormat.BF16 else QuantWeight(**_as_bf16(rw))).pad_groups(cols=(1, row)))
        self.gate_up = src.matrix(f"{prefix}.e*.up", ffn, hidden, experts).pad_groups(rows=(1, f), cols=(1, row))
        self.down = src.matrix(f"{prefix}.e*.down", hidden, ffn, experts).pad_groups(rows=(1, row), cols=(1, f))
        self.router_bias = self.gu_bias = self.down_bias = self.expert_scale = self.shared = self.mx = self._spill = None
        self.act, self.a8, self.reduce, self.group_gemv_max_tokens, self._arange = act, False, False, 0, {}


class ScaledInputMoEFFN(UnaryMoEFFN):
    """Gated experts without biases, of which each token uses the best K by router score; the weight -- the sigmoid of the chosen score, as it is --
    multiplies what the expert reads, so the branch is a plain sum of rows, to which an always-on expert may add one.  Returns the sum unformed
    (:class:`ops.ExpertSum`).  One GPU."""

    PAIR_GEMV_MAX_TOKENS = 4

    def __init__(self, src, prefix: str, hidden: int, row: int, experts: int, used: int, ffn: int, shared_ffn: int = 0, act: int = ACT_SWIGLU):
        super().__init__(src, prefix, hidden, row, experts, used, ffn, act)          # (gate_up holds the up rows so far)
        gate = src.matrix(f"{prefix}.e*.gate", ffn, hidden, experts).pad_groups(rows=(1, round_up(ffn, 32)), cols=(1, row))
        self.gate_up = QuantWeight.interleave_gate_up(gate, self.gate_up)
        self.shared = GatedFFN(src, f"{prefix}.shared", hidden, row, shared_ffn, act) if shared_ffn else None

    def __call__(self, h: torch.Tensor, par: Optional[ParallelCtx] = None):
        T, K = h.shape[0], self.K
        idx, w = ops.moe_route(self.router(h, out_f32=True), None, K, precise=h.dtype == torch.float32, sigmoid=True)
        if T <= self.PAIR_GEMV_MAX_TOKENS and h.dtype != torch.float32:
            slot_e = idx.reshape(-1)
            a = ops.expert_gemv(ops.moe_scale_rows(h, w), self.gate_up, slot_e, act=self.act)
            y = ops.expert_gemv(a, self.down, slot_e)
            if (T, h.device) not in self._arange:
                self._arange[T, h.device] = torch.arange(T * K, dtype=torch.int32, device=h.device)
            pos = self._arange[T, h.device]
        else:
            pk = ops.moe_pack(idx, self.E)
            a = ops.grouped_linear(ops.moe_scale_rows(h, w, pk), self.gate_up, pk.tile_expert, pk.num_tiles, act=self.act)
            y = ops.grouped_linear(a, self.down, pk.tile_expert, pk.num_tiles)
            pos = pk.pair_to_packed
        return ops.ExpertSum(y, pos, K, None if self.shared is None else self.shared(h))


class ClampedMoEFFN(UnaryMoEFFN):
    """Experts down(clamped SwiGLU(gate h, up h)) without biases, of which each token uses the best K by biased router logit, weighted with the softmax of
    the chosen ones; an always-on expert of the same form joins times the sigmoid of one number per token.  That number is one more row of the router's
    matrix.  Returns the sum unformed (:class:`ops.ExpertSum`).  One GPU."""

    # nine layers with 6 of 64 experts, 6 sequences: 2048 x 1024 slots 2.30 ms a step, packed 2.43; 4096 x 1536 4.96 against 4.19
    PAIR_GEMV_MAX_TOKENS = 4
    PAIR_GEMV_SMALL_BYTES = 12 << 20         # experts up to this size (gate and up rows) are streamed per pair for two tokens more

    def __init__(self, src, prefix: str, hidden: int, row: int, experts: int, used: int, ffn: int, limit: float, shared_ffn: int = 0, shared_limit: float = 0.0,
                 act: int = ACT_SWIGLU_OAI, alpha: float = 1.702):
        super().__init__(src, prefix, hidden, row, experts, used, ffn, act)          # (gate_up holds the up rows so far)
        gate = src.matrix(f"{prefix}.e*.gate", ffn, hidden, experts).pad_groups(rows=(1, round_up(ffn, 32)), cols=(1, row))
        self.gate_up = QuantWeight.interleave_gate_up(gate, self.gate_up)
        if self.gate_up.nbytes <= experts * self.PAIR_GEMV_SMALL_BYTES:
            self.PAIR_GEMV_MAX_TOKENS = 6
        self.act_kw = dict(act=act, act_alpha=alpha, act_limit=limit)
        self.shared = GatedFFN(src, f"{prefix}.shared", hidden, row, shared_ffn, **{**self.act_kw, "act_limit": shared_limit}) if shared_ffn else None
        rows = [self.router.w]
        if shared_ffn:
            sg = src.matrix(f"{prefix}.shared.sg", 1, hidden)
            rows.append((sg if sg.fmt == WFormat.BF16 else QuantWeight(**_as_bf16(sg))).pad_groups(cols=(1, row)))
        w = QuantWeight.cat_rows(rows)
        n = round_up(w.N, 8)
        bias = torch.nn.functional.pad(src.vector(f"{prefix}.router.b", experts), (0, n - experts)).contiguous()
        self.router = Linear(w.pad_groups(rows=(1, n)), bias)

    def __call__(self, h: torch.Tensor, par: Optional[ParallelCtx] = None):
        T, K = h.shape[0], self.K
        z = self.router(h, out_f32=True)
        idx, w = ops.moe_route(z, None, K, precise=h.dtype == torch.float32, experts=self.E)
        if T <= self.PAIR_GEMV_MAX_TOKENS and h.dtype != torch.float32:
            slot_e = idx.reshape(-1)
            a = ops.expert_gemv(h, self.gate_up, slot_e, x_div=K, **self.act_kw)
            y = ops.expert_gemv(a, self.down, slot_e)
            if (T, h.device) not in self._arange:
                self._arange[T, h.device] = torch.arange(T * K, dtype=torch.int32, device=h.device)
            pos = self._arange[T, h.device]
        else:
            pk = ops.moe_pack(idx, self.E)
            a = ops.grouped_linear(ops.moe_gather(h, pk), self.gate_up, pk.tile_expert, pk.num_tiles, **self.act_kw)
            y = ops.grouped_linear(a, self.down, pk.tile_expert, pk.num_tiles)
            pos = pk.pair_to_packed
        if self.shared is None:
            return ops.ExpertSum(y, pos, K, w=w)
        return ops.ExpertSum(y, pos, K, self.shared(h), w, z[:, self.E])


def _mx_experts(self, h: torch.Tensor, idx: torch.Tensor, pre=None, ksplit: int = 1):
    """Expert projections on the block-scaled MXFP4 kernel.  Returns (y bf16 [rows, H], pair_to_packed int32 [T*K]).  ``pre``: the
    pair-mode (xq, sfx) when the router launch has already quantised the rows.  ``ksplit`` (pair mode): the down projection leaves
    that many partial rows per pair, and pair_to_packed lists them all ([T, ksplit, K])."""
    from ..ops import cuda as K_
    gate_up, down = self.mx
    T = h.shape[0]
    ep = dict(e_lo=self.e_lo)
    if T <= self.MXF4_PAIR_MAX_TOKENS:
        # decode: pair i = (token i // K, slot i % K) is tile i with one live row; no sort, no gather
        n = T * self.K
        te = idx.reshape(-1)
        xq, sfx = pre if pre is not None else K_.moe_quant(h, n, n, 1, x_div=self.K)
        aq, sfa = K_.mxf4_gemm(gate_up, xq, sfx, te, n, 1, default_valid=1, bias0=self.g_bias, bias1=self.u_bias, act=self.act, **ep)
        y = K_.mxf4_gemm(down, aq, sfa, te, n, 1, default_valid=1, bias0=self.down_bias, zero_out=self.reduce, ksplit=ksplit, **ep)
        key = (T, ksplit, h.device)
        if key not in self._arange:
            # pair (t, k) sits at row t * K + k of every K range's block of n rows
            base = torch.arange(n, dtype=torch.int32, device=h.device).reshape(T, 1, self.K)
            off = (torch.arange(ksplit, dtype=torch.int32, device=h.device) * n).reshape(1, ksplit, 1)
            self._arange[key] = (base + off).reshape(-1).contiguous()
        return y, self._arange[key]
    pk = ops.moe_pack(idx, self.E, self.e_lo, self.e_hi)
    mt = pk.tile_expert.numel()
    tiles = dict(tile_valid=pk.tile_valid, num_tiles=pk.num_tiles)
    xq, sfx = K_.moe_quant(h, pk.max_rows, mt, 128, src_index=pk.packed_token, row_limit=pk.num_tiles)
    aq, sfa = K_.mxf4_gemm(gate_up, xq, sfx, pk.tile_expert, mt, 128, bias0=self.g_bias, bias1=self.u_bias, act=self.act, **tiles, **ep)
    y = K_.mxf4_gemm(down, aq, sfa, pk.tile_expert, mt, 128, bias0=self.down_bias, **tiles, **ep)
    return y, pk.pair_to_packed


MoEFFN._mx_experts = _mx_experts


def _moe_sharded(self, h: torch.Tensor, sc) -> torch.Tensor:
    """Row-sharded prefill: this rank routes only its own rows ``h`` [R, H], the rows travel as MXFP8 to the ranks that own their
    experts, and the expert outputs come back to be summed here.  Returns the fp32 contribution [R, H]."""
    from ..ops import cuda as K_
    gate_up, down = self.mx
    logits = self.router(h, out_f32=True)
    idx, w = ops.moe_route(logits, self.router_bias, self.K, True)
    if self.expert_scale is not None:
        w = w * self.expert_scale[idx.long()]
    xq, sfx, plan = sc.dispatch(h, idx)
    tiles = dict(tile_valid=plan.tile_valid, num_tiles=plan.num_tiles, e_lo=self.e_lo)
    aq, sfa = K_.mxf4_gemm(gate_up, xq, sfx, plan.tile_expert, plan.max_tiles, 128, bias0=self.g_bias, bias1=self.u_bias, act=self.act, **tiles)
    y = K_.mxf4_gemm(down, aq, sfa, plan.tile_expert, plan.max_tiles, 128, bias0=self.down_bias, **tiles)
    return sc.combine(y, plan, w)


MoEFFN.forward_sharded = _moe_sharded


def _as_bf16(w: QuantWeight) -> dict:
    d = w.dequantize(torch.bfloat16)
    return dict(fmt=ops.WFormat.BF16, N=w.N, K=w.K, E=w.E, p0=d.contiguous())


# ---------------------------------------------------------------------------------------------
class TransformerModel:
    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192):
        self.cfg, self.device = cfg, torch.device(device)
        self.par = par or ParallelCtx()
        c, par = cfg, self.par
        self.max_ctx = max_ctx
        tp = par.world if par.mode == "tp" else 1
        # layer split (pipeline) plan: contiguous layer ranges, embedding on the first rank, head on the last
        # (LayerPlan::contiguous, src/model/dense_split.cpp:24-33)
        self.pp = par.mode == "pp" and par.world > 1
        self.tap = None          # optional callable(layer, mixer_out, ffn_out, residual) used by the layer-dump tool
        self.layer_lo, self.layer_hi = ((par.rank * c.n_layers) // par.world, ((par.rank + 1) * c.n_layers) // par.world) if self.pp else (0, c.n_layers)
        self.first_stage, self.last_stage = (not self.pp or par.rank == 0), (not self.pp or par.rank == par.world - 1)
        self.tied = not src.has("output.weight") or c.tie_embeddings
        self.embed_w = self._vocab_matrix(src, "token_embd.weight") if (self.first_stage or (self.last_stage and self.tied)) else None
        head = None
        if self.last_stage:
            head = self.embed_w if self.tied else self._vocab_matrix(src, "output.weight")
        self.vocab_lo, self.vocab_hi = 0, c.vocab
        if tp > 1:
            lo, hi = _even_chunks(c.vocab, tp, 16)[par.rank] if c.vocab % (16 * tp) == 0 else (0, c.vocab)
            if (lo, hi) != (0, c.vocab):
                head = head.slice_rows(lo, hi)
                self.vocab_lo, self.vocab_hi = lo, hi
        self.lm_head = Linear(head) if head is not None else None
        self.out_norm = src.vector("output_norm.weight", c.hidden)
        ff = src.vector("rope_freqs.weight", c.n_rot // 2) if (c.arch == "llama" and getattr(src, "r", None) is not None and src.has("rope_freqs.weight")) else None
        self.rope = rope_tables(max_ctx, c.n_rot, c.rope_theta, ff, c.rope_scaling_type, c.rope_scaling_factor, c.rope_orig_ctx,
                                c.yarn_beta_fast, c.yarn_beta_slow, device=self.device)
        self.one_plus_w = c.arch in ("qwen35", "qwen35moe")
        self.layer_ids = list(range(self.layer_lo, self.layer_hi))
        self.layers = [self._build_layer(l, src) for l in self.layer_ids]
        self.attn_layers = [l for l in self.layer_ids if c.layer_is_full_attention(l)]
        self.n_kv_local = next((L["attn"].n_kv for L in self.layers if "attn" in L), 0)

    # ---- construction
    def _vocab_matrix(self, src, name: str) -> QuantWeight:
        return src.matrix(name, self.cfg.vocab, self.cfg.hidden)

    def _build_layer(self, l: int, src) -> dict:
        c, par = self.cfg, self.par
        p = f"blk.{l}"
        L = {"attn_norm": src.vector(f"{p}.attn_norm.weight", c.hidden)}
        L["attn"] = AttentionBlock(c, l, src, par)
        post = f"{p}.post_attention_norm.weight" if c.arch in ("gpt-oss",) else f"{p}.ffn_norm.weight"
        L["ffn_norm"] = src.vector(post, c.hidden)
        if c.arch == "gpt-oss":
            L["moe"] = MoEFFN(c, l, src, par, ACT_SWIGLU_OAI, with_bias=True)
        elif c.arch == "qwen3moe":
            L["moe"] = MoEFFN(c, l, src, par, ACT_SWIGLU, with_bias=False)
        else:
            L["ffn"] = DenseFFN(c, l, src, par)
        return L

    def new_kv_cache(self, num_blocks: int, dtype: str = "bf16") -> KVCache:
        return KVCache(self.cfg.n_layers, num_blocks, self.n_kv_local, self.cfg.head_dim, self.device, self.attn_layers, dtype=dtype)

    def kv_bytes_per_block(self, dtype: str = "bf16") -> int:
        return KVCache.bytes_per_block(len(self.attn_layers), self.n_kv_local, self.cfg.head_dim, dtype)

    def weight_bytes(self) -> int:
        n = (self.embed_w.nbytes if self.embed_w is not None else 0) + (0 if (self.tied or self.lm_head is None) else self.lm_head.w.nbytes)
        for L in self.layers:
            for v in L.values():
                n += _bytes_of(v)
        return n

    # ---- forward
    def forward(self, fb: ForwardBatch, kv: KVCache, state=None) -> torch.Tensor:
        """Returns fp32 logits [rows, vocab] for ``fb.logit_rows`` (default: last token of each sequence)."""
        if self.pp:
            return self._forward_pipeline(fb, kv, state)
        c = self.cfg
        if self._can_shard(fb, state):
            return self._forward_sharded(fb, kv)
        x = ops.embed(self.embed_w, fb.ids, c.embedding_scale)
        x, delta = self._run_layers(x, None, fb, kv, state)
        return self._head(x, delta, fb)

    # ---- row-sharded prefill (tensor / expert parallel ranks each keep T / W rows of the residual stream)
    def _can_shard(self, fb: ForwardBatch, state) -> bool:
        par = self.par
        sc = getattr(par, "sharded", None)
        if sc is None or par.fused is None or state is not None or self.tap is not None or fb.want_hidden or type(self) is not TransformerModel:
            return False
        if not sc.can_shard(fb.T) or fb.T < self.SHARD_MIN_TOKENS:
            return False
        return all(("moe" not in L) or (L["moe"].mx is not None and L["moe"].shared is None and not L["moe"].expert_tp and L["moe"]._spill is None)
                   for L in self.layers)

    SHARD_MIN_TOKENS = 512

    def _forward_sharded(self, fb: ForwardBatch, kv: KVCache) -> torch.Tensor:
        """Prefill with the residual stream sharded by rows: per layer one all-gather (fused into the qkv GEMM's operand load), one
        reduce-scatter (the output projection's epilogue) and, for expert layers, an all-to-all of MXFP8 rows and bf16 results; dense
        FFN layers take a second gather / scatter pair.  Norms, routing, packing and quantisation run on T / W rows."""
        c, par = self.cfg, self.par
        sc = par.sharded
        T = fb.T
        row0, R = sc.rows(T)
        x = ops.embed(self.embed_w, fb.ids[row0:row0 + R].contiguous(), c.embedding_scale)
        rs = c.residual_scale
        nk = dict(one_plus_w=self.one_plus_w, delta_scale=rs)
        delta = None
        for L in self.layers:
            _, g = sc.norm(x, L["attn_norm"], c.rms_eps, T, delta=delta, gather=True, **nk)
            a = L["attn"].forward_gathered(sc, T, g, fb, kv, self.rope, par)
            if "moe" in L:
                h2, _ = sc.norm(x, L["ffn_norm"], c.rms_eps, T, delta=a, want_local=True, **nk)
                delta = L["moe"].forward_sharded(h2, sc)
            else:
                _, g2 = sc.norm(x, L["ffn_norm"], c.rms_eps, T, delta=a, gather=True, **nk)
                delta = L["ffn"].forward_gathered(sc, T, g2, par)
        sc.norm(x, self.out_norm, c.rms_eps, T, delta=delta, **nk)            # folds the last delta into the residual rows
        # the rows that need logits, replicated: each rank contributes the ones it owns
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        local = rows.long() - row0
        mine = ((local >= 0) & (local < R)).unsqueeze(-1)
        xr = torch.where(mine, x.index_select(0, local.clamp(0, R - 1)), torch.zeros((), dtype=x.dtype, device=x.device))
        if par.world > 1:
            par.all_reduce(xr)
        hn = ops.rmsnorm(xr, self.out_norm, c.rms_eps, one_plus_w=self.one_plus_w)
        logits = self.lm_head(hn, out_f32=True)
        if self.vocab_hi - self.vocab_lo != c.vocab:
            logits = par.all_gather_cols(logits)
        if c.logit_scale != 1.0:
            logits = logits * c.logit_scale
        if c.final_logit_softcap > 0:
            logits = torch.tanh(logits / c.final_logit_softcap) * c.final_logit_softcap
        return logits

    # Decode with the norms inside the GEMVs that consume them (ops.cuda.gemv_norm).  Measured on gpt-oss-120b / 20b decode at
    # context 2048: 3.87 / 2.65 ms per token against 3.70 / 2.50 with one kernel per op: every CTA of the GEMV repeats the norm's
    # reads from L2, which costs more than the launch it saves under programmatic dependent launch.  Off; tests keep it honest.
    FUSED_DECODE = False
    FUSED_DECODE_QKV = True      # ... the attention norm inside the qkv GEMV
    FUSED_DECODE_ROUTER = True   # ... the FFN norm, routing and quantisation inside the router GEMV

    def _run_layers_decode(self, x, delta, fb, kv):
        """Single-rank decode (one or two rows): both norms of a layer run inside the GEMV that consumes them (qkv; router, whose launch
        also routes and quantises), so a layer is qkv -> head epilogue -> attention -> o-proj -> router -> gate|up -> down."""
        from ..ops import cuda as K_
        c, par = self.cfg, self.par
        nk = dict(one_plus_w=self.one_plus_w, delta_scale=c.residual_scale)
        for L in self.layers:
            at = L["attn"]
            r = None
            if self.FUSED_DECODE_QKV and isinstance(at.qkv, Linear):
                r = K_.gemv_norm(x, L["attn_norm"], c.rms_eps, at.qkv.w, at.qkv.bias, delta=delta, **nk)
            if r is None:
                qkv = at.qkv(self._norm(x, L["attn_norm"], delta))
            else:
                qkv, x, _ = r
            a = at.attend(qkv, fb, kv, self.rope, par)
            moe = L.get("moe")
            r = None
            if self.FUSED_DECODE_ROUTER and moe is not None and moe.mx is not None and moe.expert_scale is None and moe.shared is None:
                # with one token the down projection has too few (pair, column block) items for the chip: it splits K in two
                copies = K_.mxf4_ksplit(moe.mx[1].K, moe.DOWN_KSPLIT) if x.shape[0] * moe.K <= 4 else 1
                r = K_.gemv_norm(x, L["ffn_norm"], c.rms_eps, moe.router.w, moe.router.bias, delta=a, route=(moe.router_bias, moe.K, True, copies), **nk)
            if r is not None:
                _, x, _, idx, w, xq, sfx = r
                delta = moe(a, par, router_h=(idx, w, xq, sfx))        # (`a` only gives the row count here)
            else:
                h2 = self._norm(x, L["ffn_norm"], a)
                delta = moe(h2, par) if moe is not None else L["ffn"](h2, par)
        return x, delta

    def _run_layers(self, x, delta, fb, kv, state):
        par = self.par
        if (self.FUSED_DECODE and x.is_cuda and x.shape[0] <= 2 and par.world == 1 and self.tap is None and state is None
                and type(self) is TransformerModel and ops.backend() != "torch"):
            return self._run_layers_decode(x, delta, fb, kv)
        for li, L in enumerate(self.layers):
            h = self._norm(x, L["attn_norm"], delta)
            a = self._mixer(li, L, h, fb, kv, state)
            h2 = self._norm(x, L["ffn_norm"], a)
            delta = L["moe"](h2, par) if "moe" in L else L["ffn"](h2, par)
            if self.tap is not None:                 # per-layer dump hook of the parity tools (single rank, eager)
                if not isinstance(delta, torch.Tensor) and hasattr(delta, "materialize"):
                    delta = delta.materialize()
                self.tap(li, a, delta, x)
        return x, delta

    def _head(self, x, delta, fb):
        c, par = self.cfg, self.par
        rs = c.residual_scale
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        xr = x.index_select(0, rows)
        dr = delta.index_select(0, rows).contiguous() if delta is not None else None       # (a pending fused reduction is summed here)
        hidden = None
        if fb.want_hidden:
            hidden = xr + dr.to(torch.float32) * rs if dr is not None else xr.clone()
        hn = ops.rmsnorm(xr, self.out_norm, c.rms_eps, delta=dr, one_plus_w=self.one_plus_w, delta_scale=rs)
        logits = self.lm_head(hn, out_f32=True)
        if self.vocab_hi - self.vocab_lo != c.vocab:
            logits = par.all_gather_cols(logits)
        if c.logit_scale != 1.0:
            logits = logits * c.logit_scale
        if c.final_logit_softcap > 0:
            logits = torch.tanh(logits / c.final_logit_softcap) * c.final_logit_softcap
        return (logits, hidden) if fb.want_hidden else logits

    # ---- layer-split (pipeline) forward
    def _forward_pipeline(self, fb: ForwardBatch, kv: KVCache, state=None):
        """Each rank runs its contiguous layer range.  A single long prefill chunk is cut into token micro-batches that
        flow through the stages back to back (stage r works on micro-batch i while stage r+1 works on i-1; causal
        attention only needs the earlier micro-batches' KV, which that stage has already written), so the stages
        overlap instead of running strictly one after the other as in the reference (src/model/dense_split.cpp:258:
        one residual hand-off per boundary, serial).  The residual crosses a boundary as one fp32 [T, H] message over
        NCCL point-to-point; the last stage's logits are broadcast so that every rank samples the same token."""
        c, par = self.cfg, self.par
        if fb.want_hidden:
            raise NotImplementedError("speculative decoding is not combined with the layer split")
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        n_rows = rows.numel()
        out = None
        pieces = self._micro_batches(fb)
        last_logits = []
        for mb, keep in pieces:
            if self.first_stage:
                x = ops.embed(self.embed_w, mb.ids, c.embedding_scale)
            else:
                x = torch.empty(mb.T, c.hidden, dtype=torch.float32, device=self.device)
                par.recv(x, par.rank - 1)
            x, delta = self._run_layers(x, None, mb, kv, state)
            if not self.last_stage:
                d = delta if isinstance(delta, torch.Tensor) else delta.materialize()
                x = x + d.to(torch.float32) * c.residual_scale
                par.send(x.contiguous(), par.rank + 1)
            elif keep:
                last_logits.append(self._head(x, delta, mb))
        logits = torch.empty(n_rows, c.vocab, dtype=torch.float32, device=self.device)
        if self.last_stage:
            logits.copy_(torch.cat(last_logits, dim=0) if len(last_logits) > 1 else last_logits[0])
        par.broadcast(logits, src=par.world - 1)
        return logits

    def _micro_batches(self, fb: ForwardBatch, min_tokens: int = 256):
        """[(ForwardBatch, has_logit_rows)].  Only a single-sequence prefill chunk is cut (into world-size pieces of at
        least ``min_tokens``); mixed batches and decode steps go through whole."""
        n = self.par.world
        if fb.B != 1 or fb.T < 2 * min_tokens or fb.logit_rows is None or fb.state_slots is not None:
            return [(fb, True)]
        T = fb.T
        per = max(min_tokens, (T + n - 1) // n)
        per = (per + 127) // 128 * 128
        kv_end = int(fb.seq_lens[0])
        start = kv_end - T
        out, rows = [], fb.logit_rows
        for lo in range(0, T, per):
            hi = min(T, lo + per)
            sel = (rows >= lo) & (rows < hi)
            lr = (rows[sel] - lo)
            mb = ForwardBatch(fb.ids[lo:hi], fb.positions[lo:hi], fb.slot_map[lo:hi], fb.block_table,
                              torch.tensor([start + hi], dtype=torch.int32, device=fb.ids.device),
                              torch.tensor([0, hi - lo], dtype=torch.int32, device=fb.ids.device), hi - lo, logit_rows=lr if lr.numel() else None)
            out.append((mb, lr.numel() > 0))
        return out

    def _norm(self, x, w, delta):
        """Residual add + RMSNorm; a delta that still lives as per-rank partials in the collective inbox is summed here."""
        c = self.cfg
        if delta is not None and not isinstance(delta, torch.Tensor):
            if hasattr(delta, "pair_to_packed"):       # an expert combine that has not been formed (ops.cuda.CombineDelta)
                from ..ops.cuda import rmsnorm_combine
                return rmsnorm_combine(x, w, c.rms_eps, delta, one_plus_w=self.one_plus_w, delta_scale=c.residual_scale)
            return self.par.fused.rmsnorm(x, w, c.rms_eps, delta, one_plus_w=self.one_plus_w, delta_scale=c.residual_scale)
        return ops.rmsnorm(x, w, c.rms_eps, delta=delta, one_plus_w=self.one_plus_w, delta_scale=c.residual_scale)

    def _mixer(self, li, L, h, fb, kv, state):
        return L["attn"](h, fb, kv, self.rope, self.par)


def _bytes_of(v) -> int:
    if isinstance(v, torch.Tensor):
        return v.numel() * v.element_size()
    if isinstance(v, QuantWeight):
        return v.nbytes
    if isinstance(v, Linear):
        return v.w.nbytes + (_bytes_of(v.bias) if v.bias is not None else 0)
    if isinstance(v, MultiLinear):
        return sum(_bytes_of(p) for p in v.parts)
    if isinstance(v, (list, tuple)):
        return sum(_bytes_of(i) for i in v)
    if hasattr(v, "__dict__"):
        return sum(_bytes_of(i) for i in vars(v).values() if isinstance(i, (torch.Tensor, QuantWeight, Linear, MultiLinear, tuple, list)))
    return 0
