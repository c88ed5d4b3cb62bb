"""Zegelix: RG-LRU layers and attention over a window with pooled blocks before it, in any order; clamped gated experts with an always-on one; a range of
layers that runs several times and begins each pass with a mix of the residual and the embedding output; a tied head.

    x0 = scale embed[token]
    layer:  x <- x + mixer(norm(x; norm1));  x <- x + ff(norm(x; norm2))           (layers may have no feed-forward)
    loop:   layers start .. stop - 1 run ``times`` times; a pass begins with x <- W_in [x; x0] and has its own cache and state
    logits = logit_scale embed norm(x; final.norm)

norm(x; w) = x / rms(x) w, eps inside the root.
attention:  q, k, v biased; q and k rotated in half splits over rot.dims, v over its whole width; softmax over the last ``window`` tokens and the means
            of the cached keys / values of whole blocks of ``pool`` tokens before them, of cap tanh((q . k) scale temp_h / cap), exp(sink_h) in the
            denominator; the sum turned back by the query's position; the heads times sigmoid(W_g h); W_o.
rglru:      y = gelu_tanh(W_y h + b), u = conv(W_x h + b) + b; r, i = sigmoid(W_r u + b), sigmoid(W_i u + b) per block of channels;
            log a = -8 r softplus(lam); S <- a S + sqrt(1 - a^2) i u; W_o (S y).
ff:         sum over the chosen e of softmax weight times expert_e(h), + sigmoid(w_sg . h) shared(h); expert = W_down (g sigmoid(1.702 g) (u + 1)),
            g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit).

Launches of a layer: sublayer_norm (adds the previous branch -- a row, or a token's expert rows with their weights, formed as they are read -- to the fp32
residual, norms the sum), the mixer's own (see the blocks), sublayer_norm, router, routing, the experts' two projections and the shared expert's.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..formats.model_config import ModelConfig
from ..parallel.comm import ParallelCtx
from ..utils.rope import rope_tables
from .hybrid import RecurrentState, RglruBlock
from .layer_list import LayerListModel
from .transformer import ClampedMoEFFN, ForwardBatch, KVCache, Linear, PooledAttentionBlock


class ZegelixModel(LayerListModel):
    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
        self.runs = cfg.layer_runs()
        super().__init__(cfg, src, device, par, max_ctx=max_ctx, dtype=dtype)
        self.out_norm = self._row_vector(self.out_norm * cfg.logit_scale)
        self.loop_in = Linear(src.matrix("loop.in", cfg.hidden, 2 * cfg.hidden).pad_groups(rows=(1, self.row), cols=(2, self.row))) if cfg.loop_times else None

    @property
    def needs_state(self) -> bool:
        return any("lin" in L for L in self.layers)

    # ---- construction
    def _row_vector(self, v: torch.Tensor) -> torch.Tensor:
        return torch.nn.functional.pad(v, (0, self.row - v.numel())).contiguous()

    def _blocks(self, kind: str) -> dict:
        """Per layer run with such a mixer: its block."""
        return {i: self.layers[l][kind] for i, (l, _) in enumerate(self.runs) if kind in self.layers[l]}

    def _kv_geometry(self) -> dict:
        return {i: (a.n_kv, a.dk, a.dv) for i, a in self._blocks("attn").items()}

    def _kv_pools(self) -> dict:
        specs = {i: self.cfg.layer_specs[l] for i, (l, _) in enumerate(self.runs)}
        return {i: (specs[i].pool, specs[i].window) for i in self._blocks("attn") if specs[i].pool}

    def _rope(self, dims: int, base: float) -> tuple:
        return self._table((dims, base), lambda: rope_tables(self.max_ctx, dims, base, device=self.device))

    def _build_layer(self, l: int, src) -> dict:
        s, H, p = self.cfg.layer_specs[l], self.cfg.hidden, f"l{l}"
        L = {"norm1": self._row_vector(src.vector(f"{p}.norm1", H))}
        if s.mixer == "pooled_attention":
            L["attn"] = PooledAttentionBlock(src, f"{p}.mix", H, self.row, s.heads, s.kv_heads, s.key_dim, s.value_dim, s.scale, s.window, s.softcap, s.rot_dim,
                                             self._rope(s.rot_dim, s.rope_theta), self._rope(s.value_dim, s.rope_theta))
        else:
            L["lin"] = RglruBlock(src, f"{p}.mix", H, self.row, s.width, s.gate_blocks, s.conv_taps)
        if s.experts:
            L["norm2"] = self._row_vector(src.vector(f"{p}.norm2", H))
            L["moe"] = ClampedMoEFFN(src, f"{p}.mlp", H, self.row, s.experts, s.experts_used, s.expert_ffn, s.act_limit, s.shared_ffn, s.shared_limit)
        return L

    def new_state(self, n_slots: int) -> RecurrentState:
        tensors: dict = {"S": {}, "conv": {}}
        for i, block in self._blocks("lin").items():
            for name, t in block.state_tensors(n_slots, self.act_dtype, self.device).items():
                tensors[name][i] = t
        return RecurrentState(n_slots, tensors, self.device)

    # ---- forward
    def _fold(self, x, delta, w=None, out=None):
        """Residual x + a branch's output -> norm(x; w), or without w the sum itself."""
        return ops.sublayer_norm(x, delta, None, self.cfg.rms_eps, w=w, width=self.cfg.hidden, out_dtype=self.act_dtype, out=out)

    def _run_layers(self, x, delta, fb: ForwardBatch, kv: KVCache, state):
        both = None
        if self.loop_in is not None:             # [residual | embedding output]: a pass fills the first half
            both = torch.empty(x.shape[0], 2 * self.row, dtype=self.act_dtype, device=x.device)
            self._fold(x, None, out=both[:, self.row:])
        for i, (l, t) in enumerate(self.runs):
            L = self.layers[l]
            if t is not None:
                self._fold(x, delta, out=both[:, :self.row])
                x, delta = self.loop_in(both, out_f32=True), None
            h = self._fold(x, delta, L["norm1"])
            m = delta = L["attn"](h, fb, kv, i) if "attn" in L else L["lin"](h, fb, state, i)
            f = None
            if "moe" in L:
                f = delta = L["moe"](self._fold(x, m, L["norm2"]))
            if self.tap is not None:
                self.tap(i, m, f.materialize() if f is not None else torch.zeros_like(x), x)
        return x, delta

    def _head(self, x, delta, fb: ForwardBatch):
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        delta = delta.index_select(0, rows) if isinstance(delta, torch.Tensor) else delta.rows(rows)
        return self.lm_head(self._fold(x.index_select(0, rows), delta, self.out_norm), out_f32=True)
