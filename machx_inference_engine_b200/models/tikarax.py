"""Tikarax: layers listed one by one in the configuration, attention without rotation and minGRU layers in any order, RMS norms in groups
on both sides of every sublayer, a feed-forward without a gate branch.

    x = norm(embed[token]; embed.norm)
    layer:  x <- x + norm(mixer(norm(x; norm1)); norm1b)
            x <- x + norm(ff(norm(x; norm2)); norm2b)              (layers may have no feed-forward)
    logits = head norm(x; final.norm)

norm(.; w): every one of ``norm_groups`` equal parts of the row over its own root mean square, the whole times w.
attention:  q, k, v biased; q scaled by 1 + coef ln(floor((p + 1) / every) + 1) at position p; causal softmax over (q . k) scale; the heads
            times sigmoid(W_g h); W_o.
minGRU:     z = sigmoid(W_z h + b_z), u = W_x h + b_x, c = u + 1/2 (u >= 0) or sigmoid(u); S <- (1 - z) S + z c; W_o (S silu(W_g h)).
ff:         W_down xIELU(W_up h), xIELU(v) = softplus(p) v^2 + v / 2 (v > 0), (1/2 + softplus(q)) (e^v - 1 - v) + v / 2 (v <= 0).

Launches of a layer: group_norm (norms the previous branch's output, adds it to the fp32 residual, norms the sum), the fused projection,
[kv_store, attention with gate and temperature] or [recurrence with its gates], output projection, group_norm, up projection with the
activation, down projection.

The model runs in bf16 (matrix products and activations; residual, norms, scores, gates and state in fp32) or, with ``dtype="fp32"``, in
32-bit throughout.  Rows are padded to a multiple of 32 columns; the padding is zero everywhere.  One GPU.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import ops
from ..formats.model_config import ModelConfig
from ..ops import ACT_XIELU
from ..parallel.comm import ParallelCtx
from ..utils.rope import query_temperature_table
from .hybrid import MinGRUBlock, RecurrentState
from .layer_list import LayerListModel
from .transformer import ForwardBatch, KVCache, NoRopeAttentionBlock, UnaryFFN


def _softplus(v: float) -> float:
    return max(v, 0.0) + math.log1p(math.exp(-abs(v)))


class TikaraxModel(LayerListModel):
    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
        super().__init__(cfg, src, device, par, max_ctx=max_ctx, dtype=dtype)
        self.embed_norm = src.vector("embed.norm", cfg.hidden)

    @property
    def needs_state(self) -> bool:
        return any("lin" in L for L in self.layers)

    # ---- construction
    def _kv_geometry(self) -> dict:
        return {l: (L["attn"].n_kv, L["attn"].dk, L["attn"].dv) for l, L in zip(self.layer_ids, self.layers) if "attn" in L}

    def _q_scale(self, coef: float, every: float) -> Optional[torch.Tensor]:
        return None if coef == 0.0 else self._table((coef, every), lambda: query_temperature_table(self.max_ctx, coef, every, device=self.device))

    def _build_layer(self, l: int, src) -> dict:
        s, H, p = self.cfg.layer_specs[l], self.cfg.hidden, f"l{l}"
        L = {"norm1": src.vector(f"{p}.norm1", H), "norm1b": src.vector(f"{p}.norm1b", H)}
        if s.mixer == "attention":
            L["attn"] = NoRopeAttentionBlock(src, f"{p}.mix", l, H, self.row, s.heads, s.kv_heads, s.key_dim, s.value_dim, s.scale,
                                             self._q_scale(s.q_temp_coef, s.q_temp_every))
        else:
            L["lin"] = MinGRUBlock(src, f"{p}.mix", l, H, self.row, s.width)
        if s.ffn:
            a = src.vector(f"{p}.mlp.act", 2).tolist()
            L.update(norm2=src.vector(f"{p}.norm2", H), norm2b=src.vector(f"{p}.norm2b", H),
                     ffn=UnaryFFN(src, f"{p}.mlp", H, self.row, s.ffn, ACT_XIELU, _softplus(a[0]), 0.5 + _softplus(a[1])))
        return L

    def new_state(self, n_slots: int) -> RecurrentState:
        widths = {l: L["lin"].width for l, L in zip(self.layer_ids, self.layers) if "lin" in L}
        return RecurrentState(n_slots, {"S": {l: torch.zeros(n_slots, w, dtype=torch.float32, device=self.device) for l, w in widths.items()}}, self.device)

    # ---- forward
    def _group_norm(self, x, w, branch=None, fresh=False):
        """Residual x (+ norm(branch output) with the branch's own weight) -> norm(x; w)."""
        delta, delta_w = branch if branch is not None else (None, None)
        return ops.group_norm(x, w, self.cfg.rms_eps, self.cfg.norm_groups, delta=delta, delta_w=delta_w, fresh=fresh, width=self.cfg.hidden,
                              out_dtype=self.act_dtype)

    def _run_layers(self, x, delta, fb: ForwardBatch, kv: KVCache, state):
        # the embedding rows are the first branch: the residual starts as their norm
        branch, fresh = (x, self.embed_norm), True
        x = torch.empty_like(x)
        for li, L in enumerate(self.layers):
            h = self._group_norm(x, L["norm1"], branch, fresh)
            m = L["attn"](h, fb, kv) if "attn" in L else L["lin"](h, fb, state)
            branch, fresh, f = (m, L["norm1b"]), False, None
            if "ffn" in L:
                f = L["ffn"](self._group_norm(x, L["norm2"], branch))
                branch = (f, L["norm2b"])
            if self.tap is not None:
                self.tap(li, m, f if f is not None else torch.zeros_like(m), x)
        return x, branch

    def _head(self, x, branch, fb: ForwardBatch):
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        hn = self._group_norm(x.index_select(0, rows), self.out_norm, (branch[0].index_select(0, rows), branch[1]))
        return self.lm_head(hn, out_f32=True)
