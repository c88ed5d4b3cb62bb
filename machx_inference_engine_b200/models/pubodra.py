"""Pubodra: latent attention with sliding windows, dynamic-tanh norms, dense and routed feed-forwards without a gate branch, and a range of layers
that runs several times with the same weights.

    x = embed[token]
    layer:  x <- x + mixer(norm(x; norm1));  x <- x + ff(norm(x; norm2))           (layers may have no feed-forward)
    loop:   layers start .. stop - 1 run ``times`` times; pass t begins with x <- x + step[t] and has its own cache
    logits = embed norm(x; final.norm)

norm(x) = tanh(alpha x) w + b, element by element.
mixer:  [q_u | q_r] = W_q h per head; [d | k_r] = W_dkv h; c = d / rms(d) * w; keys [W_uk c | k_r], values W_uv c; q_r and k_r rotated in
        interleaved pairs (YaRN frequencies where the layer asks for them, whose magnitude factor the rotation carries); softmax over the last
        ``window`` keys of (q . k) scale; the heads times sigmoid(W_g h); W_o.  The cache holds [c | k_r].
ff:     W_down gelu_tanh(W_up h), or the weighted sum of the best ``used`` of ``experts`` W_down relu(W_up h)^2.

Launches of a layer: dyt_norm (adds the previous branch to the fp32 residual, norms the sum), the fused projection, the head epilogue (latent norm,
rotation, cache row), attention in the latent space between two per-head products or over expanded keys, output projection, dyt_norm, up projection
with the activation, down projection; expert layers: router, routing, up and down projections of the chosen experts, whose weighted sum is formed
in the next dyt_norm.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..formats.model_config import ModelConfig
from ..ops import ACT_GELU_TANH, ACT_RELU2
from ..parallel.comm import ParallelCtx
from ..utils.rope import rope_tables
from .layer_list import LayerListModel
from .transformer import ForwardBatch, KVCache, LatentAttentionBlock, UnaryFFN, UnaryMoEFFN


class DynamicTanh:
    """Weights of one norm, padded to the row width (a padded column stays zero)."""

    def __init__(self, src, name: str, hidden: int, row: int):
        self.alpha = src.scalar(f"{name}.alpha")
        pad = lambda v: torch.nn.functional.pad(v, (0, row - hidden)).contiguous()
        self.w, self.b = pad(src.vector(name, hidden)), pad(src.vector(f"{name}.b", hidden))


class PubodraModel(LayerListModel):
    split_query_len = LatentAttentionBlock.EXPAND_MIN_Q      # the engine puts shorter queries of a batch first: they take another path

    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
        self.runs = cfg.layer_runs()
        super().__init__(cfg, src, device, par, max_ctx=max_ctx, dtype=dtype)
        self.final_norm = DynamicTanh(src, "final.norm", cfg.hidden, self.row)
        self.loop_step = None
        if cfg.loop_times:
            step = src.table("loop.step", (cfg.loop_times, cfg.hidden))
            self.loop_step = torch.nn.functional.pad(step, (0, self.row - cfg.hidden)).contiguous()

    # ---- construction
    def _kv_geometry(self) -> dict:
        at = [self.layers[l]["attn"] for l, _ in self.runs]
        return {i: (1, a.R + a.r, 0) for i, a in enumerate(at)}

    def _rope(self, s) -> tuple:
        f, orig, fast, slow = s.yarn if s.yarn is not None else (1.0, 0, 32.0, 1.0)
        return self._table((s.rot_dim, s.rope_theta, s.yarn),
                           lambda: rope_tables(self.max_ctx, s.rot_dim, s.rope_theta, scaling_type="none" if s.yarn is None else "yarn", scaling_factor=f,
                                               orig_ctx=orig, beta_fast=fast, beta_slow=slow, device=self.device))

    def _build_layer(self, l: int, src) -> dict:
        s, H, p = self.cfg.layer_specs[l], self.cfg.hidden, f"l{l}"
        L = {"norm1": DynamicTanh(src, f"{p}.norm1", H, self.row),
             "attn": LatentAttentionBlock(src, f"{p}.mix", H, self.row, s.heads, s.key_dim, s.rot_dim, s.value_dim, s.kv_rank, s.scale, s.window,
                                          self.cfg.rms_eps, self._rope(s))}
        if s.ffn or s.experts:
            L["norm2"] = DynamicTanh(src, f"{p}.norm2", H, self.row)
        if s.experts:
            L["moe"] = UnaryMoEFFN(src, f"{p}.mlp", H, self.row, s.experts, s.experts_used, s.expert_ffn, ACT_RELU2)
        elif s.ffn:
            L["ffn"] = UnaryFFN(src, f"{p}.mlp", H, self.row, s.ffn, ACT_GELU_TANH)
        return L

    # ---- forward
    def _dyt(self, x, n: DynamicTanh, delta=None, step=None):
        """Residual x (+ branch output, + a pass's vector) -> norm(x)."""
        return ops.dyt_norm(x, n.alpha, n.w, n.b, delta=delta, step=step, out_dtype=self.act_dtype)

    def _run_layers(self, x, delta, fb: ForwardBatch, kv: KVCache, state):
        plans: dict = {}                  # page lists of the long queries, shared by the layers of one window
        for i, (l, t) in enumerate(self.runs):
            L = self.layers[l]
            m = L["attn"](self._dyt(x, L["norm1"], delta, None if t is None else self.loop_step[t]), fb, kv.k[i], plans)
            delta, f = m, None
            if "norm2" in L:
                h = self._dyt(x, L["norm2"], m)
                f = delta = L["moe"](h, self.par) if "moe" in L else L["ffn"](h)
            if self.tap is not None:
                if f is not None and not isinstance(f, torch.Tensor):
                    f = delta = f.materialize()
                self.tap(i, m, f if f is not None else torch.zeros_like(m), x)
        return x, delta

    def _head(self, x, delta, fb: ForwardBatch):
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        delta = delta.index_select(0, rows) if isinstance(delta, torch.Tensor) else delta.rows(rows)
        return self.lm_head(self._dyt(x.index_select(0, rows), self.final_norm, delta), out_f32=True)
