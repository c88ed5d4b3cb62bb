"""Beputar: three mixers in any order -- windowed attention whose values are its projected keys, RWKV-style time mixing, and attention beside lightning
attention -- with norms on the sublayers' outputs only, dense or routed feed-forwards whose routing weight scales the experts' input, and a tied head.

    x = scale embed[token]
    layer:  x <- x + ls1 norm(mixer(x); norm1);  x <- x + ls2 norm(ff(x); norm2)             (layers may have no feed-forward)
    logits = embed norm(x; final.norm)

norm(x; w) = x / rms(x) w, eps inside the root; the sublayers read the residual itself.
attention:  q = W_q h + b_q, k = W_k h + b_k, values k; q and k rotated in interleaved pairs (YaRN where asked for), then divided by their rms per head;
            softmax over the last ``window`` keys; W_o.
parallel:   1/2 (norm(left h; left.out) + norm(right h; right.out)).
    left:   q, k without biases, values k; per-head norms with weights, then rotation in half splits; the last ``window`` and the first ``keep_first``
            keys; one more score of 0 in the denominator; head h times sigmoid(W_g h)_h; W_o.
    right:  q, k, v = silu(W h); S <- decay S + k v^T, o = S^T q per head; (norm(o; norm) sigmoid(W_g h)) through W_o.
wkv:        mix_n = h + (h' - h) mu_n with h' the previous token's row, n = r, k, v, g, w; w = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0));
            o = (S + (u k) v^T)^T r, S <- diag(w) S + k v^T per head; (o / rms(o) per head, times norm, times silu(W_g mix_g)) through W_o.
ff:         W_down gelu_tanh(W_up h), or sum over the chosen e of expert_e(sigmoid(z_e) h) + shared(h), expert = W_down (silu(W_gate h) W_up h).

Launches of a layer: sublayer_norm (norm of the previous branch -- a row, the mean of two normed rows, or the sum of a token's expert rows, formed as
they are read --, layer scale, residual add, the next sublayer's input), the mixer's own (see the blocks), sublayer_norm, up and down projections; expert
layers: router, routing, scaled rows, the experts' two projections and the shared expert's.  Layer scale and norm weight are one vector.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..formats.model_config import ModelConfig
from ..ops import ACT_GELU_TANH
from ..parallel.comm import ParallelCtx
from ..utils.rope import rope_tables
from .hybrid import DecayAttentionBlock, ParallelMixer, RecurrentState, WkvBlock
from .layer_list import LayerListModel
from .transformer import ForwardBatch, KVCache, KeyValueAttentionBlock, ScaledInputMoEFFN, UnaryFFN


class BeputarModel(LayerListModel):
    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
        super().__init__(cfg, src, device, par, max_ctx=max_ctx, dtype=dtype)
        self.out_norm = self._row_vector(self.out_norm)

    @property
    def needs_state(self) -> bool:
        return any("lin" in L for L in self.layers)

    # ---- construction
    def _row_vector(self, v: torch.Tensor) -> torch.Tensor:
        return torch.nn.functional.pad(v, (0, self.row - v.numel())).contiguous()

    def _kv_geometry(self) -> dict:
        return {l: (L["attn"].n_kv, L["attn"].dp, L["attn"].dp) for l, L in zip(self.layer_ids, self.layers) if "attn" in L}

    def _rope(self, s) -> tuple:
        f, orig, fast, slow = s.yarn if s.yarn is not None else (1.0, 0, 32.0, 1.0)
        return self._table((s.rot_dim, s.rope_theta, s.yarn),
                           lambda: rope_tables(self.max_ctx, s.rot_dim, s.rope_theta, scaling_type="none" if s.yarn is None else "yarn", scaling_factor=f,
                                               orig_ctx=orig, beta_fast=fast, beta_slow=slow, device=self.device))

    def _attention(self, l: int, src, prefix: str, s, **kind) -> KeyValueAttentionBlock:
        return KeyValueAttentionBlock(src, prefix, l, self.cfg.hidden, self.row, s.heads, s.kv_heads, s.key_dim, s.scale, s.window, s.keep_first, s.rot_dim,
                                      self._rope(s), self.cfg.rms_eps, **kind)

    def _build_layer(self, l: int, src) -> dict:
        s, H, p, eps = self.cfg.layer_specs[l], self.cfg.hidden, f"l{l}", self.cfg.rms_eps
        vec = lambda name: src.vector(f"{p}.{name}", H)
        L = {"scale1": self._row_vector(vec("norm1") * vec("ls1"))}
        if s.mixer == "rotary_attention":
            L["attn"] = self._attention(l, src, f"{p}.mix", s, interleaved=True, biased=True, norm_after=True).own_projection()
        elif s.mixer == "wkv":
            L["lin"] = L["wkv"] = WkvBlock(src, f"{p}.mix", l, H, self.row, s.lin_heads, s.lin_key_dim, s.decay_rank, eps, self.act_dtype)
        else:
            L["attn"] = self._attention(l, src, f"{p}.mix.left", s, qk_norm=True, head_gate=True, zero_sink=True)
            L["lin"] = DecayAttentionBlock(src, f"{p}.mix.right", l, H, self.row, s.lin_heads, s.lin_key_dim, s.lin_value_dim, s.lin_decay, eps)
            L["parallel"] = ParallelMixer(L["attn"], L["lin"], self._row_vector(vec("mix.left.out")), self._row_vector(vec("mix.right.out")))
        if s.ffn or s.experts:
            L["scale2"] = self._row_vector(vec("norm2") * vec("ls2"))
        if s.experts:
            L["moe"] = ScaledInputMoEFFN(src, f"{p}.mlp", H, self.row, s.experts, s.experts_used, s.expert_ffn, s.shared_ffn)
        elif s.ffn:
            L["ffn"] = UnaryFFN(src, f"{p}.mlp", H, self.row, s.ffn, ACT_GELU_TANH)
        return L

    def new_state(self, n_slots: int) -> RecurrentState:
        tensors: dict = {"S": {}, "shift": {}}
        for l, L in zip(self.layer_ids, self.layers):
            for name, shape in (L["lin"].state_shape.items() if "lin" in L else ()):
                tensors[name][l] = torch.zeros(n_slots, *shape, dtype=torch.float32, device=self.device)
        return RecurrentState(n_slots, tensors, self.device)

    # ---- forward
    def _fold(self, x, branch, w=None, want_out=True):
        """Residual x + the normed and scaled branch; returns what the next sublayer reads (with ``w``: the norm of x)."""
        delta, scale = branch if branch is not None else (None, None)
        return ops.sublayer_norm(x, delta, scale, self.cfg.rms_eps, w=w, width=self.cfg.hidden, out_dtype=self.act_dtype, want_out=want_out)

    def _run_layers(self, x, delta, fb: ForwardBatch, kv: KVCache, state):
        branch = None
        for li, L in enumerate(self.layers):
            if "wkv" in L:                       # reads the fp32 rows, of the previous token too
                if branch is not None:
                    self._fold(x, branch, want_out=False)
                m = L["wkv"](x, fb, state)
            else:
                h = self._fold(x, branch)
                m = L["parallel"](h, fb, kv, state) if "parallel" in L else L["attn"](h, fb, kv)
            branch, f = (m, L["scale1"]), None
            if "scale2" in L:
                h = self._fold(x, branch)
                f = L["moe"](h) if "moe" in L else L["ffn"](h)
                branch = (f, L["scale2"])
            if self.tap is not None:
                rows = lambda b: b if isinstance(b, torch.Tensor) else b.materialize(self.cfg.rms_eps, self.cfg.hidden)
                self.tap(li, rows(m), rows(f) if f is not None else torch.zeros_like(x), x)
        return x, branch

    def _head(self, x, branch, fb: ForwardBatch):
        rows = fb.logit_rows if fb.logit_rows is not None else (fb.cu_q[1:].long() - 1)
        delta = branch[0].index_select(0, rows) if isinstance(branch[0], torch.Tensor) else branch[0].rows(rows)
        return self.lm_head(self._fold(x.index_select(0, rows), (delta, branch[1]), w=self.out_norm), out_f32=True)
