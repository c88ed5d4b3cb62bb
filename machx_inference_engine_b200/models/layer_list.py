"""Base of the graphs whose configuration lists its layers one by one: rows padded to whole vectors, a choice of compute dtype, cache pages with
a geometry per layer run."""
from __future__ import annotations

from typing import Optional

import torch

from ..formats.model_config import ModelConfig
from ..ops import PoolPages, QuantWeight
from ..parallel.comm import ParallelCtx
from .transformer import KVCache, TransformerModel, round_up


class LayerListModel(TransformerModel):
    """The model runs in bf16 (matrix products and activations) or, with ``dtype="fp32"``, in 32-bit throughout.  Residual and activation rows are
    padded to a multiple of 32 columns; the padding is zero everywhere.  One GPU."""

    COMPUTE_DTYPES = ("bf16", "fp32")

    def __init__(self, cfg: ModelConfig, src, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
        par = par or ParallelCtx()
        if par.world > 1:
            raise ValueError(f"the {type(self).__name__.removesuffix('Model')} graph runs on one GPU")
        self.dtype = dtype
        self.act_dtype = {"bf16": torch.bfloat16, "fp32": torch.float32}[dtype]
        self.row = round_up(cfg.hidden, 32)              # columns of a residual / activation row
        self._tables: dict = {}
        super().__init__(cfg, src, device, par, max_ctx=max_ctx)
        self.kv_geometry = self._kv_geometry()           # per layer run: (kv heads, key width, value width)
        self.n_kv_local = max([g[0] for g in self.kv_geometry.values()], default=0)

    def _kv_geometry(self) -> dict:
        raise NotImplementedError

    def _vocab_matrix(self, src, name: str) -> QuantWeight:
        return super()._vocab_matrix(src, name).pad_groups(cols=(1, self.row))

    def _table(self, key, build):
        """A position table that several layers share."""
        if key not in self._tables:
            self._tables[key] = build()
        return self._tables[key]

    def _kv_pools(self) -> dict:
        """Per layer run with pooled blocks: (tokens per block, window)."""
        return {}

    def new_kv_cache(self, num_blocks: int, dtype: str = "bf16") -> KVCache:
        if dtype == "int8":
            raise ValueError("the int8 KV cache is not built for this design")
        return KVCache(self.cfg.n_layers, num_blocks, self.n_kv_local, self.cfg.head_dim, self.device, list(self.kv_geometry), dtype=self.dtype,
                       geometry=self.kv_geometry, pools=self._kv_pools())

    def kv_bytes_per_block(self, dtype: str = "bf16") -> int:
        pools = self._kv_pools()
        rows = lambda l: KVCache.BLOCK + (PoolPages.rows_per_page(KVCache.BLOCK, pools[l][0]) if l in pools else 0)
        return sum(n * (dk + dv) * rows(l) for l, (n, dk, dv) in self.kv_geometry.items()) * (2 if self.dtype == "bf16" else 4)
