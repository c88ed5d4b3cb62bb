"""Model graphs.  ``load_model`` opens a checkpoint (a GGUF file, or a folder with config.json + safetensors); ``build_model``
random-initialises a named architecture."""
from __future__ import annotations

import os
from typing import Optional

from ..formats.model_config import ModelConfig, read_config, read_json_config
from ..parallel.comm import ParallelCtx

# file names of the tensors that every graph asks for under its GGUF name
_FOLDER_NAMES = {"tikarax": {"token_embd.weight": "embed", "output_norm.weight": "final.norm", "output.weight": "head"},
                 "pubodra": {"token_embd.weight": "embed", "output_norm.weight": "final.norm"},
                 "beputar": {"token_embd.weight": "embed", "output_norm.weight": "final.norm"},
                 "zegelix": {"token_embd.weight": "embed", "output_norm.weight": "final.norm"}}


def _graph_class(cfg: ModelConfig):
    if cfg.is_hybrid:
        from .hybrid import HybridModel
        return HybridModel
    if cfg.arch == "gemma4":
        from .gemma4 import Gemma4Model
        return Gemma4Model
    if cfg.arch == "tikarax":
        from .tikarax import TikaraxModel
        return TikaraxModel
    if cfg.arch == "pubodra":
        from .pubodra import PubodraModel
        return PubodraModel
    if cfg.arch == "beputar":
        from .beputar import BeputarModel
        return BeputarModel
    if cfg.arch == "zegelix":
        from .zegelix import ZegelixModel
        return ZegelixModel
    from .transformer import TransformerModel
    return TransformerModel


def _build(cfg: ModelConfig, src, device, par, max_ctx: int, dtype: str):
    cls = _graph_class(cfg)
    have = getattr(cls, "COMPUTE_DTYPES", ("bf16",))
    if dtype not in have:
        raise ValueError(f"{cfg.arch} models run in {' or '.join(have)}, not {dtype}")
    return cls(cfg, src, device, par or ParallelCtx(), max_ctx=max_ctx, **({"dtype": dtype} if len(have) > 1 else {}))


def build_model(cfg: ModelConfig, device, par: Optional[ParallelCtx] = None, quant: str = "q8_0", max_ctx: int = 8192, seed: int = 0,
                gen_device=None, dtype: str = "bf16"):
    """Random-init weights of architecture ``cfg`` quantised with recipe ``quant`` directly on ``device``."""
    from .sources import SynthSource, default_policy
    src = SynthSource(device, default_policy(cfg.arch, quant), seed=seed, n_layers=cfg.n_layers, gen_device=gen_device)
    return _build(cfg, src, device, par, max_ctx, dtype)


def load_model(path: str, device, par: Optional[ParallelCtx] = None, max_ctx: int = 8192, dtype: str = "bf16"):
    """Loads a checkpoint onto ``device``; returns (model, reader).  ``path``: a GGUF file (split shards are merged) or a folder with
    config.json and safetensors.  ``dtype``: "bf16", or "fp32" for graphs that also run in 32-bit."""
    if os.path.isdir(path):
        from ..formats.safetensors import SafetensorsModel
        from .sources import SafetensorsSource
        cfg = read_json_config(path)
        reader = SafetensorsModel(path)
        cfg.name = cfg.name or os.path.basename(os.path.abspath(path))
        reader.kv = {"general.architecture": cfg.arch, "general.name": cfg.name}
        src = SafetensorsSource(reader, device, _FOLDER_NAMES.get(cfg.arch))
    else:
        from ..formats.gguf import GGUFReader
        from .sources import GGUFSource
        reader = GGUFReader(path)
        cfg = read_config(reader.kv, reader.tensors.keys())
        src = GGUFSource(reader, device)
    return _build(cfg, src, device, par, min(max_ctx, max(cfg.ctx_train, 256)), dtype), reader
