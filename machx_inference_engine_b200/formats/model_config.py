"""Architecture detection and one typed config for every model family.

Reference parity: src/loaders/model_config.cpp:8-359 and include/ie/model_config.hpp:12-254
(``detect_arch``, ``read_dense_config``, ``read_{qwen35,qwen3moe,gptoss,qwen3next,gemma4}_config``,
template-family classification, sliding-window load guard, Granite scalars).  The reference
keeps one struct per family; here one dataclass serves all graphs.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field, asdict
from typing import Any, Mapping, Optional

DENSE_ARCHS = ("llama", "qwen2", "qwen3", "phi3", "granite", "mistral")
MOE_ARCHS = ("qwen3moe", "gpt-oss")
HYBRID_ARCHS = ("qwen3next", "qwen35", "qwen35moe")
GEMMA_ARCHS = ("gemma4",)
SUPPORTED_ARCHS = DENSE_ARCHS + MOE_ARCHS + HYBRID_ARCHS + GEMMA_ARCHS
# checkpoints that are a folder with config.json + safetensors and list their layers one by one: "architecture" value -> arch
LAYER_LIST_ARCHS = {"Tikarax": "tikarax", "Pubodra": "pubodra", "Beputar": "beputar", "Zegelix": "zegelix"}


class ConfigError(ValueError):
    pass


@dataclass
class LayerSpec:
    """One layer of a design whose configuration lists its layers: a mixer with its sizes and constants, and a feed-forward (``ffn`` wide, or
    ``experts`` of ``expert_ffn`` each with ``experts_used`` per token; none when both are 0)."""
    mixer: str                     # "attention" | "mingru" | "latent_attention" | "rotary_attention" | "wkv" | "parallel" | "pooled_attention" | "rglru"
    ffn: int = 0
    experts: int = 0
    experts_used: int = 0
    expert_ffn: int = 0
    # attention without rotation, with its own value width, query temperature and output gate
    heads: int = 0
    kv_heads: int = 0
    key_dim: int = 0
    value_dim: int = 0
    scale: float = 0.0
    q_temp_coef: float = 0.0       # queries at position p are multiplied by 1 + coef * ln(floor((p + 1) / every) + 1)
    q_temp_every: float = 1.0
    # latent attention: key_dim above is the unrotated part of a head, kv_heads stays 0 (one latent row per token serves all heads)
    kv_rank: int = 0
    rot_dim: int = 0
    window: int = 0                # keys a query sees, itself included (0 = all before it)
    rope_theta: float = 10000.0
    yarn: Optional[tuple] = None   # (factor, original context, fast turns, slow turns)
    # minGRU, RG-LRU
    width: int = 0
    # attention over a window and pooled blocks before it: heads .. scale, rot_dim .. rope_theta and window above
    pool: int = 0                  # tokens of a pooled block (0: what left the window is gone)
    softcap: float = 0.0           # scores are softcap * tanh(score / softcap) (0: as they are)
    # RG-LRU: width channels in gate_blocks equal parts behind a causal convolution
    gate_blocks: int = 0
    conv_taps: int = 0
    # clamped gated experts
    act_limit: float = 0.0
    shared_limit: float = 0.0
    # rotary attention (and the left half of a parallel mixer): heads .. scale and rot_dim .. yarn above
    keep_first: int = 0            # with a window: the first tokens of a sequence that stay visible
    # experts whose weight scales their input
    shared_ffn: int = 0            # width of the expert that every token uses (0: none)
    # recurrences with a matrix per head (wkv, the right half of a parallel mixer)
    lin_heads: int = 0
    lin_key_dim: int = 0
    lin_value_dim: int = 0
    lin_decay: tuple = ()          # per head; empty where the decay comes from the data
    decay_rank: int = 0            # wkv: inner width of the decay's projection (0: as the checkpoint's tensor has it)

    def kv_width(self) -> float:
        """Cached elements per token (a pooled block's rows count for its tokens)."""
        return self.kv_heads * (self.key_dim + self.value_dim) * (1 + (1 / self.pool if self.pool else 0)) + (self.kv_rank + self.rot_dim if self.kv_rank else 0)

    def state_bytes(self, hidden: int) -> int:
        """Recurrent state per sequence (fp32): the minGRU / RG-LRU row with the convolution's last inputs, or a matrix per head and, for wkv, the last
        row of its input."""
        return 4 * (self.width * max(self.conv_taps, 1) + self.lin_heads * self.lin_key_dim * self.lin_value_dim + (hidden if self.mixer == "wkv" else 0))


@dataclass
class ModelConfig:
    arch: str = "llama"
    n_layers: int = 0
    hidden: int = 0
    n_heads: int = 0
    n_kv_heads: int = 0
    head_dim: int = 0
    ffn: int = 0
    vocab: int = 0
    rms_eps: float = 1e-5
    rope_theta: float = 10000.0
    n_rot: int = 0
    ctx_train: int = 4096
    sliding_window: int = 0
    # rope scaling (YaRN for gpt-oss, llama3 frequency factors come as a tensor)
    rope_scaling_type: str = "none"
    rope_scaling_factor: float = 1.0
    rope_orig_ctx: int = 0
    yarn_beta_fast: float = 32.0
    yarn_beta_slow: float = 1.0
    # mixture of experts
    n_experts: int = 0
    n_experts_used: int = 0
    expert_ffn: int = 0
    shared_expert_ffn: int = 0
    # hybrid (gated DeltaNet) models
    full_attn_interval: int = 0
    ssm_inner: int = 0
    ssm_state: int = 0
    ssm_n_k_heads: int = 0
    ssm_n_v_heads: int = 0
    ssm_conv_kernel: int = 0
    nextn_predict_layers: int = 0
    # Gemma-4: two head geometries chosen per layer (include/ie/model_config.hpp:216-249); head_dim / n_rot / rope_theta above
    # describe the global (full-attention) layers, the *_swa fields the sliding-window layers
    head_dim_swa: int = 0
    n_rot_swa: int = 0
    rope_theta_swa: float = 10000.0
    layer_swa: list = field(default_factory=list)        # per layer: True = sliding-window layer
    layer_n_kv: list = field(default_factory=list)       # per layer: KV head count
    # designs that list their layers (LAYER_LIST_ARCHS): head_dim / n_heads / n_kv_heads / ffn above are the largest of any layer
    layer_specs: list = field(default_factory=list)      # LayerSpec per layer
    norm_groups: int = 1                                  # RMS norms run over this many equal parts of the row
    loop_start: int = 0                                   # layers loop_start .. loop_stop - 1 run loop_times times in a row (0: no loop); every
    loop_stop: int = 0                                    # pass has its own cache or state and first adds a learned vector to the residual or mixes it
    loop_times: int = 0                                   # with the embedding output
    # Granite scalars
    embedding_scale: float = 1.0
    residual_scale: float = 1.0
    attention_scale: float = 0.0       # 0 -> 1/sqrt(head_dim)
    logit_scale: float = 1.0
    final_logit_softcap: float = 0.0
    template_family: str = "auto"      # chatml | llama3 | mistral | deepseek | granite | gemma | harmony | auto
    mistral_sysprompt: bool = False
    tie_embeddings: bool = False
    name: str = ""

    # ---- derived
    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    @property
    def is_hybrid(self) -> bool:
        return self.arch in HYBRID_ARCHS

    def layer_is_full_attention(self, layer: int) -> bool:
        if self.layer_specs:
            return self.layer_specs[layer].mixer in ("attention", "latent_attention", "rotary_attention", "parallel", "pooled_attention")
        if not self.is_hybrid:
            return True
        return (layer + 1) % self.full_attn_interval == 0

    def layer_runs(self) -> list:
        """(layer, number of the pass that begins with it or None) in the order of execution."""
        if not self.loop_times:
            return [(l, None) for l in range(self.n_layers)]
        a, b = self.loop_start, self.loop_stop
        return ([(l, None) for l in range(a)] + [(l, t if l == a else None) for t in range(self.loop_times) for l in range(a, b)]
                + [(l, None) for l in range(b, self.n_layers)])

    def layer_window(self, layer: int) -> int:
        """Sliding window of a layer (0 = full).  gpt-oss windows the even layers (src/model/gptoss.cpp:133), Gemma-4 the
        layers its pattern marks (src/model/gemma4.cpp:709-714)."""
        if self.arch == "gpt-oss":
            return self.sliding_window if layer % 2 == 0 else 0
        if self.arch == "gemma4":
            return self.sliding_window if self.layer_swa[layer] else 0
        if self.layer_specs:
            return self.layer_specs[layer].window
        return self.sliding_window

    def layer_geometry(self, layer: int) -> tuple:
        """(head_dim, n_kv_heads, n_rot, rope_theta) of a layer."""
        if self.arch == "gemma4":
            swa = bool(self.layer_swa[layer])
            return (self.head_dim_swa if swa else self.head_dim, int(self.layer_n_kv[layer]), self.n_rot_swa if swa else self.n_rot,
                    self.rope_theta_swa if swa else self.rope_theta)
        return (self.head_dim, self.n_kv_heads, self.n_rot, self.rope_theta)

    def to_dict(self) -> dict:
        return asdict(self)


def detect_arch(kv: Mapping[str, Any]) -> str:
    a = kv.get("general.architecture")
    if a is None:
        raise ConfigError("GGUF has no general.architecture")
    if a not in SUPPORTED_ARCHS:
        raise ConfigError(f"unsupported architecture '{a}' (supported: {', '.join(SUPPORTED_ARCHS)})")
    return a


def classify_template_family(chat_template: str, arch: str = "") -> str:
    ct = chat_template or ""
    if "[INST]" in ct:
        return "mistral"
    if "<|start_header_id|>" in ct:
        return "llama3"
    if "<｜Assistant｜>" in ct:
        return "deepseek"
    if "<|start_of_role|>" in ct:
        return "granite"
    if "<|start|>" in ct and "<|channel|>" in ct or arch == "gpt-oss":
        return "harmony"
    if "<start_of_turn>" in ct:
        return "gemma"
    if "<|im_start|>" in ct:
        return "chatml"
    return "auto"


def read_config(kv: Mapping[str, Any], tensor_names=()) -> ModelConfig:
    arch = detect_arch(kv)
    c = ModelConfig(arch=arch, name=str(kv.get("general.name", "")))

    def get(suffix, default=None, required=False):
        k = f"{arch}.{suffix}"
        if k in kv and kv[k] is not None:
            return kv[k]
        if required:
            raise ConfigError(f"missing {k}")
        return default

    c.n_layers = int(get("block_count", required=True))
    c.hidden = int(get("embedding_length", required=True))
    c.n_heads = int(get("attention.head_count", required=True))
    hkv = get("attention.head_count_kv", c.n_heads)
    if isinstance(hkv, (list, tuple)):                                     # per-layer arrays: take the max
        c.n_kv_heads = max([int(v) for v in hkv if v] or [c.n_heads])
    else:
        c.n_kv_heads = int(hkv)
    c.ffn = int(get("feed_forward_length", 0) or 0)
    c.head_dim = int(get("attention.key_length", c.hidden // c.n_heads))
    c.n_rot = int(get("rope.dimension_count", c.head_dim))
    c.ctx_train = int(get("context_length", 4096))
    c.rope_theta = float(get("rope.freq_base", 10000.0))
    c.rms_eps = float(get("attention.layer_norm_rms_epsilon", 1e-5))
    c.sliding_window = int(get("attention.sliding_window", 0) or 0)
    if arch != "gpt-oss" and c.sliding_window and c.sliding_window < c.ctx_train:
        # every attention kernel here takes a window argument, so a windowed dense checkpoint is
        # served correctly (the reference refuses to load it); nothing to do
        pass
    if c.sliding_window >= c.ctx_train:
        c.sliding_window = 0
    c.embedding_scale = float(get("embedding_scale", 1.0))
    c.residual_scale = float(get("residual_scale", 1.0))
    c.attention_scale = float(get("attention.scale", 0.0))
    ls = float(get("logit_scale", 1.0))
    c.logit_scale = 1.0 / ls if (arch == "granite" and ls) else 1.0       # Granite divides logits by logits_scaling
    c.final_logit_softcap = float(get("final_logit_softcapping", 0.0))
    toks = kv.get("tokenizer.ggml.tokens")
    c.vocab = len(toks) if toks is not None else int(get("vocab_size", 0) or 0)
    if c.vocab == 0:
        raise ConfigError("missing tokenizer.ggml.tokens (vocabulary size unknown)")
    c.template_family = classify_template_family(str(kv.get("tokenizer.chat_template", "")), arch)
    c.mistral_sysprompt = "[SYSTEM_PROMPT]" in str(kv.get("tokenizer.chat_template", ""))
    c.rope_scaling_type = str(get("rope.scaling.type", "none"))
    c.rope_scaling_factor = float(get("rope.scaling.factor", 1.0))
    c.rope_orig_ctx = int(get("rope.scaling.original_context_length", 0) or 0)

    if arch == "gemma4":
        c.head_dim_swa = int(get("attention.key_length_swa", required=True))
        c.n_rot_swa = int(get("rope.dimension_count_swa", c.head_dim_swa))
        c.rope_theta_swa = float(get("rope.freq_base_swa", 10000.0))
        pat = get("attention.sliding_window_pattern", None)
        c.layer_swa = [bool(v) for v in pat] if isinstance(pat, (list, tuple)) else [False] * c.n_layers
        hk = get("attention.head_count_kv", required=True)
        c.layer_n_kv = [int(v) for v in hk] if isinstance(hk, (list, tuple)) else [int(hk)] * c.n_layers
        if len(c.layer_swa) != c.n_layers or len(c.layer_n_kv) != c.n_layers:
            raise ConfigError("gemma4: per-layer arrays do not match block_count")
        if any(c.n_heads % max(v, 1) for v in c.layer_n_kv):
            raise ConfigError("gemma4: attention.head_count is not a multiple of a layer's head_count_kv")
        c.embedding_scale = float(c.hidden) ** 0.5
        c.attention_scale = 1.0                 # q and k are RMS-normalised per head; the reference's net scale is 1
        if int(get("expert_count", 0) or 0) > 0:
            c.n_experts = int(get("expert_count"))
            c.n_experts_used = int(get("expert_used_count", required=True))
            c.expert_ffn = int(get("expert_feed_forward_length", required=True))
    if arch in ("qwen3moe", "gpt-oss", "qwen3next", "qwen35moe"):
        c.n_experts = int(get("expert_count", required=True))
        c.n_experts_used = int(get("expert_used_count", required=True))
        c.expert_ffn = int(get("expert_feed_forward_length", c.ffn) or c.ffn)
        c.shared_expert_ffn = int(get("expert_shared_feed_forward_length", 0) or 0)
        if c.n_experts_used > c.n_experts:
            raise ConfigError("expert_used_count exceeds expert_count")
    if arch in HYBRID_ARCHS:
        c.full_attn_interval = int(get("full_attention_interval", 4))
        if c.full_attn_interval <= 0:
            raise ConfigError(f"{arch}.full_attention_interval is zero")
        c.ssm_inner = int(get("ssm.inner_size", required=True))
        c.ssm_state = int(get("ssm.state_size", required=True))
        c.ssm_n_k_heads = int(get("ssm.group_count", required=True))
        c.ssm_n_v_heads = int(get("ssm.time_step_rank", required=True))
        c.ssm_conv_kernel = int(get("ssm.conv_kernel", required=True))
        if c.ssm_n_v_heads == 0:
            raise ConfigError(f"{arch}.ssm.time_step_rank is zero")
        c.nextn_predict_layers = int(get("nextn_predict_layers", 0) or 0)
    names = set(tensor_names)
    c.tie_embeddings = bool(names) and "output.weight" not in names
    for f in ("n_layers", "hidden", "n_heads", "head_dim"):
        if getattr(c, f) <= 0:
            raise ConfigError(f"invalid {f}={getattr(c, f)}")
    if c.n_heads % max(c.n_kv_heads, 1):
        raise ConfigError("attention.head_count is not a multiple of head_count_kv")
    return c


def _tikarax_config(d: Mapping[str, Any]) -> ModelConfig:
    c = ModelConfig(arch="tikarax", hidden=int(d["width"]), vocab=int(d["vocab"]), rms_eps=float(d["norm"]["eps"]), norm_groups=int(d["norm"]["groups"]),
                    name=str(d.get("name", "")))
    for i, e in enumerate(d["layers"]):
        m, mlp = e["mixer"], e.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ConfigError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        s = LayerSpec(e["type"], ffn=0 if mlp is None else int(mlp["ff"]))
        if s.mixer == "attention":
            s.heads, s.kv_heads, s.key_dim, s.value_dim, s.scale = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"])
            t = m.get("q_temp")
            if t is not None:
                s.q_temp_coef, s.q_temp_every = float(t["coef"]), float(t["every"])
                if s.q_temp_every <= 0:
                    raise ConfigError(f"layer {i}: q_temp.every must be positive")
            if s.kv_heads < 1 or s.heads % s.kv_heads:
                raise ConfigError(f"layer {i}: {s.heads} query heads do not divide over {s.kv_heads} key/value heads")
        elif s.mixer == "mingru":
            s.width = int(m["width"])
        else:
            raise ConfigError(f"layer {i}: unknown mixer {s.mixer!r}")
        c.layer_specs.append(s)
    if c.hidden < 1 or c.vocab < 1 or not c.layer_specs or c.norm_groups < 1 or c.hidden % c.norm_groups:
        raise ConfigError("the width must be positive and a multiple of norm.groups, with at least one layer")
    return _finish_layer_list(c)


def _pubodra_config(d: Mapping[str, Any]) -> ModelConfig:
    c = ModelConfig(arch="pubodra", hidden=int(d["width"]), vocab=int(d["vocab"]), rms_eps=float(d["norm"]["eps"]), tie_embeddings=True,
                    name=str(d.get("name", "")))
    for i, e in enumerate(d["layers"]):
        m, mlp = e["mixer"], e.get("mlp")
        if e["type"] != "latent_attention":
            raise ConfigError(f"layer {i}: unknown mixer {e['type']!r}")
        rot, mask = m["rot"], m.get("mask")
        s = LayerSpec("latent_attention", heads=int(m["heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                      rot_dim=int(m["rot_dim"]), scale=float(m["scale"]), rope_theta=float(rot["base"]))
        if min(s.heads, s.key_dim, s.value_dim, s.kv_rank, s.rot_dim) < 1 or s.rot_dim % 2 or int(rot["dims"]) != s.rot_dim:
            raise ConfigError(f"layer {i}: sizes must be positive and rot.dims the even rot_dim")
        if mask is not None:
            s.window = int(mask["size"])
            if s.window < 1:
                raise ConfigError(f"layer {i}: mask.size must be positive")
        if rot.get("scaling") is not None:
            y = rot["scaling"]
            s.yarn = (float(y["factor"]), float(y["original"]), float(y["fast"]), float(y["slow"]))
            if min(s.yarn) <= 0:
                raise ConfigError(f"layer {i}: rot.scaling values must be positive")
        kind = None if mlp is None else mlp.get("kind", "dense")
        if kind == "dense":
            s.ffn = int(mlp["ff"])
        elif kind == "moe":
            s.experts, s.experts_used, s.expert_ffn = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
            if not 1 <= s.experts_used <= s.experts:
                raise ConfigError(f"layer {i}: {s.experts_used} of {s.experts} experts per token")
        elif kind is not None:
            raise ConfigError(f"layer {i}: unknown feed-forward kind {kind!r}")
        c.layer_specs.append(s)
    _read_loop(c, d)
    if c.hidden < 1 or c.vocab < 1 or not c.layer_specs:
        raise ConfigError("the width must be positive, with at least one layer")
    return _finish_layer_list(c)


def _read_loop(c: ModelConfig, d: Mapping[str, Any]) -> None:
    if d.get("loop") is None:
        return
    c.loop_start, c.loop_stop, c.loop_times = (int(d["loop"][k]) for k in ("start", "stop", "times"))
    if not 0 <= c.loop_start < c.loop_stop <= len(c.layer_specs) or c.loop_times < 1:
        raise ConfigError("loop: start .. stop must be a range of layers that runs at least once")


def _yarn(rot: Mapping[str, Any], where: str) -> Optional[tuple]:
    y = rot.get("scaling")
    if y is None:
        return None
    out = (float(y["factor"]), float(y["original"]), float(y["fast"]), float(y["slow"]))
    if min(out) <= 0:
        raise ConfigError(f"{where}: rot.scaling values must be positive")
    return out


def _beputar_attention(s: LayerSpec, m: Mapping[str, Any], where: str) -> None:
    rot, mask = m["rot"], m.get("mask")
    s.heads, s.kv_heads, s.key_dim, s.value_dim, s.scale = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"])
    s.rot_dim, s.rope_theta, s.yarn = int(rot["dims"]), float(rot["base"]), _yarn(rot, where)
    if min(s.heads, s.kv_heads, s.key_dim) < 1 or s.heads % s.kv_heads:
        raise ConfigError(f"{where}: {s.heads} query heads do not divide over {s.kv_heads} key/value heads")
    if s.value_dim != s.key_dim:
        raise ConfigError(f"{where}: the values are the projected keys, so vdim must equal dim")
    if not 0 <= s.rot_dim <= s.key_dim or s.rot_dim % 2:
        raise ConfigError(f"{where}: rot.dims must be even and at most dim")
    if mask is not None:
        s.window, s.keep_first = int(mask["size"]), int(mask.get("keep_first", 0))
        if s.window < 1 or s.keep_first < 0:
            raise ConfigError(f"{where}: mask.size must be positive and keep_first not negative")


def _beputar_config(d: Mapping[str, Any]) -> ModelConfig:
    c = ModelConfig(arch="beputar", hidden=int(d["width"]), vocab=int(d["vocab"]), rms_eps=float(d["norm"]["eps"]), tie_embeddings=True,
                    embedding_scale=float(d["embedding"]["scale"]), name=str(d.get("name", "")))
    for i, e in enumerate(d["layers"]):
        m, mlp, where = e["mixer"], e.get("mlp"), f"layer {i}"
        if e["type"] == "attention":
            s = LayerSpec("rotary_attention")
            _beputar_attention(s, m, where)
        elif e["type"] == "wkv":
            s = LayerSpec("wkv", lin_heads=int(m["heads"]), lin_key_dim=int(m["dim"]), lin_value_dim=int(m["dim"]))
        elif e["type"] == "parallel":
            r = m["right"]
            s = LayerSpec("parallel", lin_heads=int(r["heads"]), lin_key_dim=int(r["dim"]), lin_value_dim=int(r["vdim"]),
                          lin_decay=tuple(float(v) for v in r["decay"]))
            _beputar_attention(s, m["left"], f"{where}, left")
            if len(s.lin_decay) != s.lin_heads:
                raise ConfigError(f"{where}: one decay per head")
        else:
            raise ConfigError(f"{where}: unknown mixer {e['type']!r}")
        if s.mixer != "rotary_attention" and min(s.lin_heads, s.lin_key_dim, s.lin_value_dim) < 1:
            raise ConfigError(f"{where}: sizes must be positive")
        kind = None if mlp is None else mlp.get("kind", "dense")
        if kind == "dense":
            s.ffn = int(mlp["ff"])
        elif kind == "moe":
            s.experts, s.experts_used, s.expert_ffn = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
            if mlp.get("shared") is not None:
                s.shared_ffn = int(mlp["shared"]["ff"])
            if not 1 <= s.experts_used <= s.experts:
                raise ConfigError(f"{where}: {s.experts_used} of {s.experts} experts per token")
        elif kind is not None:
            raise ConfigError(f"{where}: unknown feed-forward kind {kind!r}")
        c.layer_specs.append(s)
    if c.hidden < 1 or c.vocab < 1 or not c.layer_specs:
        raise ConfigError("the width must be positive, with at least one layer")
    return _finish_layer_list(c)


def _zegelix_config(d: Mapping[str, Any]) -> ModelConfig:
    c = ModelConfig(arch="zegelix", hidden=int(d["width"]), vocab=int(d["vocab"]), rms_eps=float(d["norm"]["eps"]), tie_embeddings=True,
                    embedding_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]), name=str(d.get("name", "")))
    for i, e in enumerate(d["layers"]):
        m, mlp, where = e["mixer"], e.get("mlp"), f"layer {i}"
        if e["type"] == "attention":
            rot, mask = m["rot"], m.get("mask")
            s = LayerSpec("pooled_attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                          scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), rot_dim=int(rot["dims"]), rope_theta=float(rot["base"]))
            if min(s.heads, s.kv_heads, s.key_dim, s.value_dim) < 1 or s.heads % s.kv_heads:
                raise ConfigError(f"{where}: {s.heads} query heads do not divide over {s.kv_heads} key/value heads")
            if not 0 <= s.rot_dim <= s.key_dim or s.rot_dim % 2 or s.value_dim % 2:
                raise ConfigError(f"{where}: rot.dims must be even and at most dim, and vdim even")
            if s.softcap < 0:
                raise ConfigError(f"{where}: softcap must not be negative")
            if mask is not None:
                s.window, s.pool = int(mask["size"]), int(mask.get("pool") or 0)
                if s.window < 1 or s.pool < 0:
                    raise ConfigError(f"{where}: mask.size must be positive and mask.pool not negative")
        elif e["type"] == "rglru":
            s = LayerSpec("rglru", width=int(m["width"]), gate_blocks=int(m["blocks"]), conv_taps=int(m["conv"]))
            if min(s.width, s.gate_blocks, s.conv_taps) < 1 or s.width % s.gate_blocks:
                raise ConfigError(f"{where}: the width must be a multiple of the blocks, with at least one tap")
        else:
            raise ConfigError(f"{where}: unknown mixer {e['type']!r}")
        if mlp is not None:
            if mlp.get("kind") != "moe":
                raise ConfigError(f"{where}: unknown feed-forward kind {mlp.get('kind')!r}")
            s.experts, s.experts_used, s.expert_ffn = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
            s.act_limit = float(mlp["expert"]["limit"])
            if mlp.get("shared") is not None:
                s.shared_ffn, s.shared_limit = int(mlp["shared"]["ff"]), float(mlp["shared"]["limit"])
            if not 1 <= s.experts_used <= s.experts:
                raise ConfigError(f"{where}: {s.experts_used} of {s.experts} experts per token")
        c.layer_specs.append(s)
    _read_loop(c, d)
    if c.hidden < 1 or c.vocab < 1 or not c.layer_specs:
        raise ConfigError("the width must be positive, with at least one layer")
    return _finish_layer_list(c)


def _finish_layer_list(c: ModelConfig) -> ModelConfig:
    """Derived fields of a layer-list config: the largest sizes of any layer (pool sizing, reports)."""
    big = lambda f, lo=0: max([lo] + [getattr(s, f) for s in c.layer_specs])
    c.n_layers = len(c.layer_specs)
    c.n_heads, c.n_kv_heads, c.ffn = big("heads", 1), big("kv_heads", 1), big("ffn")
    c.head_dim = max(big("key_dim", 1), big("value_dim"))
    c.n_experts, c.n_experts_used, c.expert_ffn = big("experts"), big("experts_used"), big("expert_ffn")
    c.shared_expert_ffn = big("shared_ffn")
    c.n_rot, c.ctx_train = 0, 1 << 20                      # rotations, where there are any, belong to the layers; positions have no limit of their own
    return c


def read_json_config(path_or_dict) -> ModelConfig:
    """config.json of a checkpoint folder (or the parsed dict) of a layer-list design."""
    d = path_or_dict
    if not isinstance(d, Mapping):
        p = os.path.join(d, "config.json") if os.path.isdir(d) else d
        with open(p) as f:
            d = json.load(f)
    a = d.get("architecture")
    readers = {"tikarax": _tikarax_config, "pubodra": _pubodra_config, "beputar": _beputar_config, "zegelix": _zegelix_config}
    if a not in LAYER_LIST_ARCHS:
        raise ConfigError(f"unsupported architecture {a!r} in config.json (supported: {', '.join(LAYER_LIST_ARCHS)})")
    try:
        return readers[LAYER_LIST_ARCHS[a]](d)
    except (KeyError, TypeError) as e:
        raise ConfigError(f"config.json of a {a} model: missing or malformed {e}") from e


def config_to_json(c: ModelConfig) -> dict:
    """Inverse of :func:`read_json_config`."""
    whole = lambda v: int(v) if float(v).is_integer() else v
    layers = []

    def rotation(s):
        rot = {"base": s.rope_theta, "dims": s.rot_dim}
        if s.yarn is not None:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), (s.yarn[0], whole(s.yarn[1]), s.yarn[2], s.yarn[3])))
        return rot

    def rotary(s):
        m = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.key_dim, "vdim": s.value_dim, "scale": s.scale, "rot": rotation(s)}
        if s.window:
            m["mask"] = {"size": s.window, **({"keep_first": s.keep_first} if s.keep_first else {})}
        return m

    for s in c.layer_specs:
        if s.mixer == "rotary_attention":
            m = rotary(s)
        elif s.mixer == "wkv":
            m = {"heads": s.lin_heads, "dim": s.lin_key_dim}
        elif s.mixer == "parallel":
            m = {"left": rotary(s), "right": {"heads": s.lin_heads, "dim": s.lin_key_dim, "vdim": s.lin_value_dim, "decay": list(s.lin_decay)}}
        elif s.mixer == "pooled_attention":
            m = {**rotary(s), **({"softcap": s.softcap} if s.softcap else {})}
            if s.pool:
                m["mask"]["pool"] = s.pool
        elif s.mixer == "rglru":
            m = {"width": s.width, "blocks": s.gate_blocks, "conv": s.conv_taps}
        elif s.mixer == "attention":
            m = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.key_dim, "vdim": s.value_dim, "scale": s.scale,
                 "q_temp": {"coef": s.q_temp_coef, "every": whole(s.q_temp_every)}}
        elif s.mixer == "latent_attention":
            m = {"heads": s.heads, "dim": s.key_dim, "rot_dim": s.rot_dim, "vdim": s.value_dim, "kv_rank": s.kv_rank, "scale": s.scale, "rot": rotation(s)}
            if s.window:
                m["mask"] = {"size": s.window}
        else:
            m = {"width": s.width}
        mlp = {"kind": "dense", "ff": s.ffn} if s.ffn else None
        if s.experts:
            mlp = {"kind": "moe", "expert": {"ff": s.expert_ffn}, "router": {"experts": s.experts, "top": s.experts_used}}
            if s.shared_ffn:
                mlp["shared"] = {"ff": s.shared_ffn}
            if c.arch == "zegelix":
                mlp["expert"]["limit"] = s.act_limit
                if s.shared_ffn:
                    mlp["shared"]["limit"] = s.shared_limit
        layers.append({"type": {"rotary_attention": "attention", "pooled_attention": "attention"}.get(s.mixer, s.mixer), "mixer": m, "mlp": mlp})
    arch = {v: k for k, v in LAYER_LIST_ARCHS.items()}[c.arch]
    norm = {"eps": c.rms_eps, "groups": c.norm_groups} if c.arch == "tikarax" else {"eps": c.rms_eps}
    out = {"architecture": arch, "layers": layers, "norm": norm, "vocab": c.vocab, "width": c.hidden}
    if c.arch in ("beputar", "zegelix"):
        out["embedding"] = {"scale": c.embedding_scale}
    if c.arch == "zegelix":
        out["logit_scale"] = c.logit_scale
    if c.loop_times:
        out["loop"] = {"start": c.loop_start, "stop": c.loop_stop, "times": c.loop_times}
    return out


def config_to_kv(c: ModelConfig) -> dict:
    """Inverse of :func:`read_config` for the synthetic-checkpoint generator."""
    a = c.arch
    kv = {
        "general.architecture": a, "general.name": c.name or f"synthetic-{a}",
        f"{a}.block_count": c.n_layers, f"{a}.embedding_length": c.hidden, f"{a}.attention.head_count": c.n_heads,
        f"{a}.attention.head_count_kv": c.n_kv_heads, f"{a}.feed_forward_length": c.ffn, f"{a}.attention.key_length": c.head_dim,
        f"{a}.attention.value_length": c.head_dim, f"{a}.rope.dimension_count": c.n_rot or c.head_dim, f"{a}.context_length": c.ctx_train,
        f"{a}.rope.freq_base": float(c.rope_theta), f"{a}.attention.layer_norm_rms_epsilon": float(c.rms_eps),
    }
    if c.sliding_window:
        kv[f"{a}.attention.sliding_window"] = c.sliding_window
    if c.rope_scaling_type != "none":
        kv[f"{a}.rope.scaling.type"] = c.rope_scaling_type
        kv[f"{a}.rope.scaling.factor"] = float(c.rope_scaling_factor)
        kv[f"{a}.rope.scaling.original_context_length"] = c.rope_orig_ctx
    if c.n_experts:
        kv[f"{a}.expert_count"] = c.n_experts
        kv[f"{a}.expert_used_count"] = c.n_experts_used
        kv[f"{a}.expert_feed_forward_length"] = c.expert_ffn
        if c.shared_expert_ffn:
            kv[f"{a}.expert_shared_feed_forward_length"] = c.shared_expert_ffn
    if c.is_hybrid:
        kv[f"{a}.full_attention_interval"] = c.full_attn_interval
        kv[f"{a}.ssm.inner_size"] = c.ssm_inner
        kv[f"{a}.ssm.state_size"] = c.ssm_state
        kv[f"{a}.ssm.group_count"] = c.ssm_n_k_heads
        kv[f"{a}.ssm.time_step_rank"] = c.ssm_n_v_heads
        kv[f"{a}.ssm.conv_kernel"] = c.ssm_conv_kernel
        if c.nextn_predict_layers:
            kv[f"{a}.nextn_predict_layers"] = c.nextn_predict_layers
    if a == "gemma4":
        kv[f"{a}.attention.head_count_kv"] = [int(v) for v in c.layer_n_kv]
        kv[f"{a}.attention.sliding_window_pattern"] = [bool(v) for v in c.layer_swa]
        kv[f"{a}.attention.key_length_swa"] = c.head_dim_swa
        kv[f"{a}.attention.value_length_swa"] = c.head_dim_swa
        kv[f"{a}.rope.dimension_count_swa"] = c.n_rot_swa or c.head_dim_swa
        kv[f"{a}.rope.freq_base_swa"] = float(c.rope_theta_swa)
        kv[f"{a}.final_logit_softcapping"] = float(c.final_logit_softcap)
    if a == "granite":
        kv[f"{a}.embedding_scale"] = float(c.embedding_scale)
        kv[f"{a}.residual_scale"] = float(c.residual_scale)
        kv[f"{a}.attention.scale"] = float(c.attention_scale)
        kv[f"{a}.logit_scale"] = float(1.0 / c.logit_scale) if c.logit_scale else 1.0
    return kv


def _tikarax_preset(hidden, n_layers, heads, kv_heads, dim, vdim, ffn, width, vocab, attn_every=4, groups=2, every=8192) -> ModelConfig:
    """Every ``attn_every``-th layer attention, the others minGRU."""
    c = ModelConfig(arch="tikarax", hidden=hidden, vocab=vocab, rms_eps=1e-6, norm_groups=groups)
    for l in range(n_layers):
        if (l + 1) % attn_every == 0:
            c.layer_specs.append(LayerSpec("attention", ffn=ffn, heads=heads, kv_heads=kv_heads, key_dim=dim, value_dim=vdim, scale=dim ** -0.5,
                                           q_temp_coef=0.1, q_temp_every=every))
        else:
            c.layer_specs.append(LayerSpec("mingru", ffn=ffn, width=width))
    return _finish_layer_list(c)


def _pubodra_preset(hidden, n_layers, heads, dim, rot_dim, vdim, kv_rank, window, ffn, vocab, experts=0, used=0, expert_ffn=0, moe_every=2, loop=None,
                    theta=1e5, yarn=(8.0, 4096.0, 32.0, 1.0)) -> ModelConfig:
    """Every ``moe_every``-th layer has experts (when there are any), the others a dense feed-forward."""
    c = ModelConfig(arch="pubodra", hidden=hidden, vocab=vocab, rms_eps=1e-6, tie_embeddings=True)
    for l in range(n_layers):
        s = LayerSpec("latent_attention", heads=heads, key_dim=dim, rot_dim=rot_dim, value_dim=vdim, kv_rank=kv_rank, window=window,
                      scale=(dim + rot_dim) ** -0.5, rope_theta=theta, yarn=yarn)
        if experts and (l + 1) % moe_every == 0:
            s.experts, s.experts_used, s.expert_ffn = experts, used, expert_ffn
        else:
            s.ffn = ffn
        c.layer_specs.append(s)
    if loop is not None:
        c.loop_start, c.loop_stop, c.loop_times = loop
    return _finish_layer_list(c)


def _beputar_preset(hidden, n_layers, heads, kv_heads, dim, window, keep_first, lin_heads, lin_dim, lin_vdim, wkv_heads, wkv_dim, decay_rank, ffn, vocab, experts=0,
                    used=0, expert_ffn=0, shared=0, order=("parallel", "rotary_attention", "wkv"), theta=5e5, yarn=(4.0, 4096.0, 32.0, 1.0)) -> ModelConfig:
    """The mixers of ``order`` in turn; the first layer has a dense feed-forward, the others experts (when there are any)."""
    c = ModelConfig(arch="beputar", hidden=hidden, vocab=vocab, rms_eps=1e-6, tie_embeddings=True, embedding_scale=16.0)
    for l in range(n_layers):
        s = LayerSpec(order[l % len(order)])
        if s.mixer == "wkv":
            s.lin_heads, s.lin_key_dim, s.lin_value_dim, s.decay_rank = wkv_heads, wkv_dim, wkv_dim, decay_rank
        else:
            s.heads, s.kv_heads, s.key_dim, s.value_dim, s.window, s.scale = heads, kv_heads, dim, dim, window, dim ** -0.5
            s.rot_dim, s.rope_theta = (dim // 4 * 2, theta) if s.mixer == "parallel" else (dim, 2e4)
            s.yarn = None if s.mixer == "parallel" else yarn
        if s.mixer == "parallel":
            s.keep_first, s.lin_heads, s.lin_key_dim, s.lin_value_dim = keep_first, lin_heads, lin_dim, lin_vdim
            s.lin_decay = tuple(math.exp(-2.0 ** (-8.0 * (h + 1) / lin_heads)) for h in range(lin_heads))
        if experts and l:
            s.experts, s.experts_used, s.expert_ffn, s.shared_ffn = experts, used, expert_ffn, shared
        else:
            s.ffn = ffn
        c.layer_specs.append(s)
    return _finish_layer_list(c)


def _zegelix_preset(hidden, n_layers, heads, kv_heads, dim, vdim, rot_dim, window, pool, softcap, width, blocks, conv, experts, used, expert_ffn, shared, vocab,
                    attn_every=3, limit=7.0, shared_limit=7.0, loop=None, theta=5e5, embedding_scale=0.0, logit_scale=1.0) -> ModelConfig:
    """Every ``attn_every``-th layer attention, the others RG-LRU; experts in every layer."""
    c = ModelConfig(arch="zegelix", hidden=hidden, vocab=vocab, rms_eps=1e-5, tie_embeddings=True, embedding_scale=embedding_scale or math.sqrt(hidden),
                    logit_scale=logit_scale)
    for l in range(n_layers):
        if (l + 1) % attn_every == 0:
            s = LayerSpec("pooled_attention", heads=heads, kv_heads=kv_heads, key_dim=dim, value_dim=vdim, rot_dim=rot_dim, scale=dim ** -0.5, window=window,
                          pool=pool, softcap=softcap, rope_theta=theta)
        else:
            s = LayerSpec("rglru", width=width, gate_blocks=blocks, conv_taps=conv)
        s.experts, s.experts_used, s.expert_ffn, s.shared_ffn, s.act_limit, s.shared_limit = experts, used, expert_ffn, shared, limit, shared_limit
        c.layer_specs.append(s)
    if loop is not None:
        c.loop_start, c.loop_stop, c.loop_times = loop
    return _finish_layer_list(c)


# ---- named architectures used by the benches and tests (random-init; see formats/synth.py)
def preset(name: str) -> ModelConfig:
    p = {
        "tiny-llama": ModelConfig(arch="llama", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=688, vocab=4096,
                                  rms_eps=1e-5, rope_theta=10000.0, n_rot=64, ctx_train=2048),
        "llama-3-8b": ModelConfig(arch="llama", n_layers=32, hidden=4096, n_heads=32, n_kv_heads=8, head_dim=128, ffn=14336,
                                  vocab=128256, rms_eps=1e-5, rope_theta=500000.0, n_rot=128, ctx_train=8192),
        "gpt-oss-20b": ModelConfig(arch="gpt-oss", n_layers=24, hidden=2880, n_heads=64, n_kv_heads=8, head_dim=64, ffn=2880,
                                   vocab=201088, rms_eps=1e-5, rope_theta=150000.0, n_rot=64, ctx_train=131072, sliding_window=128,
                                   n_experts=32, n_experts_used=4, expert_ffn=2880, rope_scaling_type="yarn", rope_scaling_factor=32.0,
                                   rope_orig_ctx=4096),
        "gpt-oss-120b": ModelConfig(arch="gpt-oss", n_layers=36, hidden=2880, n_heads=64, n_kv_heads=8, head_dim=64, ffn=2880,
                                    vocab=201088, rms_eps=1e-5, rope_theta=150000.0, n_rot=64, ctx_train=131072, sliding_window=128,
                                    n_experts=128, n_experts_used=4, expert_ffn=2880, rope_scaling_type="yarn",
                                    rope_scaling_factor=32.0, rope_orig_ctx=4096),
        "tiny-gpt-oss": ModelConfig(arch="gpt-oss", n_layers=4, hidden=256, n_heads=8, n_kv_heads=2, head_dim=64, ffn=256, vocab=2048,
                                    rms_eps=1e-5, rope_theta=150000.0, n_rot=64, ctx_train=4096, sliding_window=128, n_experts=8,
                                    n_experts_used=2, expert_ffn=256),
        "qwen3-moe-30b": ModelConfig(arch="qwen3moe", n_layers=48, hidden=2048, n_heads=32, n_kv_heads=4, head_dim=128, ffn=6144,
                                     vocab=151936, rms_eps=1e-6, rope_theta=1e6, n_rot=128, ctx_train=40960, n_experts=128,
                                     n_experts_used=8, expert_ffn=768),
        "tiny-qwen3moe": ModelConfig(arch="qwen3moe", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                     rms_eps=1e-6, rope_theta=1e6, n_rot=64, ctx_train=4096, n_experts=8, n_experts_used=2, expert_ffn=256),
        "qwen3-next-80b": ModelConfig(arch="qwen3next", n_layers=48, hidden=2048, n_heads=16, n_kv_heads=2, head_dim=256, ffn=5120,
                                      vocab=151936, rms_eps=1e-6, rope_theta=1e7, n_rot=64, ctx_train=262144, n_experts=512,
                                      n_experts_used=10, expert_ffn=512, shared_expert_ffn=512, full_attn_interval=4, ssm_inner=4096,
                                      ssm_state=128, ssm_n_k_heads=16, ssm_n_v_heads=32, ssm_conv_kernel=4, nextn_predict_layers=1),
        "tiny-qwen3next": ModelConfig(arch="qwen3next", n_layers=4, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                      rms_eps=1e-6, rope_theta=1e7, n_rot=32, ctx_train=4096, n_experts=8, n_experts_used=2,
                                      expert_ffn=256, shared_expert_ffn=256, full_attn_interval=4, ssm_inner=512, ssm_state=128,
                                      ssm_n_k_heads=2, ssm_n_v_heads=4, ssm_conv_kernel=4, nextn_predict_layers=1),
        "tiny-qwen35": ModelConfig(arch="qwen35", n_layers=4, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                   rms_eps=1e-6, rope_theta=1e7, n_rot=32, ctx_train=4096, full_attn_interval=4, ssm_inner=512,
                                   ssm_state=128, ssm_n_k_heads=2, ssm_n_v_heads=4, ssm_conv_kernel=4, nextn_predict_layers=1),
        # "crown": Qwen3.6-35B-A3B (qwen36.cpp: 40 layers, full attention every 4th, 256 experts top-8 + shared expert, MTP block)
        "qwen3.6-35b-a3b": ModelConfig(arch="qwen35moe", n_layers=40, hidden=2048, n_heads=16, n_kv_heads=2, head_dim=256, ffn=5120,
                                       vocab=248320, rms_eps=1e-6, rope_theta=1e7, n_rot=64, ctx_train=262144, n_experts=256,
                                       n_experts_used=8, expert_ffn=512, shared_expert_ffn=512, full_attn_interval=4, ssm_inner=4096,
                                       ssm_state=128, ssm_n_k_heads=16, ssm_n_v_heads=32, ssm_conv_kernel=4, nextn_predict_layers=1),
        "tiny-qwen35moe": ModelConfig(arch="qwen35moe", n_layers=4, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                      rms_eps=1e-6, rope_theta=1e7, n_rot=32, ctx_train=4096, n_experts=8, n_experts_used=2,
                                      expert_ffn=256, shared_expert_ffn=256, full_attn_interval=4, ssm_inner=512, ssm_state=128,
                                      ssm_n_k_heads=2, ssm_n_v_heads=4, ssm_conv_kernel=4, nextn_predict_layers=1),
        "qwen3.6-27b": ModelConfig(arch="qwen35", n_layers=64, hidden=5120, n_heads=24, n_kv_heads=4, head_dim=256, ffn=17408, vocab=248320,
                                   rms_eps=1e-6, rope_theta=1e7, n_rot=64, ctx_train=262144, full_attn_interval=4, ssm_inner=6144,
                                   ssm_state=128, ssm_n_k_heads=16, ssm_n_v_heads=48, ssm_conv_kernel=4, nextn_predict_layers=1),
        # Gemma-4 shape in miniature: sliding layers with more, narrower KV heads and one global layer with wide heads; MoE dual path
        "tiny-gemma4": ModelConfig(arch="gemma4", n_layers=3, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=2048,
                                   rms_eps=1e-6, rope_theta=1e6, n_rot=128, ctx_train=4096, sliding_window=128, head_dim_swa=64, n_rot_swa=64,
                                   rope_theta_swa=10000.0, layer_swa=[True, True, False], layer_n_kv=[2, 2, 1], n_experts=8, n_experts_used=2,
                                   expert_ffn=128, final_logit_softcap=30.0, embedding_scale=16.0, attention_scale=1.0, tie_embeddings=True),
        "tiny-gemma4-dense": ModelConfig(arch="gemma4", n_layers=3, hidden=256, n_heads=4, n_kv_heads=2, head_dim=128, ffn=512, vocab=2048,
                                         rms_eps=1e-6, rope_theta=1e6, n_rot=128, ctx_train=4096, sliding_window=128, head_dim_swa=64,
                                         n_rot_swa=64, rope_theta_swa=10000.0, layer_swa=[True, True, False], layer_n_kv=[2, 2, 1],
                                         final_logit_softcap=30.0, embedding_scale=16.0, attention_scale=1.0, tie_embeddings=True),
        "tiny-tikarax": _tikarax_preset(160, 4, 6, 2, 40, 56, 224, 288, 384, attn_every=2, groups=5, every=48),
        # layers of common model sizes: 1 B class and 8 B class (un-gated feed-forward with the parameters of a gated one of 2/3 its width)
        "tikarax-1b": _tikarax_preset(2048, 16, 32, 8, 64, 64, 12288, 4096, 128256),
        "tikarax-8b": _tikarax_preset(4096, 32, 32, 8, 128, 128, 21504, 6144, 128256),
        "tiny-pubodra": _pubodra_preset(160, 3, 5, 24, 8, 40, 48, 70, 224, 384, experts=6, used=2, expert_ffn=96, loop=(1, 3, 2), yarn=(4.0, 64.0, 32.0, 1.0)),
        # layers of common model sizes: 1 B class and 8 B class, the latter with 64 small experts in every other layer
        "pubodra-1b": _pubodra_preset(2048, 16, 16, 128, 64, 128, 512, 1024, 12288, 128256),
        "pubodra-8b": _pubodra_preset(4096, 32, 32, 128, 64, 128, 512, 4096, 21504, 128256, experts=64, used=6, expert_ffn=1536),
        "tiny-beputar": _beputar_preset(160, 4, 6, 2, 40, 50, 3, 5, 24, 40, 3, 40, 24, 224, 384, experts=6, used=2, expert_ffn=96, shared=64,
                                        yarn=(4.0, 64.0, 32.0, 1.0)),
        # layers of common model sizes: 1 B class and 8 B class
        "beputar-1b": _beputar_preset(2048, 15, 32, 8, 64, 1024, 16, 16, 128, 128, 32, 64, 64, 8192, 128256, experts=64, used=6, expert_ffn=1024, shared=2048),
        "beputar-8b": _beputar_preset(4096, 30, 32, 8, 128, 4096, 16, 32, 128, 128, 64, 64, 64, 16384, 128256, experts=64, used=6, expert_ffn=1536, shared=3072),
        "tiny-zegelix": _zegelix_preset(160, 3, 6, 2, 40, 56, 24, 50, 5, 30.0, 192, 3, 4, 6, 2, 96, 64, 384, attn_every=2, limit=1.5, shared_limit=2.5,
                                        loop=(1, 3, 2), theta=2e4, logit_scale=0.75),
        # layers of common model sizes: 1 B class and 8 B class
        "zegelix-1b": _zegelix_preset(2048, 15, 32, 8, 64, 64, 32, 1024, 16, 50.0, 2560, 10, 4, 64, 6, 1024, 2048, 128256),
        "zegelix-8b": _zegelix_preset(4096, 30, 32, 8, 128, 128, 64, 4096, 16, 50.0, 4096, 16, 4, 64, 6, 1536, 3072, 128256),
        "tiny-qwen2": ModelConfig(arch="qwen2", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                  rms_eps=1e-6, rope_theta=1e6, n_rot=64, ctx_train=4096),
        "tiny-phi3": ModelConfig(arch="phi3", n_layers=2, hidden=256, n_heads=4, n_kv_heads=4, head_dim=64, ffn=512, vocab=2048,
                                 rms_eps=1e-5, rope_theta=10000.0, n_rot=64, ctx_train=4096),
        "tiny-granite": ModelConfig(arch="granite", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                    rms_eps=1e-5, rope_theta=10000.0, n_rot=64, ctx_train=4096, embedding_scale=12.0, residual_scale=0.22,
                                    attention_scale=0.0078125, logit_scale=0.125),
        "tiny-qwen3": ModelConfig(arch="qwen3", n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=512, vocab=2048,
                                  rms_eps=1e-6, rope_theta=1e6, n_rot=64, ctx_train=4096),
    }
    if name not in p:
        raise KeyError(f"unknown preset {name}; have {sorted(p)}")
    c = p[name]
    c.name = name
    return c
