"""Throughput of a layer-list design beside the framework's closest models at equal size, and its kernels beside the like kernels.

    python bench.py --design tikarax|pubodra|beputar|zegelix [--design-part models|kernels|all]

Models (random-init bf16 weights, random tokens): prefill of one 4096-token prompt and decode at a 2048-token context for 1, 8 and 32
sequences, through ``LLMEngine`` (CUDA graphs as in serving), for
  tikarax:  the design as its preset orders it (one attention layer in four, minGRU otherwise), with attention in every layer; a llama of the same
            width, heads and parameters per layer (gated feed-forward of 2/3 the width); a DeltaNet hybrid (qwen35) of the same width
  pubodra:  the design with dense feed-forwards, with experts in every other layer, and with experts in every layer; a llama of the same width,
            heads, sliding window and parameters per layer; a qwen3moe with the same experts (gated, 2/3 the width) in every layer
  beputar:  the design (parallel, attention and wkv layers in turn) with dense feed-forwards, and with experts in every layer but the first; the DeltaNet
            hybrids of the same width, heads and parameters per feed-forward (qwen35: gated, 2/3 the width; qwen35moe: the same experts and shared expert)
  zegelix:  the design (one attention layer in three, RG-LRU otherwise, experts and a shared one in every layer), and with its middle third run twice; the
            DeltaNet hybrid of the same width, heads, experts and shared expert (qwen35moe); Beputar with the same experts
Weights are larger than L2 (126 MB), so every pass streams them.

Kernels: device time inside a CUDA graph over buffers that together exceed L2, as a fraction of the roofline (bytes over the measured copy
rate or FLOPs over the measured bf16 rate, whichever is longer), each beside the kernel that does the like work in the closest models.
"""
from __future__ import annotations

import gc
import json
import sys
import time

import torch

from ..formats.model_config import ModelConfig, _beputar_preset, _pubodra_preset, _tikarax_preset, _zegelix_preset

LAYERS = 8
SIZES = {"tikarax": {  # hidden, heads, kv_heads, head width, un-gated feed-forward, minGRU width
    "1b-layers": dict(hidden=2048, heads=32, kv_heads=8, dim=64, ffn=12288, width=4096),
    "8b-layers": dict(hidden=4096, heads=32, kv_heads=8, dim=128, ffn=21504, width=6144),
}, "pubodra": {       # hidden, heads, unrotated / rotated / value widths, latent, window, un-gated feed-forward; experts, per token, their width
    "1b-layers": dict(hidden=2048, heads=16, dim=128, rot=64, vdim=128, rank=512, window=1024, ffn=12288, experts=64, used=6, eff=1536),
    "8b-layers": dict(hidden=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, window=4096, ffn=21504, experts=64, used=6, eff=2304),
}, "beputar": {       # hidden, heads, kv_heads, head width, window, kept first; lightning heads of 128, wkv heads of 64; un-gated feed-forward; experts ...
    "1b-layers": dict(layers=9, hidden=2048, heads=32, kv_heads=8, dim=64, window=1024, keep=16, lin=16, wkv=32, ffn=12288, experts=64, used=6, eff=1024, shared=2048),
    "8b-layers": dict(layers=9, hidden=4096, heads=32, kv_heads=8, dim=128, window=4096, keep=16, lin=32, wkv=64, ffn=21504, experts=64, used=6, eff=1536, shared=3072),
}, "zegelix": {       # hidden, heads, kv_heads, head width, rotated, window, tokens per pooled block; RG-LRU width, blocks, taps; experts, per token, widths
    "1b-layers": dict(layers=9, hidden=2048, heads=32, kv_heads=8, dim=64, rot=32, window=1024, pool=16, width=2560, blocks=10, conv=4, experts=64, used=6, eff=1024,
                      shared=2048),
    "8b-layers": dict(layers=9, hidden=4096, heads=32, kv_heads=8, dim=128, rot=64, window=2048, pool=16, width=4096, blocks=16, conv=4, experts=64, used=6, eff=1536,
                      shared=3072),
}}
VOCAB = 32768
PREFILL, CONTEXT, DECODE = 4096, 2048, 64


def _tikarax_configs(s: dict) -> dict:
    tk = lambda every: _tikarax_preset(s["hidden"], LAYERS, s["heads"], s["kv_heads"], s["dim"], s["dim"], s["ffn"], s["width"], VOCAB, attn_every=every)
    common = dict(n_layers=LAYERS, hidden=s["hidden"], n_heads=s["heads"], n_kv_heads=s["kv_heads"], ffn=s["ffn"] * 2 // 3, vocab=VOCAB, ctx_train=16384)
    return {"tikarax": tk(4), "tikarax, attention only": tk(1),
            "llama": ModelConfig(arch="llama", head_dim=s["dim"], n_rot=s["dim"], **common),
            "qwen35 hybrid": ModelConfig(arch="qwen35", head_dim=s["dim"], n_rot=s["dim"] // 2, full_attn_interval=4, ssm_inner=32 * 128, ssm_state=128,
                                         ssm_n_k_heads=16, ssm_n_v_heads=32, ssm_conv_kernel=4, **common)}


def _pubodra_configs(s: dict) -> dict:
    pb = lambda moe_every: _pubodra_preset(s["hidden"], LAYERS, s["heads"], s["dim"], s["rot"], s["vdim"], s["rank"], s["window"], s["ffn"], VOCAB,
                                           *((s["experts"], s["used"], s["eff"], moe_every) if moe_every else ()))
    common = dict(n_layers=LAYERS, hidden=s["hidden"], n_heads=s["heads"], n_kv_heads=s["heads"] // 4, head_dim=128, n_rot=128, vocab=VOCAB, ctx_train=16384,
                  sliding_window=s["window"])
    return {"pubodra, dense": pb(0), "pubodra, experts in every other layer": pb(2), "pubodra, experts": pb(1),
            "llama": ModelConfig(arch="llama", ffn=s["ffn"] * 2 // 3, **common),
            "qwen3moe": ModelConfig(arch="qwen3moe", ffn=s["ffn"] * 2 // 3, n_experts=s["experts"], n_experts_used=s["used"], expert_ffn=s["eff"] * 2 // 3, **common)}


def _beputar_configs(s: dict) -> dict:
    bp = lambda *moe: _beputar_preset(s["hidden"], s["layers"], s["heads"], s["kv_heads"], s["dim"], s["window"], s["keep"], s["lin"], 128, 128, s["wkv"], 64, 64, s["ffn"],
                                      VOCAB, *moe)
    common = dict(n_layers=s["layers"], hidden=s["hidden"], n_heads=s["heads"], n_kv_heads=s["kv_heads"], ffn=s["ffn"] * 2 // 3, vocab=VOCAB, ctx_train=16384,
                  head_dim=s["dim"], n_rot=s["dim"] // 2, full_attn_interval=3, ssm_inner=s["lin"] * 128, ssm_state=128, ssm_n_k_heads=s["lin"] // 2,
                  ssm_n_v_heads=s["lin"], ssm_conv_kernel=4)
    return {"beputar, dense": bp(), "qwen35 hybrid": ModelConfig(arch="qwen35", **common),
            "beputar, experts": bp(s["experts"], s["used"], s["eff"], s["shared"]),
            "qwen35moe hybrid": ModelConfig(arch="qwen35moe", n_experts=s["experts"], n_experts_used=s["used"], expert_ffn=s["eff"], shared_expert_ffn=s["shared"], **common)}


def _zegelix_configs(s: dict) -> dict:
    zx = lambda loop: _zegelix_preset(s["hidden"], s["layers"], s["heads"], s["kv_heads"], s["dim"], s["dim"], s["rot"], s["window"], s["pool"], 50.0, s["width"],
                                      s["blocks"], s["conv"], s["experts"], s["used"], s["eff"], s["shared"], VOCAB, loop=loop)
    moe = dict(n_experts=s["experts"], n_experts_used=s["used"], expert_ffn=s["eff"], shared_expert_ffn=s["shared"])
    lin = s["hidden"] // 128
    third = s["layers"] // 3
    return {"zegelix": zx(None), "zegelix, middle third twice": zx((third, 2 * third, 2)),
            "qwen35moe hybrid": ModelConfig(arch="qwen35moe", n_layers=s["layers"], hidden=s["hidden"], n_heads=s["heads"], n_kv_heads=s["kv_heads"], ffn=s["eff"],
                                            vocab=VOCAB, ctx_train=16384, head_dim=s["dim"], n_rot=s["rot"], full_attn_interval=3, ssm_inner=lin * 128, ssm_state=128,
                                            ssm_n_k_heads=lin // 2, ssm_n_v_heads=lin, ssm_conv_kernel=4, **moe),
            "beputar, experts": _beputar_preset(s["hidden"], s["layers"], s["heads"], s["kv_heads"], s["dim"], s["window"], 16, lin, 128, 128, s["hidden"] // 64, 64, 64,
                                                6 * s["eff"], VOCAB, s["experts"], s["used"], s["eff"], s["shared"])}


def _timed(fn) -> float:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1)


def bench_models(design, dev, emit) -> None:
    from ..models import build_model
    from ..ops import cuda as K
    from ..runtime.engine import EngineOptions, LLMEngine, SamplingParams
    for size, s in SIZES[design].items():
        for name, cfg in {"tikarax": _tikarax_configs, "pubodra": _pubodra_configs, "beputar": _beputar_configs, "zegelix": _zegelix_configs}[design](s).items():
            model = build_model(cfg, dev, quant="bf16", max_ctx=PREFILL + 256)
            row = {"size": size, "model": name, "layers": cfg.n_layers, "weight_gb": round(model.weight_bytes() / 1e9, 2)}
            g = torch.Generator().manual_seed(0)
            prompt = lambda n: torch.randint(0, VOCAB, (n,), generator=g).tolist()
            eng = LLMEngine(model, EngineOptions(max_ctx=PREFILL + 256, max_batch_tokens=PREFILL, max_seqs=1, enable_prefix_cache=False))

            def prefill():
                eng.add_request(prompt(PREFILL), SamplingParams(max_tokens=1))
                eng.step()
            for _ in range(3):
                prefill()
            ms = sorted(_timed(prefill) for _ in range(5))[2]
            row["prefill_tok_s"] = round(PREFILL / ms * 1e3)
            row["prefill_ms"] = round(ms, 3)
            del eng
            for B in (1, 8, 32):
                eng = LLMEngine(model, EngineOptions(max_ctx=CONTEXT + 256, max_batch_tokens=CONTEXT, max_seqs=B, enable_prefix_cache=False))
                for _ in range(B):
                    eng.add_request(prompt(CONTEXT), SamplingParams(max_tokens=DECODE + 32, ignore_eos=True))
                while any(q.n_computed < len(q.prompt) for q in eng.sched.running) or eng.sched.waiting:
                    eng.step()
                for _ in range(4):
                    eng.step()
                n0, n = eng.stats["decode_tokens"], 0

                def decode():
                    for _ in range(DECODE // 2):
                        eng.step()
                ms = _timed(decode)
                n = eng.stats["decode_tokens"] - n0
                row[f"decode_b{B}_tok_s"] = round(n / ms * 1e3)
                row[f"decode_b{B}_ms"] = round(ms / (DECODE // 2), 3)
                del eng
            K.check_status()
            emit(row)
            del model
            gc.collect()
            torch.cuda.empty_cache()


def _per_call(fns: list, reps: int = 40) -> float:
    """Microseconds per call of the functions (same work on different buffers), cycled inside one CUDA graph."""
    n = max(reps, len(fns))
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for f in fns:
            f()
    torch.cuda.current_stream().wait_stream(side)
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(n):
            fns[i % len(fns)]()
    for _ in range(3):
        g.replay()
    return sorted(_timed(g.replay) for _ in range(7))[3] * 1e3 / n


class _Rows:
    """Helpers of a kernel table: buffers, and one timed row per kernel."""

    def __init__(self, dev, emit):
        from .kernel_bench import peaks
        self.dev, self.emit, self.pk = dev, emit, peaks()

    def bf(self, *sh):
        return (torch.randn(*sh, device=self.dev) * 0.5).to(torch.bfloat16)

    def i32(self, v):
        return torch.tensor(v, dtype=torch.int32, device=self.dev)

    @staticmethod
    def bufs(nbytes):
        return max(2, int(3e8 // nbytes) + 1) if nbytes < 3e8 else 1

    def row(self, kernel, role, fns, bytes_=0.0, flops=0.0):
        us = _per_call(fns)
        pk = self.pk
        roof = max(bytes_ / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)
        self.emit({"kernel": kernel, "role": role, "us": round(us, 2), "gbs": round(bytes_ / us / 1e3) if bytes_ else None,
                   "tflops": round(flops / us / 1e6, 1) if flops else None, f"fraction_of_{pk['src']}_roofline": round(roof / us, 3)})


def bench_kernels_tikarax(dev, emit) -> None:
    from ..ops import cuda as K
    from ..ops import ref
    from ..ops.weights import QuantWeight, WFormat
    from ..utils.rope import query_temperature_table, rope_tables
    t = _Rows(dev, emit)
    bf, i32, bufs, row = t.bf, t.i32, t.bufs, t.row
    for size, s in SIZES["tikarax"].items():
        H, W, F, nq, nkv, d = s["hidden"], s["width"], s["ffn"], s["heads"], s["kv_heads"], s["dim"]
        for T in (1, 32, PREFILL):
            # ---- norms: both sides of a sublayer in one pass, against residual add + norm
            nb = bufs(T * H * 12) if T > 64 else 8
            xs, ds, w = [torch.randn(T, H, device=dev) for _ in range(nb)], [bf(T, H) for _ in range(nb)], torch.ones(H, device=dev)
            by = T * H * (4 + 4 + 2 + 2)
            row(f"group_norm (branch norm + add + norm) T={T} H={H}", "new", [lambda x=x, q=q: K.group_norm(x, w, 1e-6, 2, delta=q, delta_w=w) for x, q in zip(xs, ds)], by)
            row(f"rmsnorm (add + norm) T={T} H={H}", "like", [lambda x=x, q=q: K.rmsnorm(x, w, 1e-6, delta=q) for x, q in zip(xs, ds)], by)
            # ---- up projection with its activation
            ws = [QuantWeight(WFormat.BF16, F, H, 1, bf(1, F, H)) for _ in range(bufs(F * H * 2))]
            gs = [QuantWeight(WFormat.BF16, F // 3 * 4 // 32 * 32, H, 1, bf(1, F // 3 * 4 // 32 * 32, H)) for _ in range(bufs(F * H * 2))]
            h = bf(T, H)
            fl = 2.0 * T * F * H
            row(f"up + xIELU T={T} {F}x{H}", "new", [lambda m=m: K.linear(h, m, act=ref.ACT_XIELU, act_alpha=0.8, act_limit=1.2) for m in ws], F * H * 2 + T * (H + F) * 2, fl)
            row(f"plain projection T={T} {F}x{H}", "like", [lambda m=m: K.linear(h, m) for m in ws], F * H * 2 + T * (H + F) * 2, fl)
            N = gs[0].N
            row(f"gate|up + SwiGLU T={T} {N}x{H}", "like", [lambda m=m: K.linear(h, m, act=ref.ACT_SWIGLU) for m in gs], N * H * 2 + T * (H + N // 2) * 2, 2.0 * T * N * H)
            del ws, gs
        # ---- recurrence
        for B, n in ((1, PREFILL), (8, 512), (1, 1), (32, 1)):
            T = B * n
            nb = bufs(T * W * 8) if T > 64 else 8
            ys, st = [bf(T, 3 * W) for _ in range(nb)], torch.zeros(B, W, device=dev)
            zb, slots, cu, sl = torch.zeros(W, device=dev), i32(list(range(B))), i32([i * n for i in range(B + 1)]), i32([n + 64] * B)
            row(f"mingru_scan B={B} n={n} W={W}", "new",
                [lambda y=y: K.mingru_scan(y[:, :W], y[:, W:2 * W], y[:, 2 * W:], zb, zb, st, slots, cu, sl, n) for y in ys], T * W * 8 + B * W * 8)
            C = 8192
            xs, cw, cs = [bf(T, C) for _ in range(bufs(T * C * 4) if T > 64 else 8)], torch.randn(C, 4, device=dev), torch.zeros(B, 3, C, dtype=torch.bfloat16, device=dev)
            row(f"conv1d_silu B={B} n={n} C={C}", "like", [lambda x=x: K.conv1d_silu(x, cw, cs, slots, cu, n) for x in xs], T * C * 4 + B * 3 * C * 4)
            nv, nk = 32, 16
            ab, ai, S = bf(T, 2 * nv), i32(list(range(nv))), torch.zeros(B, nv, 128, 128, device=dev)
            kv, sa = (ai // 2).to(torch.int32), -torch.rand(nv, device=dev)
            row(f"deltanet_scan B={B} n={n} heads={nk}/{nv}", "like",
                [lambda x=x: K.deltanet_scan(x, nk, ab, ai, ai + nv, kv, sa, sa, S, slots, cu, nv) for x in xs], T * C * 2 + T * nv * 128 * 4 + 2 * S.numel() * 4)
        # ---- attention, epilogue
        temp = query_temperature_table(2 * PREFILL, 0.1, 512, device=dev)
        cos, sin = rope_tables(2 * PREFILL, d, 1e4, device=dev)
        for B, n, ctx in ((1, PREFILL, PREFILL), (1, 1, 8192), (1, 1, 2048), (32, 1, 2048)):
            T, nblk = B * n, (ctx + 127) // 128
            pages = B * nblk + 1
            nb = min(16, bufs(pages * nkv * 128 * d * 4)) if n == 1 else 2
            kc, vc = [bf(pages, nkv, 128, d) for _ in range(nb)], [bf(pages, nkv, 128, d) for _ in range(nb)]
            bt = torch.arange(1, pages, dtype=torch.int32, device=dev).reshape(B, nblk)
            sl, cu = i32([ctx] * B), i32([i * n for i in range(B + 1)])
            y, q = bf(T, (2 * nq + 2 * nkv) * d), bf(T, nq, d)
            keys = n * ctx - n * (n - 1) // 2
            by, fl = B * ctx * nkv * d * 4 + T * nq * d * 4, 4.0 * B * keys * nq * d
            row(f"attention + gate + temperature B={B} n={n} ctx={ctx} {nq}/{nkv}x{d}", "new",
                [lambda k=k, v=v: K.attention(y[:, :nq * d].view(T, nq, d), k, v, bt, sl, cu, n, scale=d ** -0.5, q_scale=temp, gate=y[:, -nq * d:]) for k, v in zip(kc, vc)],
                by + T * nq * d * 2, fl)
            row(f"attention B={B} n={n} ctx={ctx} {nq}/{nkv}x{d}", "like", [lambda k=k, v=v: K.attention(q, k, v, bt, sl, cu, n, scale=d ** -0.5) for k, v in zip(kc, vc)], by, fl)
            if d == 128 and ctx != 8192:      # widths that differ and fill no tile: 96-wide keys, 128-wide values
                k96 = [bf(pages, nkv, 128, 96) for _ in range(nb)]
                q96 = bf(T, nq, 96)
                row(f"attention + gate, 96-wide keys B={B} n={n} ctx={ctx}", "new",
                    [lambda k=k, v=v: K.attention(q96, k, v, bt, sl, cu, n, scale=0.1, q_scale=temp, gate=y[:, -nq * d:]) for k, v in zip(k96, vc)],
                    B * ctx * nkv * (96 + d) * 2 + T * nq * (96 + 2 * d) * 2, 2.0 * B * keys * nq * (96 + d))
                del k96
            slots = torch.arange(128, 128 + T, dtype=torch.int64, device=dev)
            pos = torch.arange(T, dtype=torch.int32, device=dev)
            if ctx != 8192:
                nb2 = bufs(T * nkv * d * 8) if T > 64 else 8
                yk = [bf(T, (2 * nq + 2 * nkv) * d) for _ in range(min(nb2, 8))]
                row(f"kv_store T={T}", "new", [lambda t=t: K.kv_store(t[:, nq * d:(nq + nkv) * d], t[:, (nq + nkv) * d:(nq + 2 * nkv) * d], slots, kc[0], vc[0]) for t in yk], T * nkv * d * 8)
                yp = [t[:, :(nq + 2 * nkv) * d].contiguous() for t in yk]
                row(f"qkv_post T={T}", "like", [lambda t=t: K.qkv_post(t, None, None, None, pos, cos, sin, slots, kc[0], vc[0], nq, nkv, d, d) for t in yp],
                    T * (nq * d * 4 + nkv * d * 8))
            del kc, vc
            torch.cuda.empty_cache()
    K.check_status()


def bench_kernels_pubodra(dev, emit) -> None:
    from ..ops import cuda as K
    from ..ops import ref
    from ..ops.weights import QuantWeight, WFormat
    from ..utils.rope import rope_tables
    t = _Rows(dev, emit)
    bf, i32, bufs, row = t.bf, t.i32, t.bufs, t.row
    mats = lambda n, k, e=1, least=1: [QuantWeight(WFormat.BF16, n, k, e, (torch.randn(e, n, k, device=dev) * k ** -0.5).to(torch.bfloat16))
                                       for _ in range(max(least, bufs(e * n * k * 2)))]
    for size, s in SIZES["pubodra"].items():
        H, F, nh, d, r, v, R, win = s["hidden"], s["ffn"], s["heads"], s["dim"], s["rot"], s["vdim"], s["rank"], s["window"]
        E, top, ef = s["experts"], s["used"], s["eff"]
        for T in (1, 32, PREFILL):
            # ---- norms
            nb = bufs(T * H * 12) if T > 64 else 8
            xs, ds, w = [torch.randn(T, H, device=dev) for _ in range(nb)], [bf(T, H) for _ in range(nb)], torch.ones(H, device=dev)
            by = T * H * (4 + 4 + 2 + 2)
            row(f"dyt_norm (add + tanh) T={T} H={H}", "new", [lambda x=x, q=q: K.dyt_norm(x, 0.7, w, w, delta=q) for x, q in zip(xs, ds)], by)
            row(f"rmsnorm (add + norm) T={T} H={H}", "like", [lambda x=x, q=q: K.rmsnorm(x, w, 1e-6, delta=q) for x, q in zip(xs, ds)], by)
            # ---- ... that form the experts' weighted sum
            ys, pos, cw = [bf(T * top, H) for _ in range(nb)], torch.randperm(T * top, device=dev).to(torch.int32), torch.rand(T, top, device=dev)
            by = T * H * (4 + 4 + 2 + 2 * top)
            comb = [K.CombineDelta(y, pos, cw) for y in ys]
            row(f"dyt_norm + combine of {top} T={T} H={H}", "new", [lambda x=x, q=q: K.dyt_norm(x, 0.7, w, w, delta=q) for x, q in zip(xs, comb)], by)
            row(f"rmsnorm_combine of {top} T={T} H={H}", "like", [lambda x=x, q=q: K.rmsnorm_combine(x, w, 1e-6, q) for x, q in zip(xs, comb)], by)
            del xs, ds, ys, comb
            # ---- up projections with their activations
            h = bf(T, H)
            ws = mats(F, H)
            row(f"up + GELU T={T} {F}x{H}", "new", [lambda m=m: K.linear(h, m, act=ref.ACT_GELU_TANH) for m in ws], F * H * 2 + T * (H + F) * 2, 2.0 * T * F * H)
            N = F // 3 * 4 // 32 * 32
            ws = mats(N, H)
            row(f"gate|up + SwiGLU T={T} {N}x{H}", "like", [lambda m=m: K.linear(h, m, act=ref.ACT_SWIGLU) for m in ws], N * H * 2 + T * (H + N // 2) * 2, 2.0 * T * N * H)
            del ws
            # ---- experts
            idx = torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(T)]).to(torch.int32)
            live = len(set(idx.reshape(-1).tolist()))
            gf = ef * 2 // 3
            for name, role, n_up, k_dn, act in (("relu^2", "new", ef, ef, ref.ACT_RELU2), ("SwiGLU", "like", 2 * gf, gf, ref.ACT_SWIGLU)):
                ups, dns = mats(n_up, H, E), mats(H, k_dn, E)
                if T <= 8:
                    se = idx.reshape(-1)
                    a = bf(T * top, k_dn)
                    row(f"expert up + {name} T={T} {E}x{n_up}x{H}", role, [lambda m=m: K.expert_gemv(h, m, se, x_div=top, act=act) for m in ups], live * n_up * H * 2)
                    row(f"expert down T={T} {E}x{H}x{k_dn}", role, [lambda m=m: K.expert_gemv(a, m, se) for m in dns], live * k_dn * H * 2)
                else:
                    pk = K.moe_pack(idx, E)
                    xp, a = K.moe_gather(h, pk), bf(pk.max_rows, k_dn)
                    row(f"expert up + {name} T={T} {E}x{n_up}x{H}", role, [lambda m=m: K.grouped_linear(xp, m, pk.tile_expert, pk.num_tiles, act=act) for m in ups],
                        live * n_up * H * 2 + T * top * (H + k_dn) * 2, 2.0 * T * top * n_up * H)
                    row(f"expert down T={T} {E}x{H}x{k_dn}", role, [lambda m=m: K.grouped_linear(a, m, pk.tile_expert, pk.num_tiles) for m in dns],
                        live * k_dn * H * 2 + T * top * (H + k_dn) * 2, 2.0 * T * top * k_dn * H)
                del ups, dns
            # ---- head epilogue
            cos, sin = rope_tables(2 * PREFILL, r, 1e4, device=dev)
            cosl, sinl = rope_tables(2 * PREFILL, 128, 1e4, device=dev)
            pages = T // 128 + 2
            slots, pos = torch.arange(128, 128 + T, dtype=torch.int64, device=dev), torch.arange(T, dtype=torch.int32, device=dev)
            cache = torch.zeros(pages, 1, 128, R + r, dtype=torch.bfloat16, device=dev)
            nw, cq, nkv = torch.ones(R, device=dev), nh * (d + r), nh // 4
            yk = [bf(T, cq + R + r + nh * v) for _ in range(bufs(T * cq * 2) if T > 64 else 8)][:8]
            row(f"latent_post T={T}", "new", [lambda y=y: K.latent_post(y[:, :cq].view(T, nh, d + r)[..., d:], y[:, cq:cq + R + r], nw, R, 1e-6, pos, cos, sin, slots,
                cache, y[:, :cq].view(T, nh, d + r)[..., d:]) for y in yk], T * (nh * r * 4 + (R + r) * 4))
            kc, vc = torch.zeros(pages, nkv, 128, 128, dtype=torch.bfloat16, device=dev), torch.zeros(pages, nkv, 128, 128, dtype=torch.bfloat16, device=dev)
            yk = [bf(T, (nh + 2 * nkv) * 128) for _ in range(8)]
            row(f"qkv_post T={T}", "like", [lambda y=y: K.qkv_post(y, None, None, None, pos, cosl, sinl, slots, kc, vc, nh, nkv, 128, 128) for y in yk],
                T * (nh * 128 * 4 + nkv * 128 * 8))
            del yk, kc, vc
        # ---- per-head products of the latent space, against a plain projection of the same weight
        for T in (1, 8, 32):
            y, o, g = bf(T, nh, d + r), bf(T, nh, R), bf(T, nh * v)
            qc = torch.empty(T, nh, R + r, dtype=torch.bfloat16, device=dev)
            ab, vu, pl = mats(R, d, nh), mats(v, R, nh), mats(nh * R // 4, 4 * d)
            row(f"queries into the latent space T={T} {nh}x{R}x{d}", "new", [lambda m=m: K.head_linear(y[..., :d], m, out=qc[..., :R]) for m in ab],
                nh * R * d * 2 + T * nh * (d + R) * 2, 2.0 * T * nh * R * d)
            row(f"latent outputs to values + gate T={T} {nh}x{v}x{R}", "new", [lambda m=m: K.head_linear(o, m, gate=g) for m in vu],
                nh * R * v * 2 + T * nh * (2 * v + R) * 2, 2.0 * T * nh * R * v)
            h = bf(T, 4 * d)
            row(f"plain projection T={T} {nh * R // 4}x{4 * d}", "like", [lambda m=m: K.linear(h, m) for m in pl], nh * R * d * 2 + T * (4 * d + nh * R // 4) * 2, 2.0 * T * nh * R * d)
            del ab, vu, pl
        # ---- attention: decoding
        nkv = nh // 4
        for B, ctx, w_ in ((1, 8192, 0), (1, 2048, 0), (8, 2048, win), (32, 2048, win), (32, 8192, 0)):
            nblk = (ctx + 127) // 128
            pages = B * nblk + 1
            keys = min(ctx, w_) if w_ else ctx
            caches = [bf(pages, 1, 128, R + r) for _ in range(min(16, bufs(B * keys * (R + r) * 2)))]
            bt = torch.arange(1, pages, dtype=torch.int32, device=dev).reshape(B, nblk)
            sl, cu = i32([ctx] * B), i32(list(range(B + 1)))
            q = bf(B, nh, R + r)
            row(f"latent attention B={B} ctx={ctx} window={w_} {nh}x({R}+{r})", "new",
                [lambda c=c: K.latent_attention(q, c, bt, sl, cu, 1, R, window=w_, scale=0.07) for c in caches],
                B * keys * (R + r) * 2 + B * nh * (2 * R + r) * 2, 2.0 * B * keys * nh * (2 * R + r))
            del caches
            kv = [(bf(pages, nkv, 128, 128), bf(pages, nkv, 128, 128)) for _ in range(min(16, bufs(B * keys * nkv * 512)))]
            q = bf(B, nh, 128)
            row(f"attention B={B} ctx={ctx} window={w_} {nh}/{nkv}x128", "like", [lambda k=k, x=x: K.attention(q, k, x, bt, sl, cu, 1, window=w_, scale=0.09) for k, x in kv],
                B * keys * nkv * 512 + B * nh * 512, 4.0 * B * keys * nh * 128)
            del kv
            torch.cuda.empty_cache()
        # ---- attention: prompts
        for n, ctx in ((PREFILL, PREFILL), (512, PREFILL)):
            nblk = ctx // 128
            bt, sl, cu = torch.arange(1, nblk + 1, dtype=torch.int32, device=dev).reshape(1, nblk), i32([ctx]), i32([0, n])
            first = max(0, ctx - n - win + 1)
            pairs = float(sum(min(p + 1, win) for p in range(ctx - n, ctx)))
            q, g, out = bf(n, nh, d + r), bf(n, nh * v), torch.empty(n, nh, v, dtype=torch.bfloat16, device=dev)
            caches, wk = [bf(nblk + 1, 1, 128, R + r) for _ in range(4)], mats(nh * (d + v), R)
            rows_ = ctx - first // 128 * 128
            fl_up, fl_at = 2.0 * rows_ * R * nh * (d + v), 2.0 * pairs * nh * (d + r + v)
            plan = K._latent_plan(None, bt, sl, cu, n, win, 128)
            kvb = torch.empty(plan[0].numel() * 128, nh * (d + v), dtype=torch.bfloat16, device=dev)
            row(f"keys and values of {rows_} rows {nh * (d + v)}x{R}", "new",
                [lambda m=m, c=c: K.gemm_paged(c, plan, m, kvb) for m, c in zip(wk, caches * 8)], rows_ * (R + nh * (d + v)) * 2 + R * nh * (d + v) * 2, fl_up)
            hp, pm = bf(rows_, R), mats(nh * (d + v), R)
            row(f"plain projection T={rows_} {nh * (d + v)}x{R}", "like", [lambda m=m: K.linear(hp, m) for m in pm], rows_ * (R + nh * (d + v)) * 2 + R * nh * (d + v) * 2, fl_up)
            row(f"expanded attention n={n} ctx={ctx} window={win} {nh}x({d}+{r}/{v}) + gate, without forming keys", "new",
                [lambda c=c: K.expanded_attention(q, kvb, plan, c, bt, sl, cu, n, d, v, R, win, 0.07, g, out) for c in caches],
                rows_ * nh * (d + v) * 2 + n * nh * (d + r + 2 * v) * 2, fl_at)
            kc, vc = bf(nblk + 1, nkv, 128, 128), bf(nblk + 1, nkv, 128, 128)
            q1 = bf(n, nh, 128)
            row(f"attention n={n} ctx={ctx} window={win} {nh}/{nkv}x128", "like", [lambda: K.attention(q1, kc, vc, bt, sl, cu, n, window=win, scale=0.09)],
                rows_ * nkv * 512 + n * nh * 512, 4.0 * pairs * nh * 128)
            del caches, wk, kvb, kc, vc, pm
            torch.cuda.empty_cache()
    K.check_status()


def bench_kernels_beputar(dev, emit) -> None:
    from ..ops import cuda as K
    from ..ops import ref
    from ..ops.weights import QuantWeight, WFormat
    from ..utils.rope import rope_tables
    t = _Rows(dev, emit)
    bf, i32, bufs, row = t.bf, t.i32, t.bufs, t.row
    mats = lambda n, k, e=1: [QuantWeight(WFormat.BF16, n, k, e, (torch.randn(e, n, k, device=dev) * k ** -0.5).to(torch.bfloat16)) for _ in range(bufs(e * n * k * 2))]
    f32 = lambda *sh: torch.randn(*sh, device=dev)
    for size, s in SIZES["beputar"].items():
        H, nq, nkv, d, win, keep, lin, wkv = s["hidden"], s["heads"], s["kv_heads"], s["dim"], s["window"], s["keep"], s["lin"], s["wkv"]
        E, top, ef = s["experts"], s["used"], s["eff"]
        for T in (1, 32, PREFILL):
            # ---- norms on a sublayer's output
            nb = bufs(T * H * 12) if T > 64 else 8
            xs, ds, w = [f32(T, H) for _ in range(nb)], [bf(T, H) for _ in range(nb)], torch.ones(H, device=dev)
            by = T * H * (4 + 4 + 2 + 2)
            row(f"sublayer_norm (branch norm + add) T={T} H={H}", "new", [lambda x=x, q=q: K.sublayer_norm(x, q, w, 1e-6) for x, q in zip(xs, ds)], by)
            row(f"sublayer_norm of two normed branches T={T} H={H}", "new",
                [lambda x=x, q=q, r=r: K.sublayer_norm(x, ref.BranchMean(q, w, r, w), w, 1e-6) for x, q, r in zip(xs, ds, ds[1:] + ds[:1])], by + T * H * 2)
            row(f"rmsnorm (add + norm) T={T} H={H}", "like", [lambda x=x, q=q: K.rmsnorm(x, w, 1e-6, delta=q) for x, q in zip(xs, ds)], by)
            ys, pos, cw = [bf(T * top, H) for _ in range(nb)], torch.randperm(T * top, device=dev).to(torch.int32), torch.rand(T, top, device=dev)
            by = T * H * (4 + 4 + 2 + 2 * top)
            row(f"sublayer_norm of {top} experts + shared T={T} H={H}", "new",
                [lambda x=x, y=y, q=q: K.sublayer_norm(x, ref.ExpertSum(y, pos, top, q), w, 1e-6) for x, y, q in zip(xs, ys, ds)], by + T * H * 2)
            row(f"rmsnorm_combine of {top} T={T} H={H}", "like", [lambda x=x, y=y: K.rmsnorm_combine(x, w, 1e-6, K.CombineDelta(y, pos, cw)) for x, y in zip(xs, ys)], by)
            del ds, ys
            # ---- expert rows
            h, idx = bf(T, H), torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(T)]).to(torch.int32)
            pk = K.moe_pack(idx, E)
            hs = [bf(T, H) for _ in range(nb)]
            row(f"moe_scale_rows T={T} x {top}", "new", [lambda x=x: K.moe_scale_rows(x, cw, pk) for x in hs], T * H * 2 * (1 + top))
            row(f"moe_gather T={T} x {top}", "like", [lambda x=x: K.moe_gather(x, pk) for x in hs], T * H * 2 * (1 + top))
            z = f32(T, E)
            row(f"moe_route, sigmoid T={T} {top} of {E}", "new", [lambda: K.moe_route(z, None, top, sigmoid=True)], T * (E + 2 * top) * 4)
            row(f"moe_route, softmax T={T} {top} of {E}", "like", [lambda: K.moe_route(z, None, top)], T * (E + 2 * top) * 4)
            # ---- projections: the four of a wkv layer over their own inputs
            N = wkv * 64
            st, x4 = mats(N, H, 4), bf(4, T, H)
            row(f"four projections of four inputs T={T} {N}x{H}", "new", [lambda m=m: K.stacked_linear(x4, m) for m in st], 4 * N * H * 2 + 4 * T * (H + N) * 2, 8.0 * T * N * H)
            del st
            pl = mats(4 * N, H)
            row(f"plain projection T={T} {4 * N}x{H}", "like", [lambda m=m: K.linear(h, m) for m in pl], 4 * N * H * 2 + T * (H + 4 * N) * 2, 8.0 * T * N * H)
            del pl
            # ---- head epilogue
            cos, sin = rope_tables(2 * PREFILL, d, 1e4, device=dev)
            cosh, sinh = rope_tables(2 * PREFILL, d // 2, 1e4, device=dev)
            pages, bs = T // 128 + 2, 128
            slots, pos1 = torch.arange(128, 128 + T, dtype=torch.int64, device=dev), torch.arange(T, dtype=torch.int32, device=dev)
            kc, vc = torch.zeros(pages, nkv, bs, d, dtype=torch.bfloat16, device=dev), torch.zeros(pages, nkv, bs, d, dtype=torch.bfloat16, device=dev)
            ys, nw = [bf(T, (nq + 2 * nkv) * d) for _ in range(min(8, bufs(T * nq * d * 4) if T > 64 else 8))], torch.ones(d, device=dev)
            q_, k_ = (lambda y: y[:, :nq * d].view(T, nq, d)), (lambda y: y[:, nq * d:(nq + nkv) * d].view(T, nkv, d))
            by = T * (nq * d * 4 + nkv * d * 6)
            row(f"qk_post, norm then half splits T={T}", "new",
                [lambda y=y: K.qk_post(q_(y), k_(y), pos1, cosh, sinh, slots, kc, vc, d, d // 2, q_norm=nw, k_norm=nw) for y in ys], by)
            row(f"qk_post, pairs then norm T={T}", "new",
                [lambda y=y: K.qk_post(q_(y), k_(y), pos1, cos, sin, slots, kc, vc, d, d, interleaved=True, norm_after=True) for y in ys], by)
            row(f"qkv_post, norm T={T}", "like", [lambda y=y: K.qkv_post(y, None, nw, nw, pos1, cos, sin, slots, kc, vc, nq, nkv, d, d) for y in ys], by + T * nkv * d * 2)
            del ys, kc, vc
        # ---- recurrences and what is around them
        for B, n in ((1, PREFILL), (8, 512), (1, 1), (32, 1)):
            T = B * n
            slots, cu, sl = i32(list(range(B))), i32([i * n for i in range(B + 1)]), i32([n + 64] * B)
            nb = bufs(T * H * 8) if T > 64 else 8
            xs, mu, sh = [f32(T, H) for _ in range(nb)], torch.rand(5, H, device=dev), torch.zeros(B, H, device=dev)
            row(f"token_shift B={B} n={n} 5 mixes of {H}", "new", [lambda x=x: K.token_shift(x, mu, sh, slots, cu, sl) for x in xs], T * H * 14 + B * H * 8)
            C = 2 * lin * 128
            xc, cwt, cst = [bf(T, C) for _ in range(nb)], f32(C, 4), torch.zeros(B, 3, C, dtype=torch.bfloat16, device=dev)
            row(f"conv1d_silu B={B} n={n} C={C}", "like", [lambda x=x: K.conv1d_silu(x, cwt, cst, slots, cu, n) for x in xc], T * C * 4 + B * 3 * C * 4)
            W = wkv * 64
            r4, z, u, S = [bf(4, T, W) for _ in range(nb)], -2.0 + f32(T, W), f32(wkv, 64), torch.zeros(B, wkv, 64, 64, device=dev)
            hd = lambda y: y.view(T, wkv, 64)
            row(f"decay_scan, wkv B={B} n={n} {wkv} heads of 64", "new",
                [lambda y=y: K.decay_scan(hd(y[0]), hd(y[1]), hd(y[2]), S, slots, cu, sl, n, z=z, u=u) for y in r4], T * W * (6 + 4 + 4) + 2 * S.numel() * 4)
            W2 = lin * 128
            y4, dec, S2 = [bf(T, 4 * W2) for _ in range(nb)], torch.linspace(0.5, 0.999, lin, device=dev), torch.zeros(B, lin, 128, 128, device=dev)
            cut = lambda y, i: y[:, i * W2:(i + 1) * W2].view(T, lin, 128)
            row(f"decay_scan, lightning B={B} n={n} {lin} heads of 128", "new",
                [lambda y=y: K.decay_scan(cut(y, 0), cut(y, 1), cut(y, 2), S2, slots, cu, sl, n, decay=dec, silu=True) for y in y4], T * W2 * (6 + 4) + 2 * S2.numel() * 4)
            nv, nk = lin, lin // 2
            ab, ai, S3 = bf(T, 2 * nv), i32(list(range(nv))), torch.zeros(B, nv, 128, 128, device=dev)
            kv, sa = (ai // 2).to(torch.int32), -torch.rand(nv, device=dev)
            row(f"deltanet_scan B={B} n={n} heads={nk}/{nv}", "like",
                [lambda x=x: K.deltanet_scan(x, nk, ab, ai, ai + nv, kv, sa, sa, S3, slots, cu, nv) for x in xc], T * C * 2 + T * nv * 128 * 4 + 2 * S3.numel() * 4)
            os_, g, w = [f32(T, W2) for _ in range(nb)], bf(T, W2), torch.ones(W2, device=dev)
            by = T * W2 * (4 + 2 + 2)
            row(f"gated_group_norm, one group T={T} W={W2}", "new", [lambda o=o: K.gated_group_norm(o, g, w, 1e-6) for o in os_], by)
            row(f"gated_group_norm, groups of 64 T={T} W={W2}", "new", [lambda o=o: K.gated_group_norm(o, g, w, 1e-6, groups=W2 // 64, silu=True) for o in os_], by)
            row(f"gated_rmsnorm_heads T={T} W={W2}", "like", [lambda o=o: K.gated_rmsnorm_heads(o, g, w[:128], 1e-6, 128) for o in os_], by)
            del xs, xc, r4, y4, os_
            torch.cuda.empty_cache()
        # ---- attention
        for B, n, ctx in ((1, PREFILL, PREFILL), (1, 512, PREFILL), (1, 1, 8192), (1, 1, 2048), (32, 1, 2048), (32, 1, 8192)):
            T, nblk = B * n, (ctx + 127) // 128
            pages, live = B * nblk + 1, min(ctx, win + n)
            nb = min(16, bufs(B * live * nkv * d * 4)) if n == 1 else 2
            kc, vc = [bf(pages, nkv, 128, d) for _ in range(nb)], [bf(pages, nkv, 128, d) for _ in range(nb)]
            bt = torch.arange(1, pages, dtype=torch.int32, device=dev).reshape(B, nblk)
            sl, cu = i32([ctx] * B), i32([i * n for i in range(B + 1)])
            q, g, sink = bf(T, nq, d), bf(T, 40), torch.zeros(nq, device=dev)
            seen = lambda kept: float(sum(min(p + 1, win + kept) for p in range(ctx - n, ctx)))
            by, fl = B * live * nkv * d * 4 + T * nq * d * 4, 4.0 * B * nq * d
            kw = dict(window=win, scale=d ** -0.5)
            row(f"attention + kept {keep} + head gate + zero sink B={B} n={n} ctx={ctx} window={win} {nq}/{nkv}x{d}", "new",
                [lambda k=k, v=v: K.attention(q, k, v, bt, sl, cu, n, sinks=sink, keep_first=keep, gate=g[:, :nq], **kw) for k, v in zip(kc, vc)], by, fl * seen(keep))
            row(f"attention B={B} n={n} ctx={ctx} window={win} {nq}/{nkv}x{d}", "like", [lambda k=k, v=v: K.attention(q, k, v, bt, sl, cu, n, **kw) for k, v in zip(kc, vc)],
                by, fl * seen(0))
            del kc, vc
            torch.cuda.empty_cache()
    K.check_status()


def bench_kernels_zegelix(dev, emit) -> None:
    from ..models.transformer import KVCache
    from ..ops import cuda as K
    from ..ops import ref
    from ..ops.weights import QuantWeight, WFormat
    from ..utils.rope import rope_tables
    t = _Rows(dev, emit)
    bf, i32, bufs, row = t.bf, t.i32, t.bufs, t.row
    mats = lambda n, k, e=1: [QuantWeight(WFormat.BF16, n, k, e, (torch.randn(e, n, k, device=dev) * k ** -0.5).to(torch.bfloat16)) for _ in range(bufs(e * n * k * 2))]
    f32 = lambda *sh: torch.randn(*sh, device=dev)
    for size, s in SIZES["zegelix"].items():
        H, nq, nkv, d, rot, win, pool, W, blocks = (s[k] for k in ("hidden", "heads", "kv_heads", "dim", "rot", "window", "pool", "width", "blocks"))
        E, top, ef, n_blk = s["experts"], s["used"], s["eff"], s["width"] // s["blocks"]
        for T in (1, 32, PREFILL):
            # ---- residual add + norm
            nb = bufs(T * H * 12) if T > 64 else 8
            xs, ds, w = [f32(T, H) for _ in range(nb)], [bf(T, H) for _ in range(nb)], torch.ones(H, device=dev)
            by = T * H * (4 + 4 + 2 + 2)
            row(f"sublayer_norm (add + norm) T={T} H={H}", "new", [lambda x=x, q=q: K.sublayer_norm(x, q, None, 1e-6, w=w) for x, q in zip(xs, ds)], by)
            row(f"rmsnorm (add + norm) T={T} H={H}", "like", [lambda x=x, q=q: K.rmsnorm(x, w, 1e-6, delta=q) for x, q in zip(xs, ds)], by)
            ys, pos, cw, z = [bf(T * top, H) for _ in range(nb)], torch.randperm(T * top, device=dev).to(torch.int32), torch.rand(T, top, device=dev), f32(T, E + 8)
            by = T * H * (4 + 4 + 2 + 2 * top)
            row(f"sublayer_norm of {top} weighted experts + gated shared T={T} H={H}", "new",
                [lambda x=x, y=y, q=q: K.sublayer_norm(x, ref.ExpertSum(y, pos, top, q, cw, z[:, E]), None, 1e-6, w=w) for x, y, q in zip(xs, ys, ds)], by + T * H * 2)
            row(f"rmsnorm_combine of {top} T={T} H={H}", "like", [lambda x=x, y=y: K.rmsnorm_combine(x, w, 1e-6, K.CombineDelta(y, pos, cw)) for x, y in zip(xs, ys)], by)
            del ds, ys
            # ---- experts
            h, idx = bf(T, H), torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(T)]).to(torch.int32)
            row(f"moe_route over {E} of {E + 8} columns T={T}", "new", [lambda: K.moe_route(z, None, top, experts=E)], T * (E + 2 * top) * 4)
            z2 = f32(T, E)
            row(f"moe_route T={T} {top} of {E}", "like", [lambda: K.moe_route(z2, None, top)], T * (E + 2 * top) * 4)
            gu = mats(2 * ef, H, E)
            live = min(E, T * top)
            by, fl = live * 2 * ef * H * 2 + T * top * (H + ef) * 2, 4.0 * T * top * ef * H
            for name, role, act in (("clamped SwiGLU", "new", ref.ACT_SWIGLU_OAI), ("SwiGLU", "like", ref.ACT_SWIGLU)):
                if T <= 4:
                    row(f"expert slots + {name} T={T}", role, [lambda m=m: K.expert_gemv(h, m, idx.reshape(-1), x_div=top, act=act, act_limit=5.0) for m in gu], by, fl)
                else:
                    pk = K.moe_pack(idx, E)
                    xp = K.moe_gather(h, pk)
                    row(f"grouped experts + {name} T={T}", role, [lambda m=m: K.grouped_linear(xp, m, pk.tile_expert, pk.num_tiles, act=act, act_limit=5.0) for m in gu], by, fl)
            del gu
            # ---- head epilogue
            kr, vr, full = rope_tables(2 * PREFILL, rot, 1e4, device=dev), rope_tables(2 * PREFILL, d, 1e4, device=dev), rope_tables(2 * PREFILL, d, 1e4, device=dev)
            pages, bs = T // 128 + 2, 128
            slots, pos1, temp = torch.arange(128, 128 + T, dtype=torch.int64, device=dev), torch.arange(T, dtype=torch.int32, device=dev), torch.ones(nq, device=dev)
            kc, vc = torch.zeros(pages, nkv, bs, d, dtype=torch.bfloat16, device=dev), torch.zeros(pages, nkv, bs, d, dtype=torch.bfloat16, device=dev)
            C = (nq + 2 * nkv) * d
            ys = [bf(T, C) for _ in range(min(8, bufs(T * nq * d * 4) if T > 64 else 8))]
            cut = lambda y, a, n: y[:, a * d:(a + n) * d].view(T, n, d)
            by = T * (nq * d * 4 + nkv * d * 8)
            row(f"qk_post with rotated values T={T}", "new",
                [lambda y=y: K.qk_post(cut(y, 0, nq), cut(y, nq, nkv), pos1, *kr, slots, kc, vc, d, rot, interleaved=True, v=cut(y, nq + nkv, nkv), v_rope=vr, q_scale=temp)
                 for y in ys], by)
            row(f"qkv_post T={T}", "like", [lambda y=y: K.qkv_post(y, None, None, None, pos1, *full, slots, kc, vc, nq, nkv, d, d) for y in ys], by)
            del ys, kc, vc
        # ---- recurrence and what is around it
        for B, n in ((1, PREFILL), (8, 512), (1, 1), (8, 1), (32, 1)):
            T = B * n
            slots, cu, sl = i32(list(range(B))), i32([i * n for i in range(B + 1)]), i32([n + 64] * B)
            nb = bufs(T * W * 8) if T > 64 else 8
            ps, cwt, cb = [bf(T, 2 * W) for _ in range(nb)], f32(W, 4), f32(W)
            cst, S, gb, coef = torch.zeros(B, 3, W, dtype=torch.bfloat16, device=dev), torch.zeros(B, W, device=dev), f32(blocks, 2 * n_blk), -torch.rand(W, device=dev)
            gm = mats(2 * n_blk, n_blk, blocks)
            if n > 1:
                row(f"causal_conv B={B} n={n} C={W}", "new", [lambda p=p: K.causal_conv(p[:, :W], cwt, cb, cst, slots, cu, sl, n) for p in ps], T * W * 4 + B * W * 12)
                row(f"conv1d_silu B={B} n={n} C={W}", "like", [lambda p=p: K.conv1d_silu(p[:, :W], cwt, cst, slots, cu, n) for p in ps], T * W * 4 + B * W * 12)
                us = [bf(T, W) for _ in range(nb)]
                row(f"gate products per block T={T} {blocks} x {2 * n_blk}x{n_blk}, fp32 results", "new",
                    [lambda u=u: K.head_linear(u.view(T, blocks, n_blk), gm[0], out_f32=True) for u in us], T * W * (2 + 8) + gm[0].nbytes, 4.0 * T * W * n_blk)
                row(f"gate products per block T={T}, 16-bit results", "like",
                    [lambda u=u: K.head_linear(u.view(T, blocks, n_blk), gm[0]) for u in us], T * W * (2 + 4) + gm[0].nbytes, 4.0 * T * W * n_blk)
                gs = [f32(T, blocks, 2 * n_blk) for _ in range(nb)]
                row(f"rglru_scan B={B} n={n} W={W}", "new",
                    [lambda g=g, u=u, p=p: K.rglru_scan(g, u, p[:, W:], gb, coef, S, slots, cu, sl, n) for g, u, p in zip(gs, us, ps)], T * W * (8 + 6) + B * W * 8)
                del gs, us
            else:
                row(f"rglru_step (conv, gates, recurrence) B={B} W={W}", "new",
                    [lambda p=p, m=m: K.rglru_step(p[:, :W], p[:, W:], cwt, cb, m, gb, coef, cst, S, slots, cu, sl) for p, m in zip(ps * (len(gm) // len(ps) + 1), gm)],
                    gm[0].nbytes + B * W * (6 + 8 + 12))
                pl = mats(2 * n_blk * blocks // 8, n_blk * 8)
                h = bf(T, n_blk * 8)
                row(f"plain projection with as many weights T={T}", "like", [lambda m=m: K.linear(h, m) for m in pl], pl[0].nbytes)
                row(f"conv1d_silu B={B} n={n} C={W}", "like", [lambda p=p: K.conv1d_silu(p[:, :W], cwt, cst, slots, cu, n) for p in ps], T * W * 4 + B * W * 12)
                del pl
            y3, zb = [bf(T, 3 * W) for _ in range(nb)], torch.zeros(W, device=dev)
            row(f"mingru_scan B={B} n={n} W={W}", "like",
                [lambda y=y: K.mingru_scan(y[:, :W], y[:, W:2 * W], y[:, 2 * W:], zb, zb, S, slots, cu, sl, n) for y in y3], T * W * 8 + B * W * 8)
            del ps, y3, gm
            torch.cuda.empty_cache()
        # ---- attention
        for B, n, ctx in ((1, PREFILL, PREFILL), (1, 512, PREFILL), (1, PREFILL, 4 * PREFILL), (1, 1, 8192), (1, 1, 2048), (32, 1, 2048), (32, 1, 8192)):
            T, nblk = B * n, (ctx + 127) // 128
            pages, blk_seen = B * nblk + 1, max(ctx - win, 0) // pool
            live = min(ctx, win + n) + blk_seen
            nb = min(16, bufs(B * live * nkv * d * 4)) if n == 1 else 2
            kvs = [KVCache(1, pages, nkv, d, dev, [0], pools={0: (pool, win)}) for _ in range(nb)]
            for kv in kvs:
                for x in (kv.k[0], kv.v[0], kv.pools[0].k, kv.pools[0].v):
                    x.normal_(0.0, 0.5)
            bt = torch.arange(1, pages, dtype=torch.int32, device=dev).reshape(B, nblk)
            sl, cu = i32([ctx] * B), i32([i * n for i in range(B + 1)])
            q, g, sink, turn = bf(T, nq, d), bf(T, nq * d), torch.zeros(nq, device=dev), rope_tables(ctx, d, 1e4, device=dev)
            pairs = float(sum(min(p + 1, win) + max(p + 1 - win, 0) // pool for p in range(ctx - n, ctx)))
            plain = float(sum(min(p + 1, win) for p in range(ctx - n, ctx)))
            by = lambda keys, gated: B * keys * nkv * d * 4 + T * nq * d * (6 if gated else 4)
            kw = dict(window=win, scale=d ** -0.5, max_kv_len=ctx)
            name = f"B={B} n={n} ctx={ctx} window={win} {nq}/{nkv}x{d}"
            if n > 1:
                form = lambda kv: K.pool_blocks(kv.k[0], kv.v[0], kv.pools[0], bt, sl, cu, n, max_kv_len=ctx)
                row(f"pool_blocks {name}", "new", [lambda kv=kv: form(kv) for kv in kvs], (min(ctx, win + n) - win + 2 * blk_seen) * nkv * d * 4)
                src = bf(T, 2 * nkv * d)
                at = torch.arange(128, 128 + T, dtype=torch.int64, device=dev)
                row(f"kv_store T={T}", "like", [lambda kv=kv: K.kv_store(src[:, :nkv * d], src[:, nkv * d:], at, kv.k[0], kv.v[0]) for kv in kvs], T * nkv * d * 8)
                dense = [form(kv) for kv in kvs]
            else:
                dense = [None] * nb
            for cap in (50.0, 1.0, 0.0):                   # scores far below the cap, around it, and no cap
                row(f"attention + pooled blocks + cap {cap:g} + sink + gate + turn {name}", "new",
                    [lambda kv=kv, x=x: K.attention(q, kv.k[0], kv.v[0], bt, sl, cu, n, sinks=sink, softcap=cap, gate=g, pools=kv.pools[0], pool_dense=x, out_rope=turn, **kw)
                     for kv, x in zip(kvs, dense)], by(live, True), 4.0 * B * nq * d * pairs)
            if d in (64, 128, 256):
                row(f"attention + cap 50 {name}", "like", [lambda kv=kv: K.attention(q, kv.k[0], kv.v[0], bt, sl, cu, n, softcap=50.0, **kw) for kv in kvs],
                    by(min(ctx, win + n), False), 4.0 * B * nq * d * plain)
            row(f"attention {name}", "like", [lambda kv=kv: K.attention(q, kv.k[0], kv.v[0], bt, sl, cu, n, **kw) for kv in kvs], by(min(ctx, win + n), False),
                4.0 * B * nq * d * plain)
            del kvs, dense
            torch.cuda.empty_cache()
    K.check_status()


def main(design: str, part: str = "all") -> int:
    dev = torch.device("cuda:0")
    torch.cuda.set_device(dev)
    t0 = time.time()

    def emit(obj):
        print(json.dumps(obj))
        sys.stdout.flush()
    if part in ("all", "models"):
        bench_models(design, dev, emit)
    if part in ("all", "kernels"):
        {"tikarax": bench_kernels_tikarax, "pubodra": bench_kernels_pubodra, "beputar": bench_kernels_beputar, "zegelix": bench_kernels_zegelix}[design](dev, emit)
    emit({"design_bench": "done", "seconds": round(time.time() - t0, 1)})
    return 0
