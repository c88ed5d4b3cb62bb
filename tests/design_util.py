"""Shared by the tests of layer-list designs: checkpoint folders from oracle weights, engines over them, the error measure."""
import json
import os

import numpy as np
import pytest
import torch

from machx_inference_engine_b200.formats.safetensors import write_safetensors
from machx_inference_engine_b200.models import load_model
from machx_inference_engine_b200.runtime.engine import EngineOptions, LLMEngine

DEVICES = ["cpu", pytest.param("cuda:0", marks=pytest.mark.gpu)]
# (device, compute dtype): every model-level test runs in both arithmetics on both devices
ARMS = [("cpu", "fp32"), ("cpu", "bf16"), pytest.param(("cuda:0", "fp32"), marks=pytest.mark.gpu), pytest.param(("cuda:0", "bf16"), marks=pytest.mark.gpu)]
# relative error of logits against the float64 oracle
TOL = {"fp32": 2e-5, "bf16": 4e-2}


def write_folder(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    bits = {n: ("BF16", (np.array(a, dtype=np.float32, order="C").view(np.uint32) >> 16).astype(np.uint16)) for n, a in weights.items()}
    write_safetensors(os.path.join(path, "model.safetensors"), bits)
    return str(path)


def engine(path, arm, max_ctx=1024, num_blocks=0, max_seqs=4, **kw):
    device, dtype = arm
    model, _ = load_model(path, torch.device(device), max_ctx=max_ctx, dtype=dtype)
    return LLMEngine(model, EngineOptions(max_ctx=max_ctx, max_batch_tokens=max_ctx, max_seqs=max_seqs, num_blocks=num_blocks,
                                          enable_prefix_cache=kw.pop("enable_prefix_cache", False), **kw))


def logit_error(got, want):
    """Largest, over the positions, of rms(difference) / rms(logits), both with their mean taken off."""
    g, w = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = g - w
    d = d - d.mean(-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(-1)).max() / np.sqrt(((w - w.mean(-1, keepdims=True)) ** 2).mean()))


def run_portions(eng, tokens, sizes):
    """Feeds one sequence in portions of the given sizes (the rest one token at a time); logits of every position [T, vocab]."""
    seq, out, at, sizes = eng.open_sequence(), [], 0, list(sizes)
    while at < len(tokens):
        n = min(sizes.pop(0) if sizes else 1, len(tokens) - at)
        out.append(eng.feed([(seq, tokens[at:at + n], list(range(n)))]).cpu())
        at += n
    eng.abort(seq)
    return torch.cat(out).numpy()


def tokens_of(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()
