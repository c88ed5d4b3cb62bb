"""Replays a trace of token ids through the engine, step by step, and writes the logits that were asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Every line of standard input is one step, a JSON object:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
``entries``: the next tokens of each request (all of them run as one batch) and the places among these tokens whose logits are wanted;
``end``: requests that are finished after the step.  A step with wanted logits writes OUT/<step>.f32 (little-endian fp32 [wanted, vocab], in the
order of the entries and of ``want``); every step then prints "done <step>".  Nothing is sampled: the tokens come from the trace, everything else --
batch assembly, pages, state slots, kernels, graphs -- is the engine's (``LLMEngine.feed``).

``--max-tokens``: what live requests hold at most, each rounded up to a multiple of 64; the page pool is made for that many.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4                 # requests alive at the same time (sequence and state slots)
ROUND = 64


def build_engine(model_dir: str, dtype: str, max_tokens: int, device):
    from ..models import load_model
    from ..models.transformer import KV_BLOCK
    from ..runtime.engine import EngineOptions, LLMEngine
    # a request of n tokens holds ceil(n / KV_BLOCK) pages: at most KV_BLOCK - ROUND tokens more than its share of max_tokens; page 0 is the null page
    pages = (max_tokens + MAX_LIVE * (KV_BLOCK - ROUND)) // KV_BLOCK + 1
    max_ctx = (max_tokens + KV_BLOCK - 1) // KV_BLOCK * KV_BLOCK
    model, _ = load_model(model_dir, device, max_ctx=max_ctx, dtype=dtype)
    return LLMEngine(model, EngineOptions(max_ctx=max_ctx, max_batch_tokens=max_ctx, max_seqs=MAX_LIVE, num_blocks=pages, enable_prefix_cache=False,
                                          graph_batch_sizes=tuple(range(1, MAX_LIVE + 1))))


def replay(eng, lines, out_dir: str, announce) -> None:
    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        entries = []
        for e in st["entries"]:
            if e["id"] not in live:
                live[e["id"]] = eng.open_sequence()
            entries.append((live[e["id"]], [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])]))
        logits = eng.feed(entries) if entries else None
        if logits is not None:
            path = os.path.join(out_dir, f"{st['step']}.f32")
            logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tofile(path)
        for rid in st.get("end", []):
            seq = live.pop(rid, None)
            if seq is not None:
                eng.abort(seq)
        announce(f"done {st['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json + safetensors) or GGUF file")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--cpu", action="store_true", help="run the PyTorch restatement of the kernels on the CPU")
    a = ap.parse_args(argv)
    if a.max_tokens < 1:
        ap.error("--max-tokens must be positive")
    import torch
    from .. import _lib
    if not a.cpu:
        _lib.use_components("core")          # a checkout without built kernels compiles what this needs, not every family's
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device (use --cpu for the CPU restatement)")
    dev = torch.device("cpu") if a.cpu else torch.device("cuda", 0)
    eng = build_engine(a.model, {"bfloat16": "bf16", "float32": "fp32"}[a.dtype], a.max_tokens, dev)
    os.makedirs(a.out, exist_ok=True)

    def announce(text: str) -> None:
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    with torch.inference_mode():
        replay(eng, sys.stdin, a.out, announce)
    if not a.cpu:
        from ..ops import cuda as kernels
        kernels.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
