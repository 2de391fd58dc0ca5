"""Trace replay: feed given token ids through an engine, step by step, and write the logits that were asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one batch through :meth:`LLMEngine.feed`: prompt portions beside single decoded tokens, on the
paged cache, the state slots and the kernels that serving uses.  For a step with wanted places ``DIR/<step>.f32`` receives
the logits (little-endian fp32, ``[wanted, vocab]``, in the order of the entries and of ``want``); every step ends with a line
``done <step>``.  The KV pool is made for ``--max-tokens`` tokens and the state pool for ``MAX_LIVE`` requests, so pages and
slots are used again.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4              # requests that are live at the same time
BLOCK_SIZE = 16
TOKEN_ROUNDING = 64       # a request's share of --max-tokens is rounded up to this many tokens: a multiple of BLOCK_SIZE


def build_engine(path: str, dtype: str, max_tokens: int, device=None, use_cuda_graphs: bool = True):
    import torch

    from .config import EngineConfig, ModelConfig
    from .loader import Checkpoint, load_weights
    from .models import build_model
    device = device or "cuda:0"
    cfg = ModelConfig.from_pretrained(path)
    cfg.dtype = dtype
    if str(device).startswith("cuda"):
        from . import build
        from .ops import cuda as K
        if not build.kernels_current():             # a fresh checkout: only the translation units this model calls
            K.use_library(build.build_kernels(verbose=True, units=build.units_for(cfg)))
        torch.cuda.set_device(device)
    model = build_model(cfg, device=device)
    load_weights(model, Checkpoint(path))
    max_len = (max_tokens + TOKEN_ROUNDING - 1) // TOKEN_ROUNDING * TOKEN_ROUNDING
    model.finalize(max_len)
    from .engine import LLMEngine
    return LLMEngine(model, EngineConfig(max_seq_len=max_len, block_size=BLOCK_SIZE, num_kv_blocks=max_len // BLOCK_SIZE,
                                         max_num_seqs=MAX_LIVE, max_batch_size=MAX_LIVE, max_prefill_tokens=max_len,
                                         enable_prefix_caching=False, use_cuda_graphs=use_cuda_graphs))


def replay(engine, lines, out_dir: str, answer) -> int:
    """Run the steps of ``lines``; ``answer(text)`` receives one line per finished step.  Returns the number of steps."""
    import numpy as np
    n = 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = engine.feed([(e["id"], e["tokens"], e.get("want", [])) for e in step.get("entries", [])], step.get("end", []))
        wanted = [p for p in parts if p.shape[0]]
        if wanted:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            np.concatenate([p.numpy() for p in wanted]).astype("<f4").tofile(path)
        elif engine.model.device.type == "cuda":
            import torch
            torch.cuda.synchronize()                 # "done" means that the step has run
        answer(f"done {step['step']}")
        n += 1
    return n


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most at any time")
    ap.add_argument("--device", default="cuda:0", help="cuda:N, or cpu for the plain PyTorch path")
    args = ap.parse_args(argv)
    # libraries may print to descriptor 1 on their own: keep it for the answers
    sys.stdout.flush()
    answers = os.fdopen(os.dup(1), "w")
    os.dup2(2, 1)
    engine = build_engine(args.model, args.dtype, args.max_tokens, device=args.device)

    def answer(text: str) -> None:
        answers.write(text + "\n")
        answers.flush()
    replay(engine, sys.stdin, args.out, answer)
    if engine.model.device.type == "cuda":
        from .ops import cuda as K
        status = K.check_status()
        if status:
            print(f"trace_run: device status word {status:#x}", file=sys.stderr)
            return 4
    return 0
