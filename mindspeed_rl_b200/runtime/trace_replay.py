"""Replay of a request trace: given token ids go through a model step by step, logits come out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is one step::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch; ``want`` are the places among an entry's tokens whose logits are written to
``<out>/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, in the order of the entries); ``end`` releases
requests.  After every step the line ``done <step>`` is printed.  Nothing is sampled: the engine's own step
function, cache, state manager and kernels run on the ids of the trace (``LLMEngine.replay``), which makes a
trace of production requests, or a schedule that went wrong, repeatable.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

DECODE_GRAPHS = (1, 2, 4, 8, 16, 32, 64)


def parse(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=256, help="most requests that are live at any time")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: PyTorch formulation, for machines without a GPU")
    return ap.parse_args(argv)


def build_engine(args):
    import torch

    from ..models.registry import load_model, use_kernels_of
    from ..rollout.engine import LLMEngine

    if args.device == "cuda":
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device (use --device cpu for the PyTorch formulation)")
        use_kernels_of(args.model)
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    cfg, weights = load_model(args.model, getattr(torch, args.dtype), args.device)
    block = 16
    requests = max(1, min(args.max_requests, args.max_tokens))
    engine = LLMEngine(cfg, args.device, max_num_seqs=requests, max_num_batched_tokens=8192,
                       max_model_len=max(args.max_tokens, 1) + 1, block_size=block, enforce_eager=args.device == "cpu",
                       graph_batch_sizes=DECODE_GRAPHS)
    engine.runner.bind_weights(weights)
    engine.init_cache((args.max_tokens + block - 1) // block + requests)      # a part-filled block per request
    return engine


def run(engine, lines, out_dir: str, report) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.replay([(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]], step.get("end", []))
        if logits.shape[0]:
            rows = logits.float().cpu().numpy().astype("<f4", copy=False)
            np.ascontiguousarray(rows).tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        elif engine.device.type == "cuda":
            import torch

            torch.cuda.synchronize()
        report(f"done {step['step']}")


def main(argv=None) -> int:
    args = parse(argv)
    os.makedirs(args.out, exist_ok=True)
    engine = build_engine(args)
    run(engine, sys.stdin, args.out, lambda text: print(text, flush=True))
    if engine.device.type == "cuda":
        from ..ops.gemm import check_status

        check_status(engine.device, "trace replay")
    return 0
