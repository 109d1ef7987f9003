#!/usr/bin/env python
"""Generate with a model folder (config.json + safetensors) through the rollout engine.

    python cli/generate.py --model DIR --prompt-ids "5 17 3" --prompt-ids "8 1" --max-tokens 32 --temperature 0
    python cli/generate.py --model DIR --prompt "text" --tokenizer DIR

The model class is chosen by the architecture that config.json names (``mindspeed_rl_b200.models.registry``).
Prints one JSON line per prompt: token ids, log-probabilities and finish reason of every sample.
"""
import argparse
import json
import os
import sys

sys.path.insert(0, os.path.abspath(os.path.join(os.path.dirname(__file__), "..")))


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    ap.add_argument("--prompt-ids", action="append", default=[], metavar="IDS", help="token ids separated by blanks or commas")
    ap.add_argument("--prompt", action="append", default=[], metavar="TEXT", help="needs --tokenizer")
    ap.add_argument("--tokenizer", default=None, help="Hugging Face tokenizer folder")
    ap.add_argument("--n", type=int, default=1, help="samples per prompt")
    ap.add_argument("--max-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=1.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=-1)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--min-p", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--eos-token-id", type=int, default=-1)
    ap.add_argument("--max-num-seqs", type=int, default=64)
    ap.add_argument("--max-model-len", type=int, default=4096)
    ap.add_argument("--max-num-batched-tokens", type=int, default=8192)
    ap.add_argument("--block-size", type=int, default=16)
    ap.add_argument("--num-blocks", type=int, default=None, help="cache blocks (default: enough for the given prompts)")
    ap.add_argument("--enforce-eager", action="store_true", help="no CUDA graphs for decode steps")
    args = ap.parse_args(argv)

    import torch

    from mindspeed_rl_b200.models.registry import load_model
    from mindspeed_rl_b200.rollout.engine import LLMEngine
    from mindspeed_rl_b200.rollout.scheduler import SamplingParams

    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.prompt_ids]
    tokenizer = None
    if args.prompt:
        from mindspeed_rl_b200.utils.tokenizer import get_tokenizer

        if args.tokenizer is None:
            ap.error("--prompt needs --tokenizer")
        tokenizer = get_tokenizer(args.tokenizer, "HuggingFaceTokenizer")
        prompts += [list(tokenizer.tokenize(p)) for p in args.prompt]
    if not prompts:
        ap.error("give at least one --prompt-ids or --prompt")
    cfg, weights = load_model(args.model, getattr(torch, args.dtype), args.device)
    seqs = max(args.n, min(args.max_num_seqs, len(prompts) * args.n))
    longest = min(args.max_model_len, max(len(p) for p in prompts) + args.max_tokens)
    blocks = args.num_blocks or seqs * ((longest + args.block_size - 1) // args.block_size + 1)
    engine = LLMEngine(cfg, args.device, max_num_seqs=seqs, max_num_batched_tokens=args.max_num_batched_tokens,
                       max_model_len=args.max_model_len, block_size=args.block_size, seed=args.seed,
                       enforce_eager=args.enforce_eager or args.device == "cpu", graph_batch_sizes=(1, 2, 4, 8, 16, 32, 64),
                       eos_token_id=args.eos_token_id)
    engine.runner.bind_weights(weights)
    engine.init_cache(blocks)
    outs = engine.generate(prompts, SamplingParams(n=args.n, temperature=args.temperature, top_k=args.top_k, top_p=args.top_p,
                                                   min_p=args.min_p, max_tokens=args.max_tokens, seed=args.seed))
    for o in outs:
        line = {"prompt_token_ids": o.prompt_token_ids,
                "outputs": [{"token_ids": c.token_ids, "logprobs": c.logprobs, "finish_reason": c.finish_reason}
                            for c in o.outputs]}
        if tokenizer is not None:
            for c, d in zip(o.outputs, line["outputs"]):
                d["text"] = tokenizer.detokenize(c.token_ids)
        print(json.dumps(line), flush=True)
    return outs


if __name__ == "__main__":
    main()
