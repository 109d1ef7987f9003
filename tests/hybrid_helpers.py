"""Helpers of the tests of layer-by-layer decoders: an engine for a configuration, schedules, comparison."""
from __future__ import annotations

import torch

from mindspeed_rl_b200.models.hybrid_config import HybridConfig
from mindspeed_rl_b200.rollout.engine import LLMEngine
from mindspeed_rl_b200.rollout.hybrid_weights import build_hybrid_weights

# bf16: the positions of the worst rounding (nearly tied scores, small norms) reach several times the mean
TOL = {torch.float32: 3e-5, torch.bfloat16: 9e-2}


def make_engine(cfg, w, device, dtype=torch.float32, *, seqs=8, budget=512, blocks=64, block=16, model_len=512, graphs=()):
    cfg = HybridConfig.from_json(cfg, dtype)
    eng = LLMEngine(cfg, device, max_num_seqs=seqs, max_model_len=model_len, max_num_batched_tokens=budget, block_size=block,
                    enforce_eager=not graphs, graph_batch_sizes=graphs)
    eng.runner.bind_weights(build_hybrid_weights(cfg, w, device))
    eng.init_cache(blocks)
    return eng


def close(got, want, dtype=torch.float32, tol=None):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(err.max()) < (tol or TOL[dtype]), (float(err.max()), int(err.argmax()))
    if tol is None and dtype == torch.bfloat16:
        assert float(err.mean()) < 2e-2, float(err.mean())


def run_schedule(eng, seq, cuts, rid="r", end=True):
    """Logits of every token of ``seq`` fed in portions of the given sizes (the last size repeats)."""
    at, k, out = 0, 0, []
    while at < len(seq):
        n = min(cuts[min(k, len(cuts) - 1)], len(seq) - at)
        last = at + n == len(seq)
        out.append(eng.replay([(rid, seq[at:at + n], list(range(n)))], [rid] if last and end else []).float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


def dtypes(device):
    return (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16)
