"""Serving throughput of layer-by-layer decoders beside the closest repeated-block decoders of equal size.

``bench.py --workload serve`` runs it: random weights, prompts and decode batches through ``LLMEngine`` (the
scheduler, cache, graphs and sampler of generation).

Pumotar: ``latent`` has latent attention everywhere, ``mixed`` one such layer after three recurrent ones.  Closest
existing model: ``mla``, the latent-attention decoder with routed experts of the same width, heads, head sizes, latent
rank, feed-forward sizes, experts and layer count; it caches full per-head keys and values.

Sunatar: ``window`` has window attention everywhere, ``memory`` the matrix memory everywhere, ``sunatar`` one
matrix-memory layer in four.  Closest existing models: ``gqa``, the grouped-head decoder with routed and shared experts
of the same width, heads, experts and layer count (full attention), and for the recurrent layers ``mixed``.

Gapevik: ``conv`` has convolved attention in chunks everywhere, ``gated`` latent attention with a query latent, window, sink
and gates, ``delta`` the delta rule with a decay per head, ``gapevik`` the three in turn.  Closest existing models of the same
width, heads, experts and layer count: ``window``, ``latent`` and ``mixed``.

Lunelorn: ``retention``, ``turned`` (attention with turned values beside the minimal gated recurrence) and ``wkv`` have that mixer
everywhere, ``lunelorn`` the three in turn; no layer is looped.  Closest existing models: ``memory``, ``gqa`` and ``delta``.

One JSON line per measurement: tokens/s from CUDA events around the engine calls.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import List

import torch

from ..models.hybrid_config import (ChannelDeltaSpec, ChosenMoESpec, Chunk, ConvAttentionSpec, GluSpec, HeadDeltaSpec, HybridConfig,
                                    LatentAttentionSpec, LayerSpec, MatrixMemorySpec, MinGRUSpec, ParallelSpec, RetentionSpec,
                                    Rotary, ScoredMoESpec, SoftmaxMoESpec, TableMoESpec, TurnedAttentionSpec, WKVSpec,
                                    WavelengthScaling, WindowAttentionSpec)
from ..models.transformer_config import TransformerConfig
from .engine import LLMEngine
from .scheduler import SamplingParams


@dataclass(frozen=True)
class Size:
    name: str
    width: int
    heads: int
    rank: int
    ff: int
    experts: int
    top: int
    expert_ff: int
    layers: int = 4
    vocab: int = 32768
    dn: int = 64
    dr: int = 64
    dv: int = 128


SIZES = (Size("1k", 1024, 8, 256, 4096, 32, 4, 512), Size("2k", 2304, 32, 512, 9216, 64, 8, 1024),
         Size("4k", 4096, 32, 512, 12288, 64, 4, 2048))
PREFILL = ((1, 8192), (8, 2048))
DECODE = ((1, 2048), (32, 2048), (256, 2048))
NEW_TOKENS = 64
WINDOW = 1024
MODELS = ("mla", "latent", "mixed", "gqa", "window", "memory", "sunatar", "conv", "gated", "delta", "gapevik", "retention", "turned", "wkv",
          "lunelorn")


def sunatar_config(s: Size, pattern: str) -> HybridConfig:
    rot = Rotary(64, 500000.0, halves=True, scaling=WavelengthScaling(8.0, 1.0, 4.0, 8192))
    window = LayerSpec("attention", WindowAttentionSpec(s.heads, s.heads // 4, 128, 128, 128 ** -0.5, rot, WINDOW, True))
    memory = LayerSpec("mlstm", MatrixMemorySpec(s.heads, 128, 128, 15.0))
    glu = GluSpec(s.expert_ff, "silu")
    moe = ScoredMoESpec(s.experts, s.top, glu, glu)
    layers = []
    for i in range(s.layers):
        m = memory if pattern == "memory" or (pattern == "sunatar" and i % 4 == 2) else window
        layers.append(LayerSpec(m.type, m.mixer, moe))
    return HybridConfig("Sunatar", s.vocab, s.width, layers, 1e-5)


def gapevik_config(s: Size, pattern: str) -> HybridConfig:
    kinds = {"conv": ("attention", ConvAttentionSpec(s.heads, s.heads // 4, 128, 128, 4, 128 ** -0.5, Rotary(64, 500000.0), 30.0,
                                                     Chunk(WINDOW))),
             "gated": ("latent_attention", LatentAttentionSpec(s.heads, s.dn, s.dr, s.dv, s.rank, (s.dn + s.dr) ** -0.5,
                                                               Rotary(s.dr, 10000.0, halves=True), 3 * s.rank // 2, WINDOW, True, True)),
             "delta": ("delta", HeadDeltaSpec(s.heads, s.heads // 2, 128, 128, 4))}
    moe = SoftmaxMoESpec(s.experts, s.top, GluSpec(s.expert_ff, "silu"), s.experts // 8)
    layers = [LayerSpec(*kinds[pattern if pattern in kinds else tuple(kinds)[i % 3]], moe) for i in range(s.layers)]
    return HybridConfig("Gapevik", s.vocab, s.width, layers, 1e-5, residual_mult=0.5)


def lunelorn_config(s: Size, pattern: str) -> HybridConfig:
    left = TurnedAttentionSpec(s.heads, s.heads // 4, 128, 128, 128 ** -0.5, Rotary(64, 500000.0, halves=True))
    kinds = {"retention": RetentionSpec(s.heads, 128, 128, tuple(1.0 - 2.0 ** (-5 - 8 * i / s.heads) for i in range(s.heads))),
             "turned": ParallelSpec(left, MinGRUSpec(s.width), 0.7, 0.7), "wkv": WKVSpec(2 * s.heads, 64, s.width)}
    moe = ChosenMoESpec(s.experts, s.top, GluSpec(s.expert_ff, "silu"))
    layers = []
    for i in range(s.layers):
        name = pattern if pattern in kinds else ("wkv", "retention", "turned")[i % 3]
        layers.append(LayerSpec("parallel" if name == "turned" else name, kinds[name], moe))
    return HybridConfig("Lunelorn", s.vocab, s.width, layers, 1e-5, token_side=64, logit_softcap=30.0)


def hybrid_config(s: Size, pattern: str) -> HybridConfig:
    if pattern in ("retention", "turned", "wkv", "lunelorn"):
        return lunelorn_config(s, pattern)
    if pattern in ("conv", "gated", "delta", "gapevik"):
        return gapevik_config(s, pattern)
    if pattern in ("window", "memory", "sunatar"):
        return sunatar_config(s, pattern)
    latent = LayerSpec("latent_attention", LatentAttentionSpec(s.heads, s.dn, s.dr, s.dv, s.rank, (s.dn + s.dr) ** -0.5,
                                                               Rotary(s.dr, 10000.0)))
    delta = LayerSpec("channel_delta", ChannelDeltaSpec(s.heads, s.heads, 128, 128, 4))
    dense = GluSpec(s.ff, "gelu_tanh")
    act = dict(act="clamped_swish", limit=7.0, alpha=1.702)
    moe = TableMoESpec(s.experts, s.top, GluSpec(s.expert_ff, **act), GluSpec(s.expert_ff, **act))
    layers = []
    for i in range(s.layers):
        m = latent if pattern == "latent" or i % 4 == 3 else delta
        layers.append(LayerSpec(m.type, m.mixer, dense if i == 0 else moe))
    return HybridConfig("Pumotar", s.vocab, s.width, layers, 1e-5)


def random_state(cfg: HybridConfig, device) -> dict:
    """Random checkpoint tensors of a configuration (drawn on the device)."""
    g = torch.Generator(device=device).manual_seed(0)
    w, out = cfg.hidden_size, {}

    def lin(name, rows, cols):
        out[name] = (torch.randn(rows, cols, generator=g, device=device) * cols ** -0.5).to(cfg.params_dtype)

    def vec(name, n, mean=0.0):
        out[name] = torch.full((n,), mean, device=device)

    def glu(p, ff):
        lin(p + "gate", ff, w)
        lin(p + "up", ff, w)
        lin(p + "down", w, ff)

    lin("embed", cfg.vocab_size, w)
    ones = 1.0 - cfg.design.norm_offset
    vec("final.norm", w, ones)
    if not cfg.design.tied_head:
        lin("head", cfg.vocab_size, w)
    if cfg.design.embed_norm:
        vec("embed.norm", w, ones)
    if cfg.token_side:
        lin("side.embed", cfg.vocab_size, len(cfg.layers) * cfg.token_side)
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.mix.", l.mixer
        vec(f"l{i}.norm1", w, ones)
        if not cfg.design.parallel:
            vec(f"l{i}.norm2", w, ones)
        if cfg.design.sandwich:
            vec(f"l{i}.norm1b", w, ones)
            vec(f"l{i}.norm2b", w, ones)
        if cfg.token_side:
            lin(f"l{i}.side.gate", cfg.token_side, w)
            lin(f"l{i}.side.proj", w, cfg.token_side)
            vec(f"l{i}.side.norm", w, ones)
        if isinstance(m, RetentionSpec):
            for n, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
                lin(p + n, rows, w)
            lin(p + "o", w, m.heads * m.vdim)
        elif isinstance(m, ParallelSpec):
            a, r = m.left, m.right.width
            for n, rows in (("left.q", a.heads * a.dim), ("left.k", a.kv_heads * a.dim), ("left.v", a.kv_heads * a.vdim),
                            ("right.z", r), ("right.x", r), ("right.g", r)):
                lin(p + n, rows, w)
            vec(p + "right.z.b", r, -2.0)
            vec(p + "right.x.b", r)
            lin(p + "left.o", w, a.heads * a.vdim)
            lin(p + "right.o", w, r)
        elif isinstance(m, WKVSpec):
            hd = m.heads * m.dim
            for n in "rkvgw":
                vec(p + "mu." + n, w, 0.5)
            for n in "rkvg":
                lin(p + n, hd, w)
            lin(p + "w1", 64, w)
            lin(p + "w2", hd, 64)
            vec(p + "w0", hd, -3.0)
            vec(p + "u", hd, 0.5)
            vec(p + "norm", hd, 1.0)
            lin(p + "o", w, hd)
        elif isinstance(m, LatentAttentionSpec):
            if m.q_rank:
                lin(p + "dq", m.q_rank, w)
                vec(p + "dq.norm", m.q_rank, 1.0)
            lin(p + ("uq" if m.q_rank else "q"), m.heads * (m.dim + m.rot_dim), m.q_rank or w)
            if m.sink:
                vec(p + "sink", m.heads)
            if m.head_gate:
                lin(p + "g", m.heads, w)
            lin(p + "dkv", m.kv_rank + m.rot_dim, w)
            vec(p + "dkv.norm", m.kv_rank, 1.0)
            lin(p + "uk", m.heads * m.dim, m.kv_rank)
            lin(p + "uv", m.heads * m.vdim, m.kv_rank)
            lin(p + "o", w, m.heads * m.vdim)
        elif isinstance(m, ConvAttentionSpec):
            for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                lin(p + n, rows, w)
                out[p + n + ".conv"] = torch.randn(rows, m.conv, generator=g, device=device) * 0.5
            vec(p + "q.norm", m.dim, 1.0)
            vec(p + "k.norm", m.dim, 1.0)
            lin(p + "g", m.heads, w)
            lin(p + "o", w, m.heads * m.vdim)
        elif isinstance(m, WindowAttentionSpec):
            for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                lin(p + n, rows, w)
                vec(p + n + ".b", rows)
            vec(p + "q.norm", m.heads * m.dim, 1.0)
            vec(p + "k.norm", m.kv_heads * m.dim, 1.0)
            out[p + "vmix"] = torch.tensor(0.3, device=device)
            lin(p + "o", w, m.heads * m.vdim)
        elif isinstance(m, MatrixMemorySpec):
            for n, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim),
                            ("i", m.heads), ("f", m.heads)):
                lin(p + n, rows, w)
            vec(p + "i.b", m.heads)
            vec(p + "f.b", m.heads, 3.0)
            vec(p + "norm", m.heads * m.vdim, 1.0)
            lin(p + "o", w, m.heads * m.vdim)
        else:
            kd, hv = m.kv_heads * m.dim, m.heads * m.vdim
            for n, rows in (("q", kd), ("k", kd), ("v", hv)):
                lin(p + n, rows, w)
                out[p + n + ".conv"] = torch.randn(rows, m.conv, generator=g, device=device) * 0.5
            lin(p + "b", m.heads, w)
            vec(p + "A_log", m.heads, -2.0)
            vec(p + "norm", m.vdim, 1.0)
            if isinstance(m, HeadDeltaSpec):
                vec(p + "dt_bias", m.heads)
                lin(p + "a", m.heads, w)
                lin(p + "g", hv, w)
            else:
                vec(p + "dt_bias", m.heads * m.dim)
                for a, n in (("a", m.heads * m.dim), ("g", hv)):
                    lin(p + a + "1", 128, w)
                    lin(p + a + "2", n, 128)
            lin(p + "o", w, hv)
        p = f"l{i}.mlp."
        if isinstance(l.mlp, ScoredMoESpec):
            for e in range(l.mlp.experts):
                glu(f"{p}e{e}.", l.mlp.expert.ff)
            lin(p + "router", l.mlp.experts, w)
            glu(p + "shared.", l.mlp.shared.ff)
        elif isinstance(l.mlp, ChosenMoESpec):
            for e in range(l.mlp.experts):
                glu(f"{p}e{e}.", l.mlp.expert.ff)
            lin(p + "router", l.mlp.experts, w)
        elif isinstance(l.mlp, SoftmaxMoESpec):
            for e in range(l.mlp.experts):
                glu(f"{p}e{e}.", l.mlp.expert.ff)
            lin(p + "router", l.mlp.outputs, w)
            vec(p + "correction", l.mlp.outputs)
        elif isinstance(l.mlp, TableMoESpec):
            for e in range(l.mlp.experts):
                glu(f"{p}e{e}.", l.mlp.expert.ff)
            out[p + "table"] = torch.rand(cfg.vocab_size, l.mlp.experts, generator=g, device=device).topk(l.mlp.top, -1).indices
            glu(p + "shared.", l.mlp.shared.ff)
            lin(p + "shared.sg", 1, w)
        else:
            glu(p, l.mlp.ff)
    return out


def mla_config(s: Size) -> TransformerConfig:
    return TransformerConfig(num_layers=s.layers, hidden_size=s.width, ffn_hidden_size=s.ff, num_attention_heads=s.heads,
                             num_query_groups=s.heads, vocab_size=s.vocab, norm_epsilon=1e-5, max_position_embeddings=16384,
                             untie_embeddings_and_output_weights=False, num_experts=s.experts, moe_router_topk=s.top,
                             moe_ffn_hidden_size=s.expert_ff, n_shared_experts=1, first_k_dense_replace=1,
                             multi_latent_attention=True, kv_lora_rank=s.rank, qk_head_dim=s.dn, qk_pos_emb_head_dim=s.dr,
                             v_head_dim=s.dv)


def gqa_config(s: Size) -> TransformerConfig:
    return TransformerConfig(num_layers=s.layers, hidden_size=s.width, ffn_hidden_size=s.ff, num_attention_heads=s.heads,
                             num_query_groups=s.heads // 4, kv_channels=128, vocab_size=s.vocab, norm_epsilon=1e-5,
                             max_position_embeddings=16384, qk_layernorm=True, untie_embeddings_and_output_weights=True,
                             num_experts=s.experts, moe_router_topk=s.top, moe_ffn_hidden_size=s.expert_ff, n_shared_experts=1)


def build(s: Size, model: str, device):
    if model in ("mla", "gqa"):
        from ..models.gpt import GPTModel
        from ..reshard.alias import alias_rollout_weights

        cfg = mla_config(s) if model == "mla" else gqa_config(s)
        return cfg, alias_rollout_weights(GPTModel(cfg, device=device))
    from .hybrid_weights import build_hybrid_weights

    cfg = hybrid_config(s, model)
    return cfg, build_hybrid_weights(cfg, random_state(cfg, device), device)


def _timed(fn) -> float:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1)


def run(steps: int, warmup: int, sizes=None, models=None, emit=print) -> List[dict]:
    dev = torch.device("cuda")
    rows = []
    for s in SIZES:
        if sizes and s.name not in sizes:
            continue
        gen = torch.Generator().manual_seed(1)
        for model in models or MODELS:
            cfg, weights = build(s, model, dev)
            bs = max(b for b, _ in DECODE)
            ctx = max(n for _, n in DECODE) + NEW_TOKENS
            eng = LLMEngine(cfg, dev, max_num_seqs=bs, max_num_batched_tokens=16384, max_model_len=8192 + 16, block_size=16,
                            enforce_eager=False, graph_batch_sizes=tuple(b for b, _ in DECODE))
            eng.runner.bind_weights(weights)
            eng.init_cache(bs * ((ctx + 15) // 16 + 1))
            base = dict(workload="serve", model=model, size=s.name, width=s.width, heads=s.heads, layers=s.layers,
                        kv_bytes_per_token=eng.kv_bytes_per_block() // 16, state_bytes_per_seq=eng.state_bytes() // bs,
                        dtype="bf16", data="synthetic: uniform random ids, random weights")
            for b, n in PREFILL:
                prompts = torch.randint(0, s.vocab, (b, n), generator=gen).tolist()

                def prefill():
                    eng.replay([(str(i), p, [n - 1]) for i, p in enumerate(prompts)], [str(i) for i in range(b)])

                for _ in range(max(warmup, 3)):
                    prefill()
                ms = sorted(_timed(prefill) for _ in range(max(steps, 3)))[max(steps, 3) // 2]
                rows.append(dict(base, case=f"prefill {b}x{n}", ms=round(ms, 3), tokens_per_s=round(b * n / ms * 1e3)))
                emit(json.dumps(rows[-1]))
            for b, n in DECODE:
                prompts = torch.randint(0, s.vocab, (b, n), generator=gen).tolist()
                params = SamplingParams(temperature=1.0, max_tokens=NEW_TOKENS + 1, ignore_eos=True, seed=1)

                def decode():
                    for p in prompts:
                        eng.add_request(None, p, params)
                    while any(q.num_computed < len(q.prompt_ids) for q in eng.scheduler.running) or eng.scheduler.waiting:
                        eng.step()

                    def rest():
                        while eng.has_unfinished_requests():
                            eng.step()
                    return _timed(rest)

                for _ in range(1):
                    decode()
                ms = sorted(decode() for _ in range(max(steps, 3)))[max(steps, 3) // 2]
                rows.append(dict(base, case=f"decode B={b} ctx={n}", ms_per_step=round(ms / NEW_TOKENS, 4),
                                 tokens_per_s=round(b * NEW_TOKENS / ms * 1e3)))
                emit(json.dumps(rows[-1]))
            del eng, weights
            torch.cuda.empty_cache()
    return rows
