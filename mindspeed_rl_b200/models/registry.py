"""Model registry: the ``config.json`` of a model folder -> configuration and rollout weights.

A family is registered under the architecture name its configuration carries (``architecture``, or the first of
Hugging Face's ``architectures``).  ``load_model`` is what the command lines use: it reads a folder and returns
``(config, weights)`` ready for ``LLMEngine`` / ``ModelRunner.bind_weights``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional, Tuple

import torch

from .hybrid_config import HybridConfig
from .transformer_config import TransformerConfig


@dataclass(frozen=True)
class ModelFamily:
    config: Callable[[dict, torch.dtype], Any]                                  # (config.json, dtype) -> config
    weights: Callable[[Any, Dict[str, torch.Tensor], Any], Any]                 # (config, tensors, device) -> weights
    kernels: Optional[str] = None        # group of kernels that serves the family (``csrc.build.GROUPS``; None: all)


_FAMILIES: Dict[str, ModelFamily] = {}


def register(name: str, family: ModelFamily) -> None:
    _FAMILIES[name] = family


def families() -> Tuple[str, ...]:
    return tuple(sorted(_FAMILIES))


def architecture_of(cfg: dict) -> str:
    name = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]
    if name not in _FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; registered: {', '.join(families())}")
    return name


def read_config(path: str, dtype: torch.dtype = torch.bfloat16):
    with open(os.path.join(path, "config.json")) as fh:
        raw = json.load(fh)
    return _FAMILIES[architecture_of(raw)].config(raw, dtype), raw


def use_kernels_of(path: str) -> None:
    """Serve this process from the kernels that the model of a folder needs, compiling them if they are not there."""
    from ..ops import _lib

    with open(os.path.join(path, "config.json")) as fh:
        group = _FAMILIES[architecture_of(json.load(fh))].kernels
    if group is not None:
        _lib.use_group(group)


def load_model(path: str, dtype: torch.dtype = torch.bfloat16, device="cuda"):
    """``(config, rollout weights)`` of a model folder (config.json and safetensors files)."""
    from ..checkpoint.convert import load_hf_state

    cfg, raw = read_config(path, dtype)
    return cfg, _FAMILIES[architecture_of(raw)].weights(cfg, load_hf_state(path), device)


# ---- families ---------------------------------------------------------------------------------------
def _hybrid_weights(cfg, state, device):
    from ..rollout.hybrid_weights import build_hybrid_weights

    return build_hybrid_weights(cfg, state, device)


def _decoder_config(raw: dict, dtype: torch.dtype) -> TransformerConfig:
    """Hugging Face configuration of the Qwen2 / Qwen2.5 / Qwen3 / Qwen3-MoE decoders."""
    if raw.get("rope_scaling"):
        raise ValueError("rope_scaling of a Hugging Face configuration is not read here")
    arch = raw["architectures"][0]
    qwen3 = arch.startswith("Qwen3")
    moe = raw.get("num_experts")
    return TransformerConfig(
        num_layers=raw["num_hidden_layers"], hidden_size=raw["hidden_size"], ffn_hidden_size=raw["intermediate_size"],
        num_attention_heads=raw["num_attention_heads"],
        num_query_groups=raw.get("num_key_value_heads", raw["num_attention_heads"]), vocab_size=raw["vocab_size"],
        kv_channels=raw.get("head_dim"), norm_epsilon=raw.get("rms_norm_eps", 1e-6),
        rotary_base=float(raw.get("rope_theta", 10000.0)), max_position_embeddings=raw.get("max_position_embeddings", 32768),
        add_qkv_bias=not qwen3, qk_layernorm=qwen3,
        untie_embeddings_and_output_weights=not raw.get("tie_word_embeddings", False), num_experts=moe,
        moe_router_topk=raw.get("num_experts_per_tok", 2), moe_ffn_hidden_size=raw.get("moe_intermediate_size"),
        norm_topk_prob=bool(raw.get("norm_topk_prob", False)), params_dtype=dtype)


def _decoder_weights(cfg, state, device):
    from ..checkpoint.convert import hf_to_mcore
    from ..reshard.alias import alias_rollout_weights
    from .gpt import GPTModel

    model = GPTModel(cfg, device=device)
    params = dict(model.named_parameters())
    tensors = hf_to_mcore(state, cfg)[(0, 0, 0)]
    missing = sorted(set(params) - set(tensors))
    if missing:
        raise ValueError(f"checkpoint lacks {missing[:8]}")
    with torch.no_grad():
        for n, p in params.items():
            p.copy_(tensors[n].reshape(p.shape))
    return alias_rollout_weights(model)


register("Pumotar", ModelFamily(HybridConfig.from_json, _hybrid_weights, "pumotar"))
register("Sunatar", ModelFamily(HybridConfig.from_json, _hybrid_weights, "sunatar"))
register("Gapevik", ModelFamily(HybridConfig.from_json, _hybrid_weights, "gapevik"))
register("Lunelorn", ModelFamily(HybridConfig.from_json, _hybrid_weights, "lunelorn"))
for _name in ("Qwen2ForCausalLM", "Qwen3ForCausalLM", "Qwen3MoeForCausalLM"):
    register(_name, ModelFamily(_decoder_config, _decoder_weights))
