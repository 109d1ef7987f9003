"""Weights of a layer-by-layer decoder, bound by the model runner in place of ``RolloutWeights``."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import torch

from ..models.hybrid_config import HybridConfig
from .feed_forward import build_feed_forward
from .mixers import MIXERS


@dataclass
class HybridLayer:
    norm1: torch.Tensor                 # fp32
    mixer: Any
    norm2: Optional[torch.Tensor] = None
    ff: Any = None


@dataclass
class HybridWeights:
    embed: torch.Tensor
    layers: List[HybridLayer]
    final_norm: torch.Tensor
    lm_head: torch.Tensor

    def signature(self):
        """Addresses of what captured graphs read."""
        return (self.embed.data_ptr(), self.lm_head.data_ptr(), tuple(l.mixer.w_in.data_ptr() for l in self.layers))


class _Taken(dict):
    """Name -> tensor view of a checkpoint below a prefix; remembers which names were read."""

    def __init__(self, state: Dict[str, torch.Tensor], prefix: str, used: set):
        super().__init__({k[len(prefix):]: v for k, v in state.items() if k.startswith(prefix)})
        self._prefix, self._used = prefix, used

    def __getitem__(self, k):
        self._used.add(self._prefix + k)
        return super().__getitem__(k)


def build_hybrid_weights(cfg: HybridConfig, state: Dict[str, torch.Tensor], device) -> HybridWeights:
    """``state``: checkpoint tensors (``embed``, ``final.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, and
    ``l<i>.norm2`` and ``head`` where the design has them; else the LM head is the embedding table).  A layer that uses
    another one's tensors has none, and shares its objects.  A name that no layer asks for is an error."""
    dt = cfg.params_dtype
    used = {"embed", "final.norm"}

    def f32(name):
        used.add(name)
        return state[name].to(device=device, dtype=torch.float32).contiguous()

    layers: List[Optional[HybridLayer]] = [None] * len(cfg.layers)
    for i, spec in enumerate(cfg.layers):
        if cfg.owner(i) != i:
            continue
        p = f"l{i}."
        layer = HybridLayer(f32(p + "norm1"),
                            MIXERS[type(spec.mixer)](spec.mixer, _Taken(state, p + "mix.", used), cfg.norm_epsilon, dt, device))
        if spec.mlp is not None:
            if not cfg.design.parallel:
                layer.norm2 = f32(p + "norm2")
            layer.ff = build_feed_forward(spec.mlp, _Taken(state, p + "mlp.", used), dt, device)
        layers[i] = layer
    layers = [layers[cfg.owner(i)] for i in range(len(layers))]

    def table(name):
        used.add(name)
        t = state[name].to(device=device, dtype=dt).contiguous()
        if tuple(t.shape) != (cfg.vocab_size, cfg.hidden_size):
            raise ValueError(f"{name} {tuple(t.shape)} does not fit {cfg.vocab_size} x {cfg.hidden_size}")
        return t

    embed = table("embed")
    head = embed if cfg.design.tied_head else table("head")
    extra = sorted(set(state) - used)
    # a layer without a feed-forward may still carry an unused second norm
    extra = [n for n in extra if not n.endswith(".norm2")]
    if extra:
        raise ValueError(f"tensors without a place in the model: {extra[:8]}")
    return HybridWeights(embed, layers, f32("final.norm"), head)
