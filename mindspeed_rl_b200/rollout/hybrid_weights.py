"""Weights of a layer-by-layer decoder, bound by the model runner in place of ``RolloutWeights``."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import torch

from ..models.hybrid_config import HybridConfig
from ..ops import TokenSide
from .feed_forward import build_feed_forward
from .mixers import MIXERS, _pad8, _pad_cols, _pad_rows


@dataclass
class HybridLayer:
    norm1: torch.Tensor                 # fp32
    mixer: Any
    norm2: Optional[torch.Tensor] = None
    ff: Any = None
    post1: Optional[torch.Tensor] = None      # norms of the sublayers' outputs (sandwich designs)
    post2: Optional[torch.Tensor] = None
    side: Optional[TokenSide] = None          # the layer's input from the token itself, its norm
    side_norm: Optional[torch.Tensor] = None


@dataclass
class HybridWeights:
    embed: torch.Tensor
    layers: List[HybridLayer]
    final_norm: torch.Tensor
    lm_head: torch.Tensor
    embed_norm: Optional[torch.Tensor] = None
    loop_step: Optional[torch.Tensor] = None  # [passes, W] fp32

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
    ``l<i>.norm2`` and ``head`` where the design has them; else the LM head is the embedding table; ``embed.norm``,
    ``loop.step``, ``l<i>.norm1b``, ``l<i>.norm2b``, ``side.embed`` and ``l<i>.side.*`` likewise).  A layer that uses another
    one's tensors has none, and shares its objects.  A name that no layer asks for is an error."""
    dt = cfg.params_dtype
    used = {"embed", "final.norm"}

    def f32(name):
        used.add(name)
        return state[name].to(device=device, dtype=torch.float32).contiguous()

    side_rows = None
    if cfg.token_side is not None:
        used.add("side.embed")
        side_rows = state["side.embed"].to(device=device, dtype=dt).contiguous()
        if tuple(side_rows.shape) != (cfg.vocab_size, len(cfg.layers) * cfg.token_side):
            raise ValueError(f"side.embed {tuple(side_rows.shape)} does not fit {cfg.vocab_size} x {len(cfg.layers)} layers of "
                             f"{cfg.token_side}")

    def token_side(i):
        n, pad = cfg.token_side, _pad8(cfg.token_side)
        w = _Taken(state, f"l{i}.side.", used)
        gate, proj = (x.to(device=device, dtype=dt).contiguous() for x in (_pad_rows(w["gate"], pad), _pad_cols(w["proj"], pad)))
        return TokenSide(gate, proj, side_rows, i * n, n)

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
        if cfg.design.sandwich:
            layer.post1 = f32(p + "norm1b")
            layer.post2 = f32(p + "norm2b") if spec.mlp is not None else None
        if side_rows is not None:
            layer.side, layer.side_norm = token_side(i), f32(p + "side.norm")
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
    embed_norm = f32("embed.norm") if cfg.design.embed_norm else None
    loop_step = f32("loop.step") if cfg.design.loop_input and cfg.loop is not None else None
    if loop_step is not None and tuple(loop_step.shape) != (cfg.loop[2], cfg.hidden_size):
        raise ValueError(f"loop.step {tuple(loop_step.shape)} does not fit {cfg.loop[2]} passes of {cfg.hidden_size}")
    extra = sorted(set(state) - used)
    # a layer without a feed-forward may still carry unused norms of one
    extra = [n for n in extra if not n.endswith((".norm2", ".norm2b"))]
    if extra:
        raise ValueError(f"tensors without a place in the model: {extra[:8]}")
    return HybridWeights(embed, layers, f32("final.norm"), head, embed_norm, loop_step)
