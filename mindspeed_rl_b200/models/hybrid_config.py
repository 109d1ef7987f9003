"""Configuration of decoders that are composed layer by layer.

A :class:`HybridConfig` lists its layers one by one: each has a token mixer of some type with its own sizes
and a feed-forward of some kind (or none), and a range of layers may be run several times in a row with the
same weights.  The layer types are small dataclasses in two tables (``MIXERS``, ``FEED_FORWARDS``), so that
another design adds a type without touching the readers of the others.  :meth:`HybridConfig.from_json` reads
the ``config.json`` of a model folder.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch


@dataclass(frozen=True)
class Rotary:
    """Rotary positions on the first ``dims`` entries of a vector, neighbours paired (2i with 2i + 1)."""
    dims: int
    base: float


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Causal soft-max attention whose keys and values are up-projections of one cached latent per token.
    ``dim`` unrotated and ``rot_dim`` rotated query / key entries per head; the rotated key part is shared."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotary
    recurrent = False

    @classmethod
    def from_json(cls, m: dict) -> "LatentAttentionSpec":
        rot = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]))
        out = cls(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                  float(m["scale"]), rot)
        if rot.dims % 2 or rot.dims > out.rot_dim:
            raise ValueError(f"rotary dims {rot.dims} must be even and at most rot_dim ({out.rot_dim})")
        return out


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Gated delta rule with one decay per head and key channel and short convolutions on q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    unit_eps: float = 1e-6
    recurrent = True

    @classmethod
    def from_json(cls, m: dict) -> "ChannelDeltaSpec":
        out = cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        if out.heads % out.kv_heads:
            raise ValueError(f"{out.heads} heads do not divide into {out.kv_heads} key heads")
        return out


@dataclass(frozen=True)
class GluSpec:
    """Gated feed-forward ``W_down(act(W_gate h, W_up h))``; see ``ops.glu_fwd`` for the activations."""
    ff: int
    act: str
    limit: float = 0.0
    alpha: float = 1.0

    @classmethod
    def from_json(cls, m: dict) -> "GluSpec":
        return cls(int(m["ff"]), "gelu_tanh")


@dataclass(frozen=True)
class TableMoESpec:
    """Experts chosen by a table over token ids with equal weights, plus an optional gated shared expert."""
    experts: int
    top: int
    expert: GluSpec
    shared: Optional[GluSpec] = None

    @classmethod
    def from_json(cls, m: dict) -> "TableMoESpec":
        def clamped(d):
            return GluSpec(int(d["ff"]), "clamped_swish", limit=float(d["limit"]), alpha=1.702)

        r = m["router"]
        return cls(int(r["experts"]), int(r["top"]), clamped(m["expert"]),
                   clamped(m["shared"]) if m.get("shared") else None)


MIXERS = {"latent_attention": LatentAttentionSpec, "channel_delta": ChannelDeltaSpec}
FEED_FORWARDS = {"dense": GluSpec, "moe": TableMoESpec}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Any
    mlp: Any = None


@dataclass
class HybridConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    layers: List[LayerSpec]
    norm_epsilon: float
    norm_offset: float = 1.0             # the stored weight of a pre-norm is an offset from this value
    embedding_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    params_dtype: torch.dtype = torch.bfloat16
    extra: Dict[str, Any] = field(default_factory=dict)
    is_hybrid = True

    def __post_init__(self):
        if self.loop is not None:
            a, b, n = self.loop
            if not (0 <= a <= b <= len(self.layers)) or n < 1:
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")

    # ---- what a sequence runs through ----------------------------------------------------------
    @property
    def run_order(self) -> List[int]:
        """Layer index of every layer run; a looped layer appears once per pass."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return [*range(a), *(list(range(a, b)) * times), *range(b, n)]

    @property
    def num_layers(self) -> int:
        return len(self.run_order)

    @property
    def is_recurrent(self) -> bool:
        return any(l.mixer.recurrent for l in self.layers)

    @property
    def is_moe(self) -> bool:
        return any(isinstance(l.mlp, TableMoESpec) for l in self.layers)

    @classmethod
    def from_json(cls, cfg: dict, dtype: torch.dtype = torch.bfloat16) -> "HybridConfig":
        layers = []
        for i, l in enumerate(cfg["layers"]):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            mlp = l.get("mlp")
            if mlp is not None and mlp["kind"] not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerSpec(l["type"], MIXERS[l["type"]].from_json(l["mixer"]),
                                    None if mlp is None else FEED_FORWARDS[mlp["kind"]].from_json(mlp)))
        lp = cfg.get("loop")
        return cls(architecture=cfg["architecture"], vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                   layers=layers, norm_epsilon=float(cfg["norm"]["eps"]),
                   embedding_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)),
                   loop=None if not lp else (int(lp["start"]), int(lp["stop"]), int(lp["times"])),
                   params_dtype=dtype)
