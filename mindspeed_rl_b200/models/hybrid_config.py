"""Configuration of decoders that are composed layer by layer.

A :class:`HybridConfig` lists its layers one by one: each has a token mixer of some type with its own sizes
and a feed-forward of some kind (or none), and a range of layers may be run several times in a row with the
same weights.  The layer types are small dataclasses; a :class:`Design` says which of them an architecture has
under which names, its norm, how a layer adds its two sublayers and where its LM head is (``DESIGNS``), so that
another design adds a type without touching the readers of the others.  :meth:`HybridConfig.from_json` reads
the ``config.json`` of a model folder.

A mixer spec tells the cache what a sequence carries for it: ``paged_rows(dtype)``, shapes of one token's rows in
paged memory by name, and ``slot_state(dtype)``, shapes and types of the state of one sequence by name.  Specs with
paged rows have ``keys``, the range of earlier tokens that a token sees (:data:`KeyRange`).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, NamedTuple, Optional, Tuple, Union

import torch

from ..ops.latent import pad16


def padded_heads(dq: int, dv: int, dtype: torch.dtype) -> Tuple[int, int]:
    """Query / key and value head sizes as they are stored: bf16 heads are padded to a pair that the tensor-core
    attention kernels serve; other sizes and fp32 (CUDA cores) to whole 16-byte vectors."""
    if dtype != torch.bfloat16 or dv > 128 or dq > 192:
        unit = 16 // dtype.itemsize
        return -(-dq // unit) * unit, -(-dv // unit) * unit
    vp = 64 if max(dq, dv) <= 64 else 128
    return (192 if dq > 128 else vp), vp


class Chunk(NamedTuple):
    """A token sees the earlier tokens of its own chunk; chunks of ``size`` tokens count from the sequence's start."""
    size: int

    @classmethod
    def of(cls, mask: Optional[dict]) -> Optional["Chunk"]:
        return None if not mask else cls(_positive(mask["size"], "chunk"))


KeyRange = Union[None, int, Chunk]       # all earlier tokens, the last n up to the token itself, or its chunk


def first_key(keys: KeyRange, pos):
    """First position that the token at ``pos`` (an integer or an array of them) sees."""
    if keys is None:
        return pos * 0
    if isinstance(keys, Chunk):
        return pos // keys.size * keys.size
    return (pos - keys + 1) * (pos >= keys)


def _positive(n, what: str) -> int:
    if int(n) < 1:
        raise ValueError(f"a {what} of {n} tokens sees nothing")
    return int(n)


def _window_of(mask: Optional[dict]) -> Optional[int]:
    return None if not mask else _positive(mask["size"], "window")


def _check_heads(spec):
    if spec.heads % spec.kv_heads:
        raise ValueError(f"{spec.heads} heads do not divide into {spec.kv_heads} key heads")
    return spec


def _check_rotary(rot: "Rotary", limit: int, name: str) -> None:
    if rot.dims % 2 or rot.dims > limit:
        raise ValueError(f"rotary dims {rot.dims} must be even and at most {name} ({limit})")


@dataclass(frozen=True)
class WavelengthScaling:
    """Frequencies of wavelengths above ``original / low`` are divided by ``factor``, those below
    ``original / high`` kept, and the ones between are blended linearly in ``original / wavelength``."""
    factor: float
    low: float
    high: float
    original: float

    def scaled(self, f: float) -> float:
        turns = self.original * f / (2.0 * math.pi)          # whole turns over the original length
        if turns > self.high:
            return f
        if turns < self.low:
            return f / self.factor
        s = (turns - self.low) / (self.high - self.low)
        return (1.0 - s) * f / self.factor + s * f


@dataclass(frozen=True)
class Rotary:
    """Rotary positions on the first ``dims`` entries of a vector: neighbours paired (2i with 2i + 1), or
    with ``halves`` entry i with entry i + dims / 2."""
    dims: int
    base: float
    halves: bool = False
    scaling: Optional[WavelengthScaling] = None

    def frequencies(self) -> Tuple[float, ...]:
        fs = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        return tuple(self.scaling.scaled(f) if self.scaling is not None else f for f in fs)


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Causal soft-max attention whose keys and values are up-projections of one cached latent per token.
    ``dim`` unrotated and ``rot_dim`` rotated query / key entries per head; the rotated key part is shared.
    ``q_rank``: queries go through a normed latent of their own; ``sink``: a learned number per head joins the soft-max
    sum; ``head_gate``: a sigmoid per head scales the head's output."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotary
    q_rank: Optional[int] = None
    window: Optional[int] = None
    sink: bool = False
    head_gate: bool = False

    @property
    def keys(self) -> KeyRange:
        return self.window

    def paged_rows(self, dtype) -> Dict[str, Tuple[int, ...]]:
        return {"latent": (pad16(self.kv_rank) + pad16(self.rot_dim),)}

    def slot_state(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict, halves: bool = False, **options) -> "LatentAttentionSpec":
        rot = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]), halves)
        out = cls(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                  float(m["scale"]), rot, **options)
        _check_rotary(rot, out.rot_dim, "rot_dim")
        return out

    @classmethod
    def gated_from_json(cls, m: dict) -> "LatentAttentionSpec":
        """With a query latent, half-split rotation, a window, a sink and a gate per head."""
        return cls.from_json(m, halves=True, q_rank=int(m["q_rank"]), window=_window_of(m.get("mask")), sink=True, head_gate=True)


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Gated delta rule with one decay per head and key channel and short convolutions on q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    unit_eps: float = 1e-6

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def paged_rows(self, dtype) -> dict:
        return {}

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return {"ring": ((self.conv, self.channels), dtype), "state": ((self.heads, self.dim, self.vdim), torch.float32)}

    @classmethod
    def from_json(cls, m: dict) -> "ChannelDeltaSpec":
        return _check_heads(cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"])))


@dataclass(frozen=True)
class HeadDeltaSpec(ChannelDeltaSpec):
    """The delta rule with one decay per head, projected without a bottleneck, and a silu output gate."""


@dataclass(frozen=True)
class WindowAttentionSpec:
    """Soft-max attention of grouped heads over the last ``window`` tokens (None: all), with biased projections, an
    RMS norm over the whole query and the whole key projection, partial rotation, and values mixed with those of
    the first layer that has ``value_mix``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotary
    window: Optional[int] = None
    value_mix: bool = False

    @property
    def keys(self) -> KeyRange:
        return self.window

    def padded(self, dtype) -> Tuple[int, int]:
        return padded_heads(self.dim, self.vdim, dtype)

    def paged_rows(self, dtype) -> Dict[str, Tuple[int, ...]]:
        qp, vp = self.padded(dtype)
        return {"k": (self.kv_heads, qp), "v": (self.kv_heads, vp)}

    def slot_state(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict) -> "WindowAttentionSpec":
        r, sc, mask = m["rot"], m["rot"].get("scaling"), m.get("mask")
        rot = Rotary(int(r["dims"]), float(r["base"]), halves=True,
                     scaling=None if not sc else WavelengthScaling(float(sc["factor"]), float(sc["low"]), float(sc["high"]),
                                                                   float(sc["original"])))
        out = _check_heads(cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), rot,
                               _window_of(mask), bool(m.get("v_mix", False))))
        _check_rotary(rot, out.dim, "dim")
        return out


@dataclass(frozen=True)
class ConvAttentionSpec:
    """Soft-max attention of grouped heads with short convolutions on q, k and v (carried like a recurrent state), an RMS
    norm per query and key head, partial interleaved rotation, soft-capped scores (0: not capped), a key range, and a
    sigmoid gate per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    rot: Rotary
    softcap: float = 0.0
    keys: KeyRange = None

    @property
    def channels(self) -> int:
        return (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim

    def padded(self, dtype) -> Tuple[int, int]:
        return padded_heads(self.dim, self.vdim, dtype)

    def paged_rows(self, dtype) -> Dict[str, Tuple[int, ...]]:
        qp, vp = self.padded(dtype)
        return {"k": (self.kv_heads, qp), "v": (self.kv_heads, vp)}

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return {"ring": ((self.conv, self.channels), dtype)}

    @classmethod
    def from_json(cls, m: dict) -> "ConvAttentionSpec":
        rot = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]))
        out = _check_heads(cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]),
                               float(m["scale"]), rot, float(m.get("softcap") or 0.0), Chunk.of(m.get("mask"))))
        _check_rotary(rot, out.dim, "dim")
        if out.softcap < 0.0:
            raise ValueError(f"scores cannot be capped at {out.softcap}")
        return out


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Matrix memory with exponential gates, stabilised by a running maximum that starts at zero; gate logits are
    soft-capped at ``gate_cap``.  Heads are stored in multiples of 16."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    floor: float = 1e-6                  # added to the normaliser

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        f32, dp, vp = torch.float32, pad16(self.dim), pad16(self.vdim)
        return {"memory": ((self.heads, dp, vp), f32), "norm": ((self.heads, dp), f32), "peak": ((self.heads,), f32)}

    def paged_rows(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict) -> "MatrixMemorySpec":
        return cls(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))


@dataclass(frozen=True)
class RetentionSpec:
    """Linear attention over a matrix state whose heads forget at constant rates.  Heads are stored in multiples of 16."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return {"memory": ((self.heads, pad16(self.dim), pad16(self.vdim)), torch.float32)}

    def paged_rows(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict) -> "RetentionSpec":
        out = cls(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(x) for x in m["decay"]))
        if len(out.decay) != out.heads or not all(0.0 <= x <= 1.0 for x in out.decay):
            raise ValueError(f"{out.heads} heads need as many decays between 0 and 1, got {out.decay}")
        return out


@dataclass(frozen=True)
class TurnedAttentionSpec:
    """Soft-max attention of grouped heads over all earlier tokens, with partial half-split rotation of queries and keys.
    Values are normed per head and turned by their own position over all their entries; an output is turned back by the
    query's."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotary
    keys: KeyRange = None

    @property
    def value_rot(self) -> Rotary:
        return Rotary(self.vdim, self.rot.base, halves=True)

    def padded(self, dtype) -> Tuple[int, int]:
        return padded_heads(self.dim, self.vdim, dtype)

    def paged_rows(self, dtype) -> Dict[str, Tuple[int, ...]]:
        qp, vp = self.padded(dtype)
        return {"k": (self.kv_heads, qp), "v": (self.kv_heads, vp)}

    def slot_state(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict) -> "TurnedAttentionSpec":
        out = _check_heads(cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                               Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]), halves=True)))
        _check_rotary(out.rot, out.dim, "dim")
        _check_rotary(out.value_rot, out.vdim, "vdim")
        return out


@dataclass(frozen=True)
class MinGRUSpec:
    """An element-wise recurrence; its gate and its candidate are functions of the token, not of the state."""
    width: int

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return {"state": ((self.width,), torch.float32)}

    def paged_rows(self, dtype) -> dict:
        return {}


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and a gated recurrence side by side on the same input; their outputs are scaled and added."""
    left: TurnedAttentionSpec
    right: MinGRUSpec
    left_scale: float
    right_scale: float

    @property
    def keys(self) -> KeyRange:
        return self.left.keys

    def paged_rows(self, dtype) -> Dict[str, Tuple[int, ...]]:
        return self.left.paged_rows(dtype)

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return self.right.slot_state(dtype)

    @classmethod
    def from_json(cls, m: dict) -> "ParallelSpec":
        return cls(TurnedAttentionSpec.from_json(m["left"]), MinGRUSpec(int(m["right"]["width"])), float(m["left_scale"]),
                   float(m["right_scale"]))


@dataclass(frozen=True)
class WKVSpec:
    """Linear attention whose state decays per head and key channel by what the token says, with a bonus for the current
    token.  Its projections read mixes of the token's input and the one before, which is carried (``model_width`` entries)."""
    heads: int
    dim: int
    model_width: int

    def slot_state(self, dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        return {"last": ((self.model_width,), torch.float32), "state": ((self.heads, self.dim, self.dim), torch.float32)}

    def paged_rows(self, dtype) -> dict:
        return {}

    @classmethod
    def from_json(cls, m: dict) -> "WKVSpec":
        return cls(int(m["heads"]), int(m["dim"]), int(m["model_width"]))


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


@dataclass(frozen=True)
class ScoredMoESpec:
    """Experts of the largest router scores (sigmoid of 32-bit logits), each run on its input times its score, plus
    an optional shared expert."""
    experts: int
    top: int
    expert: GluSpec
    shared: Optional[GluSpec] = None

    @classmethod
    def from_json(cls, m: dict) -> "ScoredMoESpec":
        r, sh = m["router"], m.get("shared")
        out = cls(int(r["experts"]), int(r["top"]), GluSpec(int(m["expert"]["ff"]), "silu"),
                  GluSpec(int(sh["ff"]), "silu") if sh else None)
        if not 0 < out.top <= out.experts:
            raise ValueError(f"top {out.top} of {out.experts} experts")
        return out


@dataclass(frozen=True)
class SoftmaxMoESpec:
    """Experts of the largest corrected scores: the score is a soft-max (32-bit) over all router outputs, the correction a
    stored number per output that counts for the choice only.  Outputs past ``experts`` are ``identity`` experts, which
    give back their input.  A chosen expert's output is weighted by its score."""
    experts: int
    top: int
    expert: GluSpec
    identity: int = 0
    shared: Optional[GluSpec] = None

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    @classmethod
    def from_json(cls, m: dict) -> "SoftmaxMoESpec":
        r = m["router"]
        out = cls(int(r["experts"]), int(r["top"]), GluSpec(int(m["expert"]["ff"]), "silu"), int(r.get("identity") or 0))
        if not 0 < out.top <= out.outputs:
            raise ValueError(f"top {out.top} of {out.outputs} experts")
        return out


@dataclass(frozen=True)
class ChosenMoESpec:
    """Experts of the largest router logits (32-bit), their outputs weighted by a soft-max over the chosen logits only."""
    experts: int
    top: int
    expert: GluSpec
    shared: Optional[GluSpec] = None

    @classmethod
    def from_json(cls, m: dict) -> "ChosenMoESpec":
        r = m["router"]
        out = cls(int(r["experts"]), int(r["top"]), GluSpec(int(m["expert"]["ff"]), "silu"))
        if not 0 < out.top <= out.experts:
            raise ValueError(f"top {out.top} of {out.experts} experts")
        return out


@dataclass(frozen=True)
class Design:
    """What the layers of one architecture have in common.  ``mixers`` and ``feed_forwards``: readers of a layer's entry
    by its type.  ``parallel``: both sublayers read one norm and are added together; ``post_norm``: the sublayers read the
    residual itself and their outputs are normed before they are added; ``sandwich``: a norm before and one after each
    sublayer; otherwise the feed-forward reads a second norm of the sum.  ``embed_norm``: token embeddings are normed.
    ``loop_input``: every pass of a loop adds a vector of its own before it runs, and passes after the first what the
    embedding gave.  ``centered``: norms subtract the mean.  ``norm_offset``: the stored weight of a norm is an offset from
    this value.  Readers of mixers find the model's width under ``model_width``."""
    mixers: Dict[str, Callable[[dict], Any]]
    feed_forwards: Dict[str, Callable[[dict], Any]]
    parallel: bool = False
    post_norm: bool = False
    sandwich: bool = False
    embed_norm: bool = False
    loop_input: bool = False
    centered: bool = False
    norm_offset: float = 0.0
    tied_head: bool = True


DESIGNS = {
    "Pumotar": Design({"latent_attention": LatentAttentionSpec.from_json, "channel_delta": ChannelDeltaSpec.from_json},
                      {"dense": GluSpec.from_json, "moe": TableMoESpec.from_json}, norm_offset=1.0),
    "Sunatar": Design({"attention": WindowAttentionSpec.from_json, "mlstm": MatrixMemorySpec.from_json},
                      {"moe": ScoredMoESpec.from_json}, parallel=True, centered=True, tied_head=False),
    "Gapevik": Design({"attention": ConvAttentionSpec.from_json, "latent_attention": LatentAttentionSpec.gated_from_json,
                       "delta": HeadDeltaSpec.from_json}, {"moe": SoftmaxMoESpec.from_json}, post_norm=True),
    "Lunelorn": Design({"retention": RetentionSpec.from_json, "parallel": ParallelSpec.from_json, "wkv": WKVSpec.from_json},
                       {"moe": ChosenMoESpec.from_json}, sandwich=True, embed_norm=True, loop_input=True, tied_head=False),
}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Any
    mlp: Any = None
    weights_of: Optional[int] = None     # the layer whose tensors this one uses (None: its own)


@dataclass
class HybridConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    layers: List[LayerSpec]
    norm_epsilon: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0                       # factor on what a sublayer adds (post-norm designs)
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    token_side: Optional[int] = None                 # entries of a token's row per layer (designs with token inputs)
    logit_softcap: float = 0.0                       # logits <- cap tanh(logits / cap); 0: as they are
    params_dtype: torch.dtype = torch.bfloat16
    extra: Dict[str, Any] = field(default_factory=dict)
    is_hybrid = True

    def __post_init__(self):
        if self.loop is not None:
            a, b, n = self.loop
            if not (0 <= a <= b <= len(self.layers)) or n < 1:
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")
        for i in range(len(self.layers)):
            self.owner(i)
        mixed = {l.mixer.kv_heads * l.mixer.vdim for l in self.layers if getattr(l.mixer, "value_mix", False)}
        if len(mixed) > 1:
            raise ValueError(f"layers that mix values with the first one's have different value sizes: {sorted(mixed)}")

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        j, seen = i, set()
        while self.layers[j].weights_of is not None:
            seen.add(j)
            j = self.layers[j].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ValueError(f"layer {i} uses the tensors of layer {j}, which has none")
        mine, other = self.layers[i], self.layers[j]
        if (mine.type, mine.mixer, mine.mlp) != (other.type, other.mixer, other.mlp):
            raise ValueError(f"layer {i} uses the tensors of layer {j} but differs from it")
        return j

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
    def pass_starts(self) -> Dict[int, int]:
        """Layer run -> number of the pass of the loop that begins with it."""
        if self.loop is None:
            return {}
        a, b, times = self.loop
        return {a + p * (b - a): p for p in range(times)} if b > a else {}

    @property
    def num_layers(self) -> int:
        return len(self.run_order)

    @property
    def is_recurrent(self) -> bool:
        """Sequences carry state besides paged rows."""
        return any(l.mixer.slot_state(self.params_dtype) for l in self.layers)

    @property
    def is_moe(self) -> bool:
        return any(isinstance(l.mlp, (TableMoESpec, ScoredMoESpec, SoftmaxMoESpec, ChosenMoESpec)) for l in self.layers)

    @property
    def windows(self) -> Tuple[KeyRange, ...]:
        """Distinct key ranges of the attention layers."""
        return tuple({l.mixer.keys: None for l in self.layers if l.mixer.paged_rows(self.params_dtype)})

    @classmethod
    def from_json(cls, cfg: dict, dtype: torch.dtype = torch.bfloat16) -> "HybridConfig":
        layers, design = [], DESIGNS[cfg["architecture"]]
        for i, l in enumerate(cfg["layers"]):
            if l["type"] not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            mlp = l.get("mlp")
            if mlp is not None and mlp["kind"] not in design.feed_forwards:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            of = l.get("weights_of")
            layers.append(LayerSpec(l["type"], design.mixers[l["type"]]({"model_width": int(cfg["width"]), **l["mixer"]}),
                                    None if mlp is None else design.feed_forwards[mlp["kind"]](mlp),
                                    None if of is None else int(of)))
        lp, side = cfg.get("loop"), cfg.get("token_side")
        return cls(architecture=cfg["architecture"], vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                   layers=layers, norm_epsilon=float(cfg["norm"]["eps"]),
                   embedding_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(cfg.get("residual_mult", 1.0)),
                   loop=None if not lp else (int(lp["start"]), int(lp["stop"]), int(lp["times"])),
                   token_side=int(side["dim"]) if side else None, logit_softcap=float(cfg.get("logit_softcap") or 0.0),
                   params_dtype=dtype)
