"""Matrix memory with exponential gates over state slots: prompt portions and decode steps.

Per head, with log gates ``i = cap tanh(z_i / cap)`` and ``f = log sigmoid(cap tanh(z_f / cap))`` and a running maximum m::

    m' = max(f + m, i)
    S' = exp(f + m - m') S + exp(i - m') k v^T,   n' likewise with k alone
    o  = S'^T q / (max(|n' . q|, exp(-m')) + floor),    y = o / rms(o) * norm * sigmoid(gate)

``MemoryWeights.decay`` puts a constant decay per head in place of the gates: linear attention without a denominator::

    S' = decay S + k v^T,   o = S'^T q

``MemoryLayout.silu_gate``: the output gate is ``silu(gate)``.

A sequence starts with S, n and m zero.  ``slots`` holds the state of all sequences: ``memory [slots, H, dim, vdim]``,
``norm [slots, H, dim]`` and ``peak [slots, H]``, all fp32 (with ``decay`` the memory alone); a sequence's first token
ignores what its slot holds.  CUDA path: ``csrc/matrix_memory.cu``, ``csrc/matrix_memory_tcgen05.cu``; CPU tensors run the PyTorch formulation.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Optional

import torch
import torch.nn.functional as F

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .elementwise import _workspace
from .gemm import _status_word
from .residual import _is_f32

CHUNK = 128            # tokens that the chunked prompt kernels take at a time


@dataclass(frozen=True)
class MemoryLayout:
    """Stored sizes of a layer (``dim`` and ``vdim`` with their padding, ``rms_dim`` entries of a value head count in its
    root mean square) and the columns of its sections in the fused projection row."""
    heads: int
    dim: int
    vdim: int
    rms_dim: int
    q_col: int
    k_col: int
    v_col: int
    g_col: int
    scale: float
    cap: float = 1.0
    floor: float = 1e-6
    silu_gate: bool = False

    def ints(self):
        return (ctypes.c_int * 9)(self.heads, self.dim, self.vdim, self.rms_dim, self.q_col, self.k_col, self.v_col, self.g_col,
                                  self.silu_gate)

    def floats(self, eps: float):
        return (ctypes.c_float * 4)(self.scale, self.cap, self.floor, eps)


@dataclass
class MemoryWeights:
    bias: Optional[torch.Tensor]            # [2 * heads] fp32: input gates, forget gates
    norm: torch.Tensor                      # [heads * vdim] fp32
    decay: Optional[torch.Tensor] = None    # [2 * heads] fp32: decays, their logarithms


def constant_decay(decay) -> torch.Tensor:
    """``MemoryWeights.decay`` of the given numbers in ``[0, 1]`` (a decay of zero is one too small to leave a trace)."""
    d = torch.tensor(list(decay), dtype=torch.float64)
    return torch.cat([d, d.clamp(min=1e-43).log()]).float()


def _retain(q, k, v, lay: MemoryLayout, decay: torch.Tensor, s: torch.Tensor) -> torch.Tensor:
    """One sequence of linear attention in fp32; ``s`` is updated in place."""
    o = torch.empty_like(v)
    for x in range(q.shape[0]):
        s.mul_(decay[:lay.heads, None, None]).add_(k[x][:, :, None] * v[x][:, None])
        o[x] = torch.einsum("hdv,hd->hv", s, q[x] * lay.scale)
    return o


def _gated(q, k, v, z, lay: MemoryLayout, w: MemoryWeights, s, n, m) -> torch.Tensor:
    t, hn = q.shape[:2]
    gates = lay.cap * torch.tanh((z + w.bias) / lay.cap)
    gi, gf = gates[:, :hn], F.logsigmoid(gates[:, hn:])
    o = torch.empty(t, hn, lay.vdim)
    for x in range(t):
        top = torch.maximum(gf[x] + m, gi[x])
        keep, take = torch.exp(gf[x] + m - top), torch.exp(gi[x] - top)
        s.mul_(keep[:, None, None]).add_(take[:, None, None] * k[x][:, :, None] * v[x][:, None])
        n.mul_(keep[:, None]).add_(take[:, None] * k[x])
        m.copy_(top)
        qx = q[x] * lay.scale
        den = torch.maximum((n * qx).sum(-1).abs(), torch.exp(-m)) + lay.floor
        o[x] = torch.einsum("hdv,hd->hv", s, qx) / den[:, None]
    return o


def _recur(proj, z, lay: MemoryLayout, w: MemoryWeights, s, n, m, eps):
    """One sequence in fp32; ``s``, ``n``, ``m`` are updated in place."""
    t, hn = proj.shape[0], lay.heads
    q, k = (proj[:, c:c + hn * lay.dim].float().view(t, hn, lay.dim) for c in (lay.q_col, lay.k_col))
    v, g = (proj[:, c:c + hn * lay.vdim].float().view(t, hn, lay.vdim) for c in (lay.v_col, lay.g_col))
    if w.decay is not None:
        o = _retain(q, k, v, lay, w.decay, s)
    else:
        o = _gated(q, k, v, z, lay, w, s, n, m)
    y = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / lay.rms_dim + eps)
    gate = (F.silu if lay.silu_gate else torch.sigmoid)(g.reshape(t, -1))
    return (y.view(t, -1) * w.norm * gate).to(proj.dtype)


def _run(proj, z, lay, w, slots, starts, cu, owner, eps):
    y = torch.empty(proj.shape[0], lay.heads * lay.vdim, dtype=proj.dtype)
    for b, (first, slot) in enumerate(zip(starts, owner)):
        rows = slice(cu[b], cu[b + 1])
        state = [None if k not in slots else slots[k][slot] if slot >= 0 else torch.zeros_like(slots[k][0])
                 for k in ("memory", "norm", "peak")]
        if first == 0:
            for x in state:
                if x is not None:
                    x.zero_()
        y[rows] = _recur(proj[rows], None if z is None else z[rows], lay, w, *state, eps)
    return y


def _arguments(proj, z, lay: MemoryLayout, w: MemoryWeights, slots, eps: float):
    """What the kernels of both kinds of steps take first."""
    return (ptr(proj), c_ll(proj.stride(0)), ptr(z), c_ll(0 if z is None else z.stride(0)), lay.ints(), lay.floats(eps), ptr(w.bias),
            ptr(w.decay), ptr(w.norm), ptr(slots["memory"]), ptr(slots.get("norm")), ptr(slots.get("peak")))


def memory_prefill(proj: torch.Tensor, z: Optional[torch.Tensor], lay: MemoryLayout, w: MemoryWeights,
                   slots: Dict[str, torch.Tensor], cu_q: torch.Tensor, max_q: int, start_pos: torch.Tensor,
                   state_slots: torch.Tensor, eps: float, chunked: bool = True) -> torch.Tensor:
    """Prompt portions: ``proj [T, ...]``, gate logits ``z [T, 2 * heads]`` fp32 (None with a constant decay) ->
    ``y [T, heads * vdim]``.  bf16 rows of the sizes that the tensor-core kernels serve run in chunks (``chunked=False`` keeps to the token-by-token kernel)."""
    t, batch = proj.shape[0], cu_q.numel() - 1
    if _lib.use_kernels(proj, cu_q, state_slots):
        L = _lib.load()
        y = guard.empty(t, lay.heads * lay.vdim, device=proj.device, dtype=proj.dtype)
        args = (*_arguments(proj, z, lay, w, slots, eps), ptr(cu_q), ptr(start_pos), ptr(state_slots))
        if chunked and proj.dtype == torch.bfloat16 and L.msrl_memory_chunked_serves(lay.ints()):
            size = L.msrl_memory_chunk_scratch
            size.restype = ctypes.c_longlong
            scratch = _workspace("memory_chunks", int(size(lay.ints(), c_int(t), c_int(batch))), proj.device)
            check(L.msrl_memory_prefill_chunked(*args, ptr(scratch), ptr(y), c_int(t), c_int(batch), c_int(max_q),
                                                ptr(_status_word(proj.device)), stream()), "memory_prefill_chunked")
            return y
        o = _workspace("memory_out", t * lay.heads * lay.vdim, proj.device)
        check(L.msrl_memory_prefill(*args, ptr(o), ptr(y), c_int(t), c_int(batch), _is_f32(proj), stream()), "memory_prefill")
        return y
    return _run(proj, z, lay, w, slots, start_pos.tolist(), cu_q.tolist(), state_slots.tolist(), eps)


def memory_decode(proj: torch.Tensor, z: Optional[torch.Tensor], lay: MemoryLayout, w: MemoryWeights,
                  slots: Dict[str, torch.Tensor], positions: torch.Tensor, state_slots: torch.Tensor, eps: float) -> torch.Tensor:
    """One token per sequence: state read and written once (``state_slots[b] < 0``: neither)."""
    b = proj.shape[0]
    if _lib.use_kernels(proj, positions, state_slots):
        y = guard.empty(b, lay.heads * lay.vdim, device=proj.device, dtype=proj.dtype)
        check(_lib.load().msrl_memory_decode(*_arguments(proj, z, lay, w, slots, eps), ptr(positions), ptr(state_slots), ptr(y),
                                             c_int(b), _is_f32(proj), stream()), "memory_decode")
        return y
    return _run(proj, z, lay, w, slots, positions.tolist(), range(b + 1), state_slots.tolist(), eps)
