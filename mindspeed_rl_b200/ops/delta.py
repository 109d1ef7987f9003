"""Gated delta rule with a decay per key channel or per head over state slots: prompt portions and decode steps.

The weights of a layer (:class:`DeltaWeights`) and the carried state of all sequences (``ring``, ``state``) are
described in ``csrc/delta_rule.cu``, the CUDA path; CPU tensors run the PyTorch formulation.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .residual import _is_f32


@dataclass(frozen=True)
class DeltaLayout:
    """Sizes of a layer and the columns of its sections in the fused projection row."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    q_col: int
    k_col: int
    v_col: int
    b_col: int
    unit_eps: float = 1e-6
    head_decay: bool = False      # one decay per head instead of one per key channel
    silu_gate: bool = False       # the output gate is silu instead of sigmoid

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def ints(self):
        return (ctypes.c_int * 11)(self.taps, self.heads, self.kv_heads, self.dim, self.vdim, self.q_col, self.k_col,
                                   self.v_col, self.b_col, int(self.head_decay), int(self.silu_gate))


@dataclass
class DeltaWeights:
    conv: torch.Tensor        # [channels, taps] fp32 (q, k, v channels in order)
    a_log: torch.Tensor       # [heads] fp32
    dt_bias: torch.Tensor     # [heads * dim] fp32, or [heads] with one decay per head
    norm: torch.Tensor        # [vdim] fp32


def _recur(proj, a, gate, lay: DeltaLayout, w: DeltaWeights, hist, s, eps):
    """One sequence, fp32: ``hist [taps - 1, channels]`` earlier inputs, ``s [H, dim, vdim]`` (updated in place)."""
    t, kd = proj.shape[0], lay.kv_heads * lay.dim
    x = torch.cat([proj[:, lay.q_col:lay.q_col + kd], proj[:, lay.k_col:lay.k_col + kd],
                   proj[:, lay.v_col:lay.v_col + lay.heads * lay.vdim]], dim=1).float()
    ext = torch.cat([hist, x])
    y = F.silu(sum(ext[j:j + t] * w.conv[:, j] for j in range(lay.taps)))
    rep = lay.heads // lay.kv_heads

    def unit(z):
        z = z.view(t, lay.kv_heads, lay.dim)
        return (z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) + lay.unit_eps)).repeat_interleave(rep, dim=1)

    q, k, v = unit(y[:, :kd]) / math.sqrt(lay.dim), unit(y[:, kd:2 * kd]), y[:, 2 * kd:].view(t, lay.heads, lay.vdim)
    beta = torch.sigmoid(proj[:, lay.b_col:lay.b_col + lay.heads].float())
    g = torch.exp(-torch.exp(w.a_log).view(1, -1, 1)
                  * F.softplus(a.float() + w.dt_bias, threshold=60.0).view(t, lay.heads, -1))
    o = torch.empty(t, lay.heads, lay.vdim)
    for i in range(t):
        s.mul_(g[i].unsqueeze(-1))
        u = beta[i].unsqueeze(-1) * (v[i] - torch.einsum("hdv,hd->hv", s, k[i]))
        s.add_(k[i].unsqueeze(-1) * u.unsqueeze(1))
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w.norm * (F.silu if lay.silu_gate else torch.sigmoid)(gate.float()).view_as(o)
    return o.view(t, -1).to(proj.dtype), ext


def _reference(proj, a, gate, lay, w, ring, state, bounds, starts, slots, eps):
    out = torch.zeros(proj.shape[0], lay.heads * lay.vdim, dtype=proj.dtype)
    for b, slot in enumerate(slots.tolist()):
        lo, hi, start = bounds[b], bounds[b + 1], int(starts[b])
        if hi == lo or slot < 0:
            continue
        hist = torch.zeros(lay.taps - 1, lay.channels)
        for j in range(lay.taps - 1):
            p = start - (lay.taps - 1) + j
            if p >= 0:
                hist[j] = ring[slot, p % lay.taps].float()
        if start == 0:
            state[slot].zero_()
        out[lo:hi], ext = _recur(proj[lo:hi], a[lo:hi], gate[lo:hi], lay, w, hist, state[slot], eps)
        for p in range(max(start, start + hi - lo - lay.taps), start + hi - lo):
            ring[slot, p % lay.taps] = ext[lay.taps - 1 + p - start].to(ring.dtype)
    return out


def delta_prefill(proj: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, lay: DeltaLayout, w: DeltaWeights,
                  ring: torch.Tensor, state: torch.Tensor, tok_seq: torch.Tensor, cu: torch.Tensor,
                  start_pos: torch.Tensor, slots: torch.Tensor, eps: float) -> torch.Tensor:
    """Packed prompt portions (``cu [B + 1]``; sequence b starts at position ``start_pos[b]`` and carries its state
    in slot ``slots[b]``; ``a [T, heads * dim or heads]``: decay projection) -> gated, normed outputs ``[T, heads * vdim]``; ring and state are updated."""
    t, batch = proj.shape[0], cu.numel() - 1
    if _lib.use_kernels(proj, a, gate, ring, state, cu):
        L, ints = _lib.load(), lay.ints()
        L.msrl_delta_prefill_scratch.restype = c_ll
        n = L.msrl_delta_prefill_scratch(ints, c_ll(proj.stride(0)), c_ll(a.stride(0)), c_int(t), c_int(batch))
        scratch = guard.empty(int(n), device=proj.device, dtype=torch.float32)
        y = guard.empty(t, lay.heads * lay.vdim, device=proj.device, dtype=proj.dtype)
        check(L.msrl_delta_prefill(
            ptr(proj), c_ll(proj.stride(0)), ptr(a), c_ll(a.stride(0)), ptr(w.conv), ptr(w.a_log), ptr(w.dt_bias),
            ptr(ring), ptr(state), ints, c_float(lay.unit_eps), ptr(gate), c_ll(gate.stride(0)), ptr(w.norm),
            c_float(eps), ptr(tok_seq), ptr(cu), ptr(start_pos), ptr(slots), c_int(t), c_int(batch), ptr(scratch), ptr(y),
            _is_f32(proj), stream()), "delta_prefill")
        return y
    return _reference(proj, a, gate, lay, w, ring, state, cu.tolist(), start_pos, slots, eps)


def delta_decode(proj: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, lay: DeltaLayout, w: DeltaWeights,
                 ring: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                 eps: float) -> torch.Tensor:
    """One token per sequence (``slots[b] < 0``: row not in use)."""
    b = proj.shape[0]
    if _lib.use_kernels(proj, a, gate, ring, state, positions, slots):
        y = guard.empty(b, lay.heads * lay.vdim, device=proj.device, dtype=proj.dtype)
        check(_lib.load().msrl_delta_decode(
            ptr(proj), c_ll(proj.stride(0)), ptr(a), c_ll(a.stride(0)), ptr(w.conv), ptr(w.a_log), ptr(w.dt_bias),
            ptr(ring), ptr(state), lay.ints(), c_float(lay.unit_eps), ptr(gate), c_ll(gate.stride(0)), ptr(w.norm),
            c_float(eps), ptr(positions), ptr(slots), c_int(b), ptr(y), _is_f32(proj), stream()), "delta_decode")
        return y
    return _reference(proj, a, gate, lay, w, ring, state, list(range(b + 1)), positions, slots, eps)
