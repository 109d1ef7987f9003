"""Minimal gated recurrence over state slots: prompt portions and decode steps.

Element by element; gate and candidate do not depend on the state::

    z = sigmoid(z_proj + z_bias),  u = x_proj + x_bias,  c = u + 1/2 where u >= 0, else sigmoid(u)
    S <- (1 - z) S + z c,          y = S * silu(g_proj) * scale

A sequence starts with S zero; ``state [slots, width]`` is fp32, and a sequence's first token ignores what its slot holds.
Outputs become columns of a wider row.  CUDA path: ``csrc/min_gru.cu``; CPU tensors run the PyTorch formulation.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .elementwise import _workspace
from .residual import _is_f32


@dataclass(frozen=True)
class GRULayout:
    """``width`` channels, stored as ``padded`` output columns; the columns of the sections in the fused projection row and
    of the output in its row."""
    width: int
    padded: int
    z_col: int
    x_col: int
    g_col: int
    out_col: int = 0
    scale: float = 1.0


def _reference(proj, lay: GRULayout, z_bias, x_bias, state, out, bounds, starts, slots) -> None:
    z, x, g = (proj[:, c:c + lay.width].float() for c in (lay.z_col, lay.x_col, lay.g_col))
    z, u = torch.sigmoid(z + z_bias), x + x_bias
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    y = torch.zeros(proj.shape[0], lay.padded)
    for b, (first, slot) in enumerate(zip(starts, slots)):
        s = state[slot].clone() if first > 0 and slot >= 0 else torch.zeros(lay.width)
        for t in range(bounds[b], bounds[b + 1]):
            s = (1.0 - z[t]) * s + z[t] * cand[t]
            y[t, :lay.width] = s
        if slot >= 0:
            state[slot] = s
    y[:, :lay.width] *= F.silu(g) * lay.scale
    out[:, lay.out_col:lay.out_col + lay.padded] = y.to(out.dtype)


def _launch(proj, lay: GRULayout, z_bias, x_bias, state, out, cu, start, slots, batch: int, max_q: int) -> None:
    L, t = _lib.load(), proj.shape[0]
    L.msrl_min_gru_scratch.restype = c_ll
    n = L.msrl_min_gru_scratch(c_int(lay.width), c_int(t), c_int(batch), c_int(max_q))
    check(L.msrl_min_gru(ptr(proj[:, lay.z_col:]), ptr(proj[:, lay.x_col:]), ptr(proj[:, lay.g_col:]), c_ll(proj.stride(0)),
                         ptr(z_bias), ptr(x_bias), ptr(state), ptr(cu), ptr(start), ptr(slots), c_float(lay.scale),
                         ptr(out[:, lay.out_col:]), c_ll(out.stride(0)), c_int(lay.width), c_int(lay.padded), c_int(t),
                         c_int(batch), c_int(max_q), ptr(_workspace("min_gru", int(n), proj.device)), _is_f32(proj), stream()),
          "min_gru")


def min_gru_prefill(proj: torch.Tensor, lay: GRULayout, z_bias: torch.Tensor, x_bias: torch.Tensor, state: torch.Tensor,
                    out: torch.Tensor, cu: torch.Tensor, max_q: int, start_pos: torch.Tensor, slots: torch.Tensor) -> None:
    """Packed prompt portions (``cu [B + 1]``) into the columns ``[out_col, out_col + padded)`` of ``out``."""
    if _lib.use_kernels(proj, state, out, cu):
        _launch(proj, lay, z_bias, x_bias, state, out, cu, start_pos, slots, cu.numel() - 1, max_q)
        return
    _reference(proj, lay, z_bias, x_bias, state, out, cu.tolist(), start_pos.tolist(), slots.tolist())


def min_gru_decode(proj: torch.Tensor, lay: GRULayout, z_bias: torch.Tensor, x_bias: torch.Tensor, state: torch.Tensor,
                   out: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor) -> None:
    """One token per sequence (``slots[b] < 0``: no state)."""
    b = proj.shape[0]
    if _lib.use_kernels(proj, state, out, positions):
        _launch(proj, lay, z_bias, x_bias, state, out, None, positions, slots, b, 1)
        return
    _reference(proj, lay, z_bias, x_bias, state, out, range(b + 1), positions.tolist(), slots.tolist())
