"""Between a q | k | v projection and grouped-head attention: short causal convolutions over time on every channel, an RMS
norm per query and key head, rotation of neighbouring entries, and the cache write, in one kernel (``csrc/conv_qkv.cu``).

The projection's heads are stored as they are (:class:`ConvHeads`); the prepared rows and the cache hold them padded, as
:class:`ops.window.GroupedHeads` describes.  A sequence carries the last inputs of its convolutions in a ring of ``taps``
entries per state slot (entry p % taps holds position p).  CPU tensors run the PyTorch formulation.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .latent import _turn
from .residual import _is_f32
from .window import GroupedHeads


@dataclass(frozen=True)
class ConvHeads:
    """Columns of the sections in the projection row, and where the prepared rows have theirs (``out``)."""
    out: GroupedHeads
    taps: int
    q_col: int
    k_col: int
    v_col: int

    @property
    def channels(self) -> int:
        o = self.out
        return (o.heads + o.kv_heads) * o.dim + o.kv_heads * o.vdim

    @property
    def row(self) -> int:
        o = self.out
        return (o.heads + o.kv_heads) * o.qp + o.kv_heads * o.vp

    def sections(self):
        o = self.out
        return ((self.q_col, o.heads, o.dim, o.q_col, o.qp), (self.k_col, o.kv_heads, o.dim, o.k_col, o.qp),
                (self.v_col, o.kv_heads, o.vdim, o.v_col, o.vp))


@dataclass
class ConvNormWeights:
    conv: torch.Tensor        # [channels, taps] fp32 (q, k, v channels in order, last tap = current token)
    q_norm: torch.Tensor      # [dim] fp32
    k_norm: torch.Tensor      # [dim] fp32


def _launch(proj, lay: ConvHeads, w: ConvNormWeights, eps, table, positions, slots, k_cache, v_cache, ring, state_slots,
            tok_seq=None, cu=None, start_pos=None) -> torch.Tensor:
    t, o, prompt = proj.shape[0], lay.out, cu is not None
    out = guard.empty(t, lay.row if prompt else o.heads * o.qp, device=proj.device, dtype=proj.dtype)
    ints = (ctypes.c_int * 16)(o.heads, o.kv_heads, o.dim, o.vdim, o.qp, o.vp, lay.taps, lay.q_col, lay.k_col, lay.v_col, o.q_col,
                               o.k_col, o.v_col, table.shape[1], table.shape[0], 0 if cu is None else cu.numel() - 1)
    check(_lib.load().msrl_conv_qkv(
        ptr(proj), c_ll(proj.stride(0)), ints, ptr(w.conv), ptr(w.q_norm), ptr(w.k_norm), c_float(eps), ptr(table), ptr(positions),
        ptr(slots), ptr(k_cache), ptr(v_cache), ptr(ring), ptr(state_slots), ptr(tok_seq), ptr(cu), ptr(start_pos), ptr(out),
        c_ll(out.stride(0)), c_int(t), _is_f32(proj), stream()), "conv_qkv")
    return out


def _reference(proj, lay: ConvHeads, w, eps, table, positions, slots, k_cache, v_cache, ring, state_slots, bounds, starts):
    t, o, taps = proj.shape[0], lay.out, lay.taps
    x = torch.cat([proj[:, c:c + n * d] for c, n, d, _, _ in lay.sections()], dim=1).float()
    y = torch.zeros_like(x)
    for b, slot in enumerate(state_slots.tolist()):
        lo, hi, start = bounds[b], bounds[b + 1], int(starts[b])
        if hi == lo:
            continue
        hist = torch.zeros(taps - 1, lay.channels)
        for j in range(taps - 1):
            p = start - (taps - 1) + j
            if p >= 0 and slot >= 0:
                hist[j] = ring[slot, p % taps].float()
        ext = torch.cat([hist, x[lo:hi]])
        y[lo:hi] = sum(ext[j:j + hi - lo] * w.conv[:, j] for j in range(taps))
        for p in range(max(start, start + hi - lo - taps), start + hi - lo):
            if slot >= 0:
                ring[slot, p % taps] = ext[taps - 1 + p - start].to(ring.dtype)
    out = torch.zeros(t, lay.row, dtype=proj.dtype)
    cs, at = table[positions.long()], 0
    for i, (_, n, d, col, pad) in enumerate(lay.sections()):
        f = y[:, at:at + n * d].view(t, n, d)
        at += n * d
        if i < 2:
            f = f / torch.sqrt(f.pow(2).mean(-1, keepdim=True) + eps) * (w.q_norm, w.k_norm)[i]
            f = _turn(f, cs, table.shape[1])
        out[:, col:col + n * pad].view(t, n, pad)[..., :d] = f.to(out.dtype)
    ok = slots >= 0
    for cache, part in zip((k_cache, v_cache), o.split(out)[1:]):
        cache.view(-1, *cache.shape[2:])[slots[ok]] = part[ok]
    return out


def conv_qkv_prefill(proj: torch.Tensor, lay: ConvHeads, w: ConvNormWeights, eps: float, table: torch.Tensor,
                     positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                     ring: torch.Tensor, state_slots: torch.Tensor, tok_seq: torch.Tensor, cu: torch.Tensor,
                     start_pos: torch.Tensor) -> torch.Tensor:
    """Packed prompt portions (``cu [B + 1]``; sequence b starts at position ``start_pos[b]`` and carries its ring in slot
    ``state_slots[b]``) -> prepared rows ``[T, row]``; keys and values also go to the cache (``slots[t] < 0``: not
    written), the last inputs to the ring."""
    if _lib.use_kernels(proj, w.conv, positions, slots, k_cache, ring, cu):
        return _launch(proj, lay, w, eps, table, positions, slots, k_cache, v_cache, ring, state_slots, tok_seq, cu, start_pos)
    return _reference(proj, lay, w, eps, table, positions, slots, k_cache, v_cache, ring, state_slots, cu.tolist(), start_pos)


def conv_qkv_decode(proj: torch.Tensor, lay: ConvHeads, w: ConvNormWeights, eps: float, table: torch.Tensor,
                    positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                    ring: torch.Tensor, state_slots: torch.Tensor) -> torch.Tensor:
    """One token per sequence -> its prepared query heads (``[B, heads * qp]``, or whole rows on the CPU); keys and values
    go to the cache and the inputs to the ring (negative slots: row not in use)."""
    if _lib.use_kernels(proj, w.conv, positions, slots, k_cache, ring):
        return _launch(proj, lay, w, eps, table, positions, slots, k_cache, v_cache, ring, state_slots)
    return _reference(proj, lay, w, eps, table, positions, slots, k_cache, v_cache, ring, state_slots,
                      list(range(proj.shape[0] + 1)), positions)
