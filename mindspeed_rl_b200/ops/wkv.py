"""Linear attention whose state decays per head and key channel by what the token says (wkv): prompt portions and decode steps.

``wkv_mix_*`` gives the rows that the projections read, ``h + (h' - h) mu_m`` with h' the previous token's h (zero before a
sequence's first token); the last token's h is carried in ``last [slots, W]`` fp32.  Per head, S zero at a sequence's start::

    w = exp(-exp(tanh(a) w2^T + w0))
    o = S^T r + (sum_k r u k) v,   S <- diag(w) S + k v^T,   y = o / rms(o) * norm * silu(gate)

``state [slots, H, dim, dim]`` fp32; a sequence's first token ignores what its slots hold.  CUDA path: ``csrc/wkv.cu``, ``csrc/wkv_chunk.cu``; CPU
tensors run the PyTorch formulation.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .elementwise import _workspace
from .residual import _is_f32

MIXES = 5
DECAY_IN_DECODE = 8            # sequences up to which a decode step computes its decays inside the recurrence


@dataclass
class WKVWeights:
    mu: torch.Tensor          # [MIXES, W] fp32
    w2: torch.Tensor          # [heads * dim, rank]
    w0: torch.Tensor          # [heads * dim] fp32, as u and norm
    u: torch.Tensor
    norm: torch.Tensor
    heads: int
    dim: int


def _mix_reference(h, mu, last, bounds, starts, slots):
    out = torch.empty(MIXES, *h.shape, dtype=h.dtype)
    for b, (first, slot) in enumerate(zip(starts, slots)):
        lo, hi = bounds[b], bounds[b + 1]
        if hi == lo:
            continue
        x = h[lo:hi].float()
        before = last[slot][None] if first > 0 and slot >= 0 else torch.zeros_like(x[:1])
        out[:, lo:hi] = (x + (torch.cat([before, x[:-1]]) - x) * mu[:, None, :]).to(h.dtype)
        if slot >= 0:
            last[slot] = x[-1]
    return out


def _mix(h, mu, last, tok_seq, cu, start, slots):
    t, width = h.shape
    out = guard.empty(MIXES, t, width, device=h.device, dtype=h.dtype)
    check(_lib.load().msrl_wkv_mix(ptr(h.contiguous()), ptr(mu), ptr(last), ptr(tok_seq), ptr(cu), ptr(start), ptr(slots), ptr(out),
                                   c_ll(t), c_int(width), _is_f32(h), stream()), "wkv_mix")
    return out


def wkv_mix_prefill(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, tok_seq: torch.Tensor, cu: torch.Tensor,
                    start_pos: torch.Tensor, slots: torch.Tensor) -> torch.Tensor:
    """``h [T, W]`` -> mixed rows ``[MIXES, T, W]`` of packed prompt portions; ``last`` is updated."""
    if _lib.use_kernels(h, mu, last, cu):
        return _mix(h, mu, last, tok_seq, cu, start_pos, slots)
    return _mix_reference(h, mu, last, cu.tolist(), start_pos.tolist(), slots.tolist())


def wkv_mix_decode(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor
                   ) -> torch.Tensor:
    """The same for one token per sequence (``slots[b] < 0``: nothing carried)."""
    if _lib.use_kernels(h, mu, last, positions):
        return _mix(h, mu, last, None, None, positions, slots)
    return _mix_reference(h, mu, last, range(h.shape[0] + 1), positions.tolist(), slots.tolist())


def wkv_decay(a: torch.Tensor, w: WKVWeights) -> torch.Tensor:
    """Bottleneck rows ``a [T, rank]`` fp32 -> decays ``[T, heads * dim]`` fp32."""
    t, rank = a.shape
    n = w.w0.numel()
    if _lib.use_kernels(a, w.w2, w.w0):
        out = guard.empty(t, n, device=a.device, dtype=torch.float32)
        check(_lib.load().msrl_wkv_decay(ptr(a.contiguous()), ptr(w.w2), ptr(w.w0), ptr(out), c_int(t), c_int(rank), c_int(n),
                                         _is_f32(w.w2), stream()), "wkv_decay")
        return out
    return torch.exp(-torch.exp(torch.tanh(a) @ w.w2.float().t() + w.w0))


def _reference(r, k, v, g, a, w: WKVWeights, state, bounds, starts, slots, eps):
    t, hn, d = r.shape[0], w.heads, w.dim
    decay = wkv_decay(a, w).view(t, hn, d)
    rf, kf, vf = (x.float().view(t, hn, d) for x in (r, k, v))
    u = w.u.view(hn, d)
    o = torch.zeros(t, hn, d)
    for b, (first, slot) in enumerate(zip(starts, slots)):
        s = state[slot].clone() if first > 0 and slot >= 0 else torch.zeros(hn, d, d)
        for i in range(bounds[b], bounds[b + 1]):
            o[i] = torch.einsum("hkv,hk->hv", s, rf[i]) + (rf[i] * u * kf[i]).sum(-1, keepdim=True) * vf[i]
            s = decay[i][:, :, None] * s + kf[i][:, :, None] * vf[i][:, None, :]
        if slot >= 0:
            state[slot] = s
    y = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps)
    return (y.view(t, -1) * w.norm * F.silu(g.float())).to(r.dtype)


def wkv_prefill(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, a: torch.Tensor, w: WKVWeights,
                state: torch.Tensor, cu: torch.Tensor, max_q: int, start_pos: torch.Tensor, slots: torch.Tensor, eps: float,
                segment: int = 0, chunked: bool = True) -> torch.Tensor:
    """Packed prompt portions, rows ``[T, heads * dim]`` -> ``[T, heads * dim]``.  ``segment``: tokens of the pieces that
    sequences are cut into (0: what fills the machine).  bf16 rows of the sizes that the tensor-core kernel serves go through
    it (``chunked=False`` keeps to the token-by-token kernel)."""
    t, batch = r.shape[0], cu.numel() - 1
    if _lib.use_kernels(r, k, v, g, a, state, cu):
        L, decay = _lib.load(), wkv_decay(a, w)
        L.msrl_wkv_scratch.restype = c_ll
        n = L.msrl_wkv_scratch(c_int(w.heads), c_int(w.dim), c_int(t), c_int(batch), c_int(max_q), c_int(segment))
        y = guard.empty(t, w.heads * w.dim, device=r.device, dtype=r.dtype)
        check(L.msrl_wkv_prefill(*(ptr(x.contiguous()) for x in (r, k, v, g)), ptr(decay), ptr(w.u), ptr(w.norm), ptr(state), ptr(cu),
                                 ptr(start_pos), ptr(slots), c_int(w.heads), c_int(w.dim), c_float(eps), c_int(t), c_int(batch),
                                 c_int(max_q), c_int(segment), c_int(chunked), ptr(_workspace("wkv", int(n), r.device)), ptr(y), _is_f32(r), stream()),
              "wkv_prefill")
        return y
    return _reference(r, k, v, g, a, w, state, cu.tolist(), start_pos.tolist(), slots.tolist(), eps)


def wkv_decode(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, a: torch.Tensor, w: WKVWeights,
               state: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, eps: float) -> torch.Tensor:
    """One token per sequence: state read and written once (``slots[b] < 0``: neither)."""
    b = r.shape[0]
    if _lib.use_kernels(r, k, v, g, a, state, positions):
        y = guard.empty(b, w.heads * w.dim, device=r.device, dtype=r.dtype)
        decay = wkv_decay(a, w) if b > DECAY_IN_DECODE else None
        check(_lib.load().msrl_wkv_decode(*(ptr(x.contiguous()) for x in (r, k, v, g)), ptr(decay), ptr(a.contiguous()), ptr(w.w2),
                                          ptr(w.w0), ptr(w.u), ptr(w.norm), ptr(state), ptr(positions), ptr(slots), c_int(w.heads),
                                          c_int(w.dim), c_int(a.shape[1]), c_float(eps), c_int(b), ptr(y), _is_f32(r), stream()),
              "wkv_decode")
        return y
    return _reference(r, k, v, g, a, w, state, range(b + 1), positions.tolist(), slots.tolist(), eps)
