"""Kernels around an fp32 residual stream: embedding, residual add and expert combine, each with the norm that
follows fused in, and the gated activations.

The residual ``[T, W]`` is fp32 and updated in place; norm weights are fp32, the activations bf16 or fp32.
``norm(x) = x / sqrt(mean(x^2) + eps) * (offset + w)`` in fp32; ``centered`` norms subtract the row's mean from x
first (a layer norm without bias).  ``post_*`` functions norm what a sublayer gives before it is added and hand on the
residual itself, rounded to the activation type, or a norm of it; ``entry``: what a pass of a loop adds in between.  CUDA
path: ``csrc/residual_stream.cu``; CPU tensors run the PyTorch formulation.
"""
from __future__ import annotations

from typing import NamedTuple, Optional, Tuple

import torch
import torch.nn.functional as F

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .gemm import linear_fwd


def _is_f32(t: torch.Tensor):
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"bf16 or fp32 activations expected, got {t.dtype}")
    return c_int(1 if t.dtype == torch.float32 else 0)


class Norm(NamedTuple):
    """Arguments of a norm in the order of the functions below."""
    weight: torch.Tensor
    eps: float
    offset: float = 0.0
    centered: bool = False


class PostNorm(NamedTuple):
    """Norm of a sublayer's output ``d`` and its factor: ``resid += mult * d / sqrt(mean(d^2) + eps) * weight``."""
    weight: torch.Tensor
    eps: float
    mult: float = 1.0


class PassEntry(NamedTuple):
    """What a pass of a loop adds to the residual before it runs: ``again [T, W]`` (or None) and ``step [W]``, fp32."""
    again: Optional[torch.Tensor]
    step: torch.Tensor


class TokenSide(NamedTuple):
    """A layer's input from the token itself: ``proj (gelu_tanh(gate x) * table[id, col:col + dim])``.  ``gate [pad, W]`` and
    ``proj [W, pad]`` are padded with zeros to whole vectors."""
    gate: torch.Tensor
    proj: torch.Tensor
    table: torch.Tensor
    col: int
    dim: int


def _norm_ref(x: torch.Tensor, w: torch.Tensor, eps: float, offset: float, centered: bool, dtype) -> torch.Tensor:
    if centered:
        x = x - x.mean(-1, keepdim=True)
    return (x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (offset + w)).to(dtype)


def embed_norm(ids: torch.Tensor, table: torch.Tensor, scale: float, w: torch.Tensor, eps: float,
               offset: float = 0.0, centered: bool = False) -> Tuple[torch.Tensor, torch.Tensor]:
    """``(residual fp32, norm(residual))`` of ``residual = table[ids] * scale``."""
    t, h = ids.numel(), table.shape[1]
    if _lib.use_kernels(ids, table, w):
        resid = guard.empty(t, h, device=table.device, dtype=torch.float32)
        y = guard.empty(t, h, device=table.device, dtype=table.dtype)
        check(_lib.load().msrl_embed_norm(ptr(ids), ptr(table), c_float(scale), ptr(resid), ptr(w), ptr(y), c_ll(t),
                                          c_int(h), c_float(eps), c_float(offset), c_int(centered), _is_f32(table), stream()),
              "embed_norm")
        return resid, y
    resid = table[ids].float() * scale
    return resid, _norm_ref(resid, w, eps, offset, centered, table.dtype)


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """``(residual fp32, residual in the table's type)`` of ``residual = table[ids] * scale``."""
    t, h = ids.numel(), table.shape[1]
    if _lib.use_kernels(ids, table):
        resid = guard.empty(t, h, device=table.device, dtype=torch.float32)
        y = guard.empty(t, h, device=table.device, dtype=table.dtype)
        check(_lib.load().msrl_embed_norm(ptr(ids), ptr(table), c_float(scale), ptr(resid), None, ptr(y), c_ll(t),
                                          c_int(h), c_float(0.0), c_float(0.0), c_int(0), _is_f32(table), stream()), "embed")
        return resid, y
    resid = table[ids].float() * scale
    return resid, resid.to(table.dtype, copy=True)


def _enter_ref(resid, entry: Optional[PassEntry]) -> None:
    if entry is not None:
        if entry.again is not None:
            resid.add_(entry.again)
        resid.add_(entry.step)


def _post_ref(resid, d, post: PostNorm, after: Optional[Norm], dtype, entry: Optional[PassEntry] = None):
    resid.add_(post.mult * (d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + post.eps) * post.weight))
    _enter_ref(resid, entry)
    return resid.to(dtype, copy=True) if after is None else _norm_ref(resid, *after, dtype)


def post_embed(ids: torch.Tensor, table: torch.Tensor, post: PostNorm, after: Norm, keep: bool = False,
               step: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, Optional[torch.Tensor], torch.Tensor]:
    """Normed embeddings: ``(residual fp32, a copy of it before step or None, after(residual))``; ``step [W]`` is added to the
    residual, ``keep`` asks for the copy."""
    t, width = ids.numel(), table.shape[1]
    if _lib.use_kernels(ids, table, post.weight):
        _plain(after)
        resid = guard.empty(t, width, device=table.device, dtype=torch.float32)
        first = guard.empty(t, width, device=table.device, dtype=torch.float32) if keep else None
        y = guard.empty(t, width, device=table.device, dtype=table.dtype)
        check(_lib.load().msrl_post_embed(
            ptr(ids), ptr(table), ptr(resid), ptr(first), ptr(post.weight), c_float(post.eps), c_float(post.mult),
            ptr(after.weight), c_float(after.eps), ptr(step), ptr(y), c_ll(t), c_int(width), _is_f32(table), stream()), "post_embed")
        return resid, first, y
    resid = torch.zeros(t, width)
    _post_ref(resid, table[ids].float(), post, None, table.dtype)
    first = resid.clone() if keep else None
    if step is not None:
        resid.add_(step)
    return resid, first, _norm_ref(resid, *after, table.dtype)


def post_add_(resid: torch.Tensor, delta: torch.Tensor, post: PostNorm, after: Optional[Norm] = None,
              entry: Optional[PassEntry] = None) -> torch.Tensor:
    """Add the normed ``delta`` in place; returns the sum (or, with ``after``, that norm of it) in ``delta``'s type."""
    if _lib.use_kernels(resid, delta, post.weight):
        return _post(resid, post, after, delta.dtype, entry, delta=delta.contiguous())
    return _post_ref(resid, delta.float(), post, after, delta.dtype, entry)


def moe_post_add_(resid: torch.Tensor, expert_rows: torch.Tensor, pos: torch.Tensor, weights: torch.Tensor, post: PostNorm,
                  after: Optional[Norm] = None, shared: Optional[torch.Tensor] = None,
                  entry: Optional[PassEntry] = None) -> torch.Tensor:
    """The same for ``d[t] = sum_j weights[t, j] * expert_rows[pos[t, j]] (+ shared[t])``; a negative ``pos`` is an expert
    that gives back its input, the residual's row.  ``weights [T, top]`` fp32."""
    if _lib.use_kernels(resid, expert_rows, pos, weights):
        return _post(resid, post, after, expert_rows.dtype, entry, rows=expert_rows, pos=pos, weights=weights.contiguous(),
                     shared=shared)
    pos = pos.long().view(resid.shape[0], -1)
    rows = torch.where((pos < 0)[..., None], resid[:, None, :], expert_rows[pos.clamp(min=0)].float())
    d = (rows * weights[..., None]).sum(1)
    return _post_ref(resid, d if shared is None else d + shared.float(), post, after, expert_rows.dtype, entry)


def _plain(after: Optional[Norm]) -> None:
    if after is not None and (after.centered or after.offset):
        raise ValueError("the norm behind a post-normed sublayer is a plain RMS norm")


def _post(resid, post, after, dtype, entry=None, delta=None, rows=None, pos=None, weights=None, shared=None):
    t, width = resid.shape
    _plain(after)
    again, step = entry or (None, None)
    y = guard.empty(t, width, device=resid.device, dtype=dtype)
    check(_lib.load().msrl_post_add(
        ptr(delta), ptr(rows), ptr(pos), ptr(weights), c_int(0 if weights is None else weights.shape[1]), ptr(shared), ptr(resid),
        ptr(post.weight), c_float(post.eps), c_float(post.mult), ptr(after.weight if after else None),
        c_float(after.eps if after else 0.0), ptr(again), ptr(step), ptr(y), c_ll(t), c_int(width), _is_f32(y), stream()),
        "post_add")
    return y


FUSED_SIDE_TOKENS = 64         # up to here the gate's product and activation are one kernel, beyond a matrix product


def token_side_(resid: torch.Tensor, x: torch.Tensor, ids: torch.Tensor, side: TokenSide, post: PostNorm,
                after: Optional[Norm] = None, entry: Optional[PassEntry] = None,
                fused_tokens: Optional[int] = None) -> torch.Tensor:
    """Add a layer's token input to the residual like :func:`post_add_`; ``x`` is the residual in the activation type."""
    t, width = resid.shape
    if _lib.use_kernels(resid, x, ids, side.gate, side.table):
        L, pad = _lib.load(), side.gate.shape[0]
        row = (ptr(side.table), ptr(ids), c_ll(side.table.shape[1]), c_int(side.col))
        if t <= (FUSED_SIDE_TOKENS if fused_tokens is None else fused_tokens):
            g = guard.empty(t, pad, device=x.device, dtype=x.dtype)
            check(L.msrl_side_gate_product(ptr(x), ptr(side.gate), ptr(g), c_ll(pad), *row, c_int(side.dim), c_ll(t), c_int(width),
                                           _is_f32(x), stream()), "side_gate_product")
        else:
            g = linear_fwd(x, side.gate)
            check(L.msrl_side_gate(ptr(g), c_ll(pad), *row, c_int(side.dim), c_ll(t), _is_f32(x), stream()), "side_gate")
        return post_add_(resid, linear_fwd(g, side.proj), post, after, entry)
    g = F.gelu(linear_fwd(x, side.gate)[:, :side.dim].float(), approximate="tanh")
    g = (g * side.table[ids, side.col:side.col + side.dim].float()).to(x.dtype)
    return post_add_(resid, linear_fwd(g, side.proj[:, :side.dim]), post, after, entry)


def soft_cap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``x <- cap * tanh(x / cap)`` in place (contiguous), computed in 32-bit."""
    if _lib.use_kernels(x):
        check(_lib.load().msrl_soft_cap(ptr(x), c_ll(x.numel()), c_float(cap), _is_f32(x), stream()), "soft_cap")
        return x
    return x.copy_(cap * torch.tanh(x.float() / cap))


def add_norm_(resid: torch.Tensor, delta: torch.Tensor, w: torch.Tensor, eps: float, offset: float = 0.0,
              centered: bool = False, delta2: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``resid += delta (+ delta2)`` in place; returns ``norm(resid)`` in ``delta``'s type."""
    t, h = resid.shape
    if _lib.use_kernels(resid, delta, w):
        delta = delta.contiguous()
        delta2 = None if delta2 is None else delta2.contiguous()
        y = guard.empty(t, h, device=resid.device, dtype=delta.dtype)
        check(_lib.load().msrl_add_norm(ptr(delta), ptr(delta2), ptr(resid), ptr(w), ptr(y), c_ll(t), c_int(h), c_float(eps),
                                        c_float(offset), c_int(centered), _is_f32(delta), stream()), "add_norm")
        return y
    resid.add_(delta.float() if delta2 is None else delta.float() + delta2.float())
    return _norm_ref(resid, w, eps, offset, centered, delta.dtype)


def moe_combine_norm_(resid: torch.Tensor, expert_rows: torch.Tensor, pos: torch.Tensor, top: int, expert_w: float,
                      h: torch.Tensor, shared: Optional[torch.Tensor], shared_gate: Optional[torch.Tensor],
                      w: torch.Tensor, eps: float, offset: float = 0.0, centered: bool = False,
                      delta: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``resid[t] += expert_w * sum_j expert_rows[pos[t, j]] + sigmoid(h[t] . shared_gate) * shared[t] + delta[t]`` in
    place; returns ``norm(resid)``.  ``pos [T * top]`` are the rows of a dispatch plan (``ops.moe``); without
    ``shared`` or ``delta`` their term is left out, without ``shared_gate`` the shared term counts in full."""
    t, width = resid.shape
    if _lib.use_kernels(resid, expert_rows, pos, h):
        y = guard.empty(t, width, device=resid.device, dtype=h.dtype)
        delta = None if delta is None else delta.contiguous()
        check(_lib.load().msrl_moe_combine_norm(
            ptr(expert_rows), ptr(pos), c_int(top), c_float(expert_w), ptr(h.contiguous()), ptr(shared_gate),
            ptr(shared), ptr(delta), ptr(resid), ptr(w), ptr(y), c_ll(t), c_int(width), c_float(eps), c_float(offset),
            c_int(centered), _is_f32(h), stream()), "moe_combine_norm")
        return y
    add = expert_rows[pos.long()].float().view(t, top, width).sum(1) * expert_w
    if shared is not None:
        sig = 1.0 if shared_gate is None else torch.sigmoid(h.float() @ shared_gate.float().reshape(-1, 1))
        add = add + sig * shared.float()
    if delta is not None:
        add = add + delta.float()
    resid.add_(add)
    return _norm_ref(resid, w, eps, offset, centered, h.dtype)


GLU_KINDS = {"silu": 0, "gelu_tanh": 1, "clamped_swish": 2}


def glu_fwd(gate_up: torch.Tensor, act: str, limit: float = 0.0, alpha: float = 1.0, plan=None) -> torch.Tensor:
    """Gated activation of ``[rows, gate | up]``: ``silu(g) * u``, ``gelu_tanh(g) * u`` or ``clamped_swish``:
    ``g' sigmoid(alpha g') (u' + 1)`` with ``g' = min(g, limit)``, ``u' = clamp(u, -limit, limit)``.  With a
    dispatch ``plan`` the rows are expert-grouped and pad rows are left untouched."""
    kind = GLU_KINDS[act]
    rows, f = gate_up.shape[0], gate_up.shape[-1] // 2
    if _lib.use_kernels(gate_up):
        x = gate_up.contiguous()
        y = guard.empty(rows, f, device=x.device, dtype=x.dtype)
        check(_lib.load().msrl_glu_fwd(ptr(x), ptr(y), c_ll(rows), c_int(f), c_int(kind), c_float(limit), c_float(alpha),
                                       ptr(plan.tile_expert if plan is not None else None),
                                       ptr(plan.counts if plan is not None else None),
                                       ptr(plan.offsets if plan is not None else None), _is_f32(x), stream()), "glu_fwd")
        return y
    g, u = gate_up.float().split(f, dim=-1)
    if act == "silu":
        y = F.silu(g) * u
    elif act == "gelu_tanh":
        y = F.gelu(g, approximate="tanh") * u
    else:
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        y = g * torch.sigmoid(alpha * g) * (u + 1.0)
    return y.to(gate_up.dtype)
