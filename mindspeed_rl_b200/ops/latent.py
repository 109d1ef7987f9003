"""Latent attention ops: cache rows of ``[latent | rotated key part]``, prompt attention over expanded heads and
decode attention over the rows themselves.

A cache is ``[num_blocks, block_size, CP]``; row columns ``[0, RP)`` hold the normed latent (zero padded from
``rank``), ``[RP, CP)`` the rotated key part (zero padded from ``dr``).  :class:`LatentLayout` describes the
columns.  CUDA path: ``csrc/latent_attention.cu`` and the flash attention kernels; CPU tensors run the PyTorch
formulation.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .attention import _NOT_SUPPORTED, use_tcgen05_attention
from .elementwise import _workspace
from .residual import _is_f32
from .score_form import PLAIN, ScoreForm


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass(frozen=True)
class LatentLayout:
    """Columns of the projection rows and of the cache rows of one latent attention layer."""
    heads: int
    dn: int            # unrotated query / key entries per head
    dr: int            # rotated entries
    dv: int            # value entries
    rank: int
    qp: int            # padded query / key head size (head h's query starts at h * qp)
    vp: int            # padded value head size
    dkv_col: int       # column of the latent projection in the fused projection row
    rot_dims: int
    halves: bool = False   # rotated pairs are (i, i + rot_dims / 2) instead of neighbours
    q_rank: int = 0    # size of the queries' own latent (0: the heads are in the projection row)
    dq_col: int = 0    # its column in the projection row

    @property
    def RP(self) -> int:
        return pad16(self.rank)

    @property
    def QP(self) -> int:
        return (self.q_rank + 7) // 8 * 8

    @property
    def CP(self) -> int:
        return self.RP + pad16(self.dr)


def _turn(x: torch.Tensor, cs: torch.Tensor, dims: int, halves: bool = False) -> torch.Tensor:
    """Rotate the pairs of the last axis' first ``dims`` entries; ``cs [T, dims] = [cos | sin]`` (fp32)."""
    cs = cs.view(cs.shape[0], *([1] * (x.dim() - 2)), dims)
    c, s = cs[..., :dims // 2], cs[..., dims // 2:]
    if halves:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


def _rms(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.float()
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def latent_prep(proj: torch.Tensor, lay: LatentLayout, norm_w: torch.Tensor, eps: float, table: torch.Tensor,
                positions: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor, want_rows: bool,
                decode_q: Optional[torch.Tensor] = None, q_norm: Optional[torch.Tensor] = None):
    """Norm and rotate one step's projections and write their cache rows (``slots[t] < 0``: not written).

    Prompts (``decode_q`` None) rotate the query heads of ``proj`` in place; decode steps write the rotated part
    into ``decode_q [T, heads, CP]`` instead.  Returns the rows ``[T, CP]`` when ``want_rows``.

    With a query latent (``lay.q_rank``, norm weight ``q_norm``) the heads are not there yet: their part is left to
    ``latent_rotate_queries`` and the normed latent ``[T, QP]`` (zero padded) is returned after the rows."""
    t = proj.shape[0]
    if _lib.use_kernels(proj, norm_w, positions, slots, cache):
        rows = guard.empty(t, lay.CP, device=proj.device, dtype=proj.dtype) if want_rows else None
        cq = guard.empty(t, lay.QP, device=proj.device, dtype=proj.dtype) if lay.q_rank else None
        _prep(proj, 0 if lay.q_rank else lay.heads, lay, table, positions, decode_q, t, norm_w=norm_w, eps=eps, slots=slots,
              cache=cache, rows=rows, latent=proj.view(-1)[lay.dkv_col:], cq=cq, q_norm=q_norm)
        return (rows, cq) if lay.q_rank else rows
    cs = table[positions.long()]
    c = _rms(proj[:, lay.dkv_col:lay.dkv_col + lay.rank], norm_w, eps)
    kr = _turn(proj[:, lay.dkv_col + lay.rank:lay.dkv_col + lay.rank + lay.dr].float(), cs, lay.rot_dims, lay.halves)
    rows = torch.zeros(t, lay.CP, dtype=proj.dtype)
    rows[:, :lay.rank] = c.to(proj.dtype)
    rows[:, lay.RP:lay.RP + lay.dr] = kr.to(proj.dtype)
    ok = slots >= 0
    cache.view(-1, lay.CP)[slots[ok]] = rows[ok]
    if lay.q_rank:
        cq = _rms(proj[:, lay.dq_col:lay.dq_col + lay.q_rank], q_norm, eps)
        return rows if want_rows else None, torch.nn.functional.pad(cq, (0, lay.QP - lay.q_rank)).to(proj.dtype)
    latent_rotate_queries(proj, lay, table, positions, decode_q)
    return rows if want_rows else None


def _prep(q, heads, lay: LatentLayout, table, positions, decode_q, t, norm_w=None, eps=0.0, slots=None, cache=None, rows=None,
          latent=None, cq=None, q_norm=None):
    ints = (ctypes.c_int * 13)(heads, lay.qp, lay.dn, lay.dr, lay.rank, lay.rot_dims, table.shape[0], lay.RP, lay.CP,
                               int(lay.halves), lay.q_rank, lay.QP, lay.dq_col - lay.dkv_col)
    check(_lib.load().msrl_latent_prep(ptr(q), c_ll(q.stride(0)), ptr(latent), ints, ptr(norm_w), c_float(eps), ptr(q_norm),
                                       ptr(table), ptr(positions), ptr(slots), ptr(cache), ptr(rows), ptr(cq), ptr(decode_q),
                                       c_int(t), _is_f32(q), stream()), "latent_prep")


def latent_rotate_queries(q: torch.Tensor, lay: LatentLayout, table: torch.Tensor, positions: torch.Tensor,
                          decode_q: Optional[torch.Tensor] = None) -> None:
    """Rotate the query heads ``q [T, >= heads * qp]`` in place, or into ``decode_q [T, heads, CP]``."""
    t = q.shape[0]
    if _lib.use_kernels(q, table, positions):
        return _prep(q, lay.heads, lay, table, positions, decode_q, t)
    part = q[:, :lay.heads * lay.qp].view(t, lay.heads, lay.qp)[..., lay.dn:lay.dn + lay.dr]
    turned = _turn(part.float(), table[positions.long()], lay.rot_dims, lay.halves).to(q.dtype)
    if decode_q is None:
        part.copy_(turned)
    else:
        decode_q[..., lay.RP:] = 0
        decode_q[..., lay.RP:lay.RP + lay.dr] = turned


def latent_gather(cache: torch.Tensor, block_tables: torch.Tensor, token_seq: torch.Tensor,
                  token_pos: torch.Tensor) -> torch.Tensor:
    """Cache rows ``[T, CP]`` of tokens given as (block-table row, position)."""
    bs, cp = cache.shape[1], cache.shape[2]
    t = token_seq.numel()
    if _lib.use_kernels(cache, block_tables, token_seq, token_pos):
        out = guard.empty(t, cp, device=cache.device, dtype=cache.dtype)
        check(_lib.load().msrl_rows_gather(ptr(cache), ptr(block_tables), c_int(block_tables.shape[1]), c_int(bs),
                                             ptr(token_seq), ptr(token_pos), ptr(out), c_ll(t),
                                             c_int(cp * cache.element_size()), stream()), "latent_gather")
        return out
    blk = block_tables[token_seq.long(), (token_pos // bs).long()].long()
    return cache.view(-1, cp)[blk * bs + (token_pos % bs).long()]


def latent_spread_(kv: torch.Tensor, rows: torch.Tensor, lay: LatentLayout) -> torch.Tensor:
    """Copy the rotated key part of ``rows`` into every head's expanded key in ``kv [T, heads * (qp + vp)]``."""
    t = kv.shape[0]
    if _lib.use_kernels(kv, rows):
        check(_lib.load().msrl_latent_spread(ptr(rows), c_int(lay.CP), c_int(lay.RP), ptr(kv), c_ll(kv.stride(0)),
                                             c_int(lay.heads), c_int(lay.qp), c_int(lay.dn), c_int(lay.dr), c_int(t),
                                             _is_f32(kv), stream()), "latent_spread")
        return kv
    k = kv[:, :lay.heads * lay.qp].view(t, lay.heads, lay.qp)
    k[..., lay.dn:lay.dn + lay.dr] = rows[:, None, lay.RP:lay.RP + lay.dr]
    return kv


def latent_prefill_attention(proj: torch.Tensor, kv: torch.Tensor, lay: LatentLayout, cu_q: torch.Tensor,
                             cu_k: torch.Tensor, max_q: int, scale: float, window: Optional[int] = None,
                             form: ScoreForm = PLAIN) -> torch.Tensor:
    """Causal attention of the query heads of ``proj`` over expanded keys / values ``kv [Tk, K heads | V heads]``
    (bottom-right aligned when a sequence has more keys than queries) -> ``[T, heads * vp]``.  ``window``: keys a query
    sees, itself included (None: all)."""
    t, h, batch = proj.shape[0], lay.heads, cu_q.numel() - 1
    if _lib.use_kernels(proj, kv, cu_q, cu_k):
        v = kv.view(-1)[h * lay.qp:]
        out = guard.empty(t, h * lay.vp, device=proj.device, dtype=proj.dtype)
        if proj.dtype == torch.bfloat16 and (lay.qp, lay.vp) in ((64, 64), (128, 128), (192, 128)):
            from .gemm import _status_word
            st = (proj.stride(0), kv.stride(0))
            spec = (ctypes.c_longlong * 12)(st[0], 0, h, lay.qp, st[1], 0, h, lay.qp, st[1], 0, h, lay.vp)
            lse = guard.empty(h, t, device=proj.device, dtype=torch.float32)
            if lay.qp >= 128 and use_tcgen05_attention():
                rc = _lib.load().msrl_flash_attn_varlen_fwd_tcgen05(
                    ptr(proj), ptr(kv), ptr(v), spec, ptr(out), c_ll(h * lay.vp), ptr(lse), ptr(cu_q), ptr(cu_k),
                    c_int(batch), c_int(max_q), c_int(h), c_int(h), c_ll(t), c_ll(kv.shape[0]), c_int(lay.qp),
                    c_float(scale), c_int(1), c_int(window or 0), *form.args(), ptr(_status_word(proj.device)), stream())
                if rc != _NOT_SUPPORTED:
                    check(rc, "flash_attn_varlen_fwd_tcgen05")
                    return out
            if lay.qp <= 128:
                check(_lib.load().msrl_flash_attn_varlen_fwd(
                    ptr(proj), ptr(kv), ptr(v), spec, ptr(out), c_ll(h * lay.vp), ptr(lse), ptr(cu_q), ptr(cu_k),
                    c_int(batch), c_int(max_q), c_int(h), c_int(h), c_ll(t), c_int(lay.qp), c_float(scale), c_int(1),
                    c_int(window or 0), *form.args(), stream()), "flash_attn_varlen_fwd")
                return out
        lds = (ctypes.c_longlong * 4)(proj.stride(0), kv.stride(0), kv.stride(0), h * lay.vp)
        ints = (ctypes.c_int * 8)(lay.qp, lay.qp, lay.vp, lay.vp, lay.dn + lay.dr, lay.vp, 1, window or 0)
        check(_lib.load().msrl_attn_simt(ptr(proj), ptr(kv), ptr(v), ptr(out), lds, ints, ptr(cu_q), ptr(cu_k),
                                         c_int(batch), c_int(max_q), c_int(h), c_float(scale), *form.args(), _is_f32(proj),
                                         stream()), "attn_simt")
        return out
    q = proj[:, :h * lay.qp].view(t, h, lay.qp).float()
    k = kv[:, :h * lay.qp].view(-1, h, lay.qp).float()
    v = kv[:, h * lay.qp:].view(-1, h, lay.vp).float()
    out = torch.zeros(t, h, lay.vp)
    cq, ck = cu_q.tolist(), cu_k.tolist()
    for b in range(batch):
        qi, ki, vi = q[cq[b]:cq[b + 1]], k[ck[b]:ck[b + 1]], v[ck[b]:ck[b + 1]]
        lq, lk = qi.shape[0], ki.shape[0]
        s = torch.einsum("qhd,khd->hqk", qi, ki) * scale
        back = torch.arange(lq).unsqueeze(1) + (lk - lq) - torch.arange(lk)
        p = form.weights(s, (back < 0) | (back >= (window or lk + 1)))
        out[cq[b]:cq[b + 1]] = torch.einsum("hqk,khd->qhd", p, vi)
    return form.gated(out).view(t, h * lay.vp).to(proj.dtype)


def latent_decode_attention(q: torch.Tensor, cache: torch.Tensor, lay: LatentLayout, block_tables: torch.Tensor,
                            context_lens: torch.Tensor, max_context: int, scale: float,
                            nsplit: Optional[int] = None, use_tcgen05: bool = True, window: Optional[int] = None,
                            form: ScoreForm = PLAIN) -> torch.Tensor:
    """One query per sequence, ``q [B, heads, CP]`` in cache-row space, over the sequence's cached rows (the last
    ``window`` of them) -> weighted latents ``[B, heads, RP]``; without a soft cap.  ``nsplit``: key ranges per sequence (default: what fills the machine);
    ``use_tcgen05=False`` keeps to the ``mma.sync`` kernel (comparison runs)."""
    b, h, cp = q.shape
    bs = cache.shape[1]
    assert not form.softcap
    if _lib.use_kernels(q, cache, block_tables, context_lens):
        L = _lib.load()
        out = guard.empty(b, h, lay.RP, device=q.device, dtype=q.dtype)
        extra = (c_int(window or 0), *form.args()[1:])
        if q.dtype == torch.bfloat16:
            n = nsplit or int(L.msrl_latent_decode_nsplit(c_int(b), c_int(h), c_int(min(int(max_context), (window or 1 << 30) + 64))))
            part_o = part_ml = None
            if n > 1:
                part_o = _workspace("latent_part_o", b * h * n * lay.RP, q.device)
                part_ml = _workspace("latent_part_ml", b * h * n * 2, q.device)
            if use_tcgen05:
                from .gemm import _status_word
                rc = L.msrl_latent_decode_tcgen05(
                    ptr(q), ptr(cache), c_ll(cache.shape[0]), ptr(block_tables), c_int(block_tables.shape[1]), c_int(bs),
                    ptr(context_lens), c_float(scale), c_int(b), c_int(h), c_int(cp), c_int(lay.RP), c_int(n), *extra, ptr(part_o),
                    ptr(part_ml), ptr(out), ptr(_status_word(q.device)), stream())
                if rc != _NOT_SUPPORTED:
                    check(rc, "latent_decode_tcgen05")
                    if n > 1:
                        check(L.msrl_latent_decode_combine(ptr(part_o), ptr(part_ml), c_int(b), c_int(h), c_int(lay.RP),
                                                           c_int(n), *extra[1:], ptr(out), stream()), "latent_decode_combine")
                    return out
            rc = L.msrl_latent_decode_mma(ptr(q), ptr(cache), ptr(block_tables), c_int(block_tables.shape[1]), c_int(bs),
                                          ptr(context_lens), c_float(scale), c_int(b), c_int(h), c_int(cp),
                                          c_int(lay.RP), c_int(n), *extra, ptr(part_o), ptr(part_ml), ptr(out), stream())
            if rc != _NOT_SUPPORTED:
                check(rc, "latent_decode_mma")
                return out
        check(L.msrl_latent_decode_simt(ptr(q), ptr(cache), ptr(block_tables), c_int(block_tables.shape[1]), c_int(bs),
                                        ptr(context_lens), c_float(scale), c_int(b), c_int(h), c_int(cp), c_int(lay.RP),
                                        *extra, ptr(out), _is_f32(q), stream()), "latent_decode_simt")
        return out
    out = torch.zeros(b, h, lay.RP)
    flat = cache.view(-1, cp)
    for i in range(b):
        n = int(context_lens[i])
        pos = torch.arange(max(0, n - (window or n)), n)
        rows = flat[block_tables[i, (pos // bs).long()].long() * bs + pos % bs].float()
        out[i] = form.weights(q[i].float() @ rows.t() * scale) @ rows[:, :lay.RP]
    return form.gated(out).to(q.dtype)
