"""Grouped-head soft-max attention over a window of paged keys and values.

Query / key heads of ``dim`` and value heads of ``vdim`` entries are stored padded to ``qp`` / ``vp``
(:class:`GroupedHeads`); the pad entries are zero.  ``qkv_prep_`` turns fused projection rows into what attention and
the cache take: RMS norm over the whole query and the whole key projection, partial rotation (entry i with entry
i + dims / 2), and values mixed with those of another layer, in one kernel (``csrc/qkv_prep.cu``).  Token i sees the
``window`` tokens up to and including itself (None: all); decode steps may see their ``chunk`` of tokens instead (prompts in
chunks are packed as one sequence per chunk).  ``ops.ScoreForm``: soft cap, sink and gates.  Prompt attention: ``csrc/attention_tcgen05.cu``,
``csrc/attention.cu``; decode: ``csrc/decode.cu``; fp32 and head sizes outside those: ``csrc/attention_simt.cu``.  CPU
tensors run the PyTorch formulation.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import NamedTuple, Optional, Tuple

import torch

from . import guard

from . import _lib
from ._lib import c_float, c_int, c_ll, check, ptr, stream
from .attention import _NOT_SUPPORTED, use_tcgen05_attention
from .elementwise import _workspace
from .latent import latent_gather
from .residual import _is_f32
from .score_form import PLAIN, ScoreForm

TENSOR_CORE_HEADS = ((64, 64), (128, 128), (192, 128))


class ValueSource(NamedTuple):
    """Value heads of another layer for the same tokens: ``x [T, >= kv_heads * vp]`` (rows may be strided)."""
    x: torch.Tensor
    vdim: int
    vp: int


@dataclass(frozen=True)
class GroupedHeads:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    qp: int
    vp: int
    q_col: int         # columns of the sections in a fused projection row
    k_col: int
    v_col: int

    def values(self, proj: torch.Tensor) -> ValueSource:
        return ValueSource(proj[:, self.v_col:self.v_col + self.kv_heads * self.vp], self.vdim, self.vp)

    def split(self, proj: torch.Tensor):
        t = proj.shape[0]
        return (proj[:, self.q_col:self.q_col + self.heads * self.qp].view(t, self.heads, self.qp),
                proj[:, self.k_col:self.k_col + self.kv_heads * self.qp].view(t, self.kv_heads, self.qp),
                proj[:, self.v_col:self.v_col + self.kv_heads * self.vp].view(t, self.kv_heads, self.vp))


_tables = {}


def angle_table(length: int, frequencies: Tuple[float, ...], device) -> torch.Tensor:
    """``[length, 2 * len(frequencies)]`` fp32 ``[cos | sin]`` of ``position * frequency`` (angles in fp64)."""
    key = (length, frequencies, str(device))
    if key not in _tables:
        a = torch.arange(length, dtype=torch.float64)[:, None] * torch.tensor(frequencies, dtype=torch.float64)
        _tables[key] = torch.cat([a.cos(), a.sin()], dim=1).float().contiguous().to(device)
    return _tables[key]


def qkv_prep_(proj: torch.Tensor, lay: GroupedHeads, q_norm: torch.Tensor, k_norm: torch.Tensor, eps: float,
              table: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
              v_cache: torch.Tensor, first: Optional[ValueSource] = None, mix: Optional[torch.Tensor] = None) -> None:
    """Norm, rotate and mix the rows of ``proj`` in place and write their keys and values to the cache
    (``slots[t] < 0``: not written).  ``first`` and ``mix [1]``: ``v <- (1 - mix) v + mix v_first``."""
    t = proj.shape[0]
    rot = table.shape[1]
    if _lib.use_kernels(proj, q_norm, positions, slots, k_cache, v_cache):
        ints = (ctypes.c_int * 13)(lay.heads, lay.kv_heads, lay.dim, lay.vdim, lay.qp, lay.vp, lay.q_col, lay.k_col, lay.v_col,
                                   rot, table.shape[0], first.vdim if first else lay.vdim, first.vp if first else lay.vp)
        check(_lib.load().msrl_qkv_prep(
            ptr(proj), c_ll(proj.stride(0)), ints, ptr(q_norm), ptr(k_norm), c_float(eps), ptr(table), ptr(positions), ptr(slots),
            ptr(k_cache), ptr(v_cache), ptr(first.x if first else None), c_ll(first.x.stride(0) if first else 0),
            ptr(mix if first else None), c_int(t), _is_f32(proj), stream()), "qkv_prep")
        return
    cs = table[positions.long()][:, None, :]
    c, s = cs[..., :rot // 2], cs[..., rot // 2:]
    q, k, v = lay.split(proj)
    for x, w in ((q, q_norm), (k, k_norm)):
        f = x.float().reshape(t, -1)
        f = f / torch.sqrt(f.pow(2).sum(-1, keepdim=True) / (x.shape[1] * lay.dim) + eps) * w
        f = f.view(x.shape)
        a, b = f[..., :rot // 2], f[..., rot // 2:rot]
        x.copy_(torch.cat([a * c - b * s, b * c + a * s, f[..., rot:]], dim=-1))
    if first is not None:
        other = first.x.float().reshape(t, -1, first.vp)[..., :first.vdim].reshape(t, lay.kv_heads, lay.vdim)
        v[..., :lay.vdim] = ((1.0 - mix) * v[..., :lay.vdim].float() + mix * other).to(v.dtype)
    ok = slots >= 0
    k_cache.view(-1, *k_cache.shape[2:])[slots[ok]] = k[ok]
    v_cache.view(-1, *v_cache.shape[2:])[slots[ok]] = v[ok]


def _turned(x: torch.Tensor, cs: torch.Tensor, back: bool = False) -> torch.Tensor:
    """``x [T, heads, n]`` with entry i turned with entry i + n / 2 by the angles of ``cs [T, n]`` (cos | sin)."""
    half = cs.shape[1] // 2
    c, s = cs[:, None, :half], cs[:, None, half:] * (-1.0 if back else 1.0)
    a, b = x[..., :half], x[..., half:]
    return torch.cat([a * c - b * s, b * c + a * s], dim=-1)


def turned_prep_(proj: torch.Tensor, lay: GroupedHeads, eps: float, table: torch.Tensor, value_table: torch.Tensor,
                 positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor) -> None:
    """Rotate queries and keys, norm (RMS per head, no weight) and turn values over all their entries, in place, and write keys
    and values to the cache (``slots[t] < 0``: not written).  ``value_table [length, vdim]``."""
    t, rot = proj.shape[0], table.shape[1]
    if _lib.use_kernels(proj, positions, slots, k_cache, v_cache):
        ints = (ctypes.c_int * 11)(lay.heads, lay.kv_heads, lay.dim, lay.vdim, lay.qp, lay.vp, lay.q_col, lay.k_col, lay.v_col,
                                   rot, table.shape[0])
        check(_lib.load().msrl_turned_prep(
            ptr(proj), c_ll(proj.stride(0)), ints, c_float(eps), ptr(table), ptr(value_table), ptr(positions), ptr(slots),
            ptr(k_cache), ptr(v_cache), c_int(t), _is_f32(proj), stream()), "turned_prep")
        return
    at = positions.long()
    q, k, v = lay.split(proj)
    for x in (q, k):
        x[..., :rot] = _turned(x[..., :rot].float(), table[at]).to(x.dtype)
    f = v[..., :lay.vdim].float()
    f = f / torch.sqrt(f.pow(2).mean(-1, keepdim=True) + eps)
    v[..., :lay.vdim] = _turned(f, value_table[at]).to(v.dtype)
    ok = slots >= 0
    k_cache.view(-1, *k_cache.shape[2:])[slots[ok]] = k[ok]
    v_cache.view(-1, *v_cache.shape[2:])[slots[ok]] = v[ok]


def turn_back(attn: torch.Tensor, lay: GroupedHeads, value_table: torch.Tensor, positions: torch.Tensor, scale: float,
              out: torch.Tensor) -> None:
    """Attention outputs ``[T, heads * vp]`` turned back by their token's position and scaled, into the first columns of
    ``out``."""
    t = attn.shape[0]
    if _lib.use_kernels(attn, positions, out):
        check(_lib.load().msrl_turn_back(
            ptr(attn), ptr(out), c_ll(out.stride(0)), c_int(lay.heads), c_int(lay.vdim), c_int(lay.vp), ptr(value_table),
            c_int(value_table.shape[0]), ptr(positions), c_float(scale), c_int(t), _is_f32(attn), stream()), "turn_back")
        return
    x = attn.view(t, lay.heads, lay.vp).float()
    y = _turned(x[..., :lay.vdim], value_table[positions.long()], back=True) * scale
    out[:, :lay.heads * lay.vp] = torch.cat([y, x[..., lay.vdim:] * 0.0], dim=-1).reshape(t, -1).to(out.dtype)


def rows_gather(cache: torch.Tensor, block_tables: torch.Tensor, token_seq: torch.Tensor, token_pos: torch.Tensor
                ) -> torch.Tensor:
    """Cache rows ``[T, *row]`` of tokens given as (block-table row, position)."""
    nb, bs = cache.shape[:2]
    return latent_gather(cache.view(nb, bs, -1), block_tables, token_seq, token_pos).view(-1, *cache.shape[2:])


def window_prefill_attention(proj: torch.Tensor, lay: GroupedHeads, cu_q: torch.Tensor, cu_k: torch.Tensor, max_q: int,
                             scale: float, window: Optional[int], kv: Optional[Tuple[torch.Tensor, torch.Tensor]] = None,
                             use_tcgen05: bool = True, form: ScoreForm = PLAIN) -> torch.Tensor:
    """Causal window attention of the query heads of prepared rows -> ``[T, heads * vp]``.  Keys and values are those of
    the same rows, or ``kv = (k [Tk, kv_heads, qp], v [Tk, kv_heads, vp])`` delimited by ``cu_k`` (bottom-right aligned
    when a sequence has more keys than queries)."""
    t, h, g, batch = proj.shape[0], lay.heads, lay.kv_heads, cu_q.numel() - 1
    if _lib.use_kernels(proj, cu_q, cu_k):
        flat, L = proj.view(-1), _lib.load()
        ld = proj.stride(0)
        if kv is None:
            k, v, kld, vld, tk = flat[lay.k_col:], flat[lay.v_col:], ld, ld, t
        else:
            k, v, kld, vld, tk = kv[0], kv[1], g * lay.qp, g * lay.vp, kv[0].shape[0]
        q = flat[lay.q_col:]
        out = guard.empty(t, h * lay.vp, device=proj.device, dtype=proj.dtype)
        win = c_int(window or 0)
        if proj.dtype == torch.bfloat16 and (lay.qp, lay.vp) in TENSOR_CORE_HEADS:
            from .gemm import _status_word
            spec = (ctypes.c_longlong * 12)(ld, 0, h, lay.qp, kld, 0, g, lay.qp, vld, 0, g, lay.vp)
            lse = guard.empty(h, t, device=proj.device, dtype=torch.float32)
            if lay.qp >= 128 and use_tcgen05 and use_tcgen05_attention():
                rc = L.msrl_flash_attn_varlen_fwd_tcgen05(
                    ptr(q), ptr(k), ptr(v), spec, ptr(out), c_ll(h * lay.vp), ptr(lse), ptr(cu_q), ptr(cu_k), c_int(batch),
                    c_int(max_q), c_int(h), c_int(g), c_ll(t), c_ll(tk), c_int(lay.qp), c_float(scale), c_int(1), win,
                    *form.args(), ptr(_status_word(proj.device)), stream())
                if rc != _NOT_SUPPORTED:
                    check(rc, "flash_attn_varlen_fwd_tcgen05")
                    return out
            if lay.qp <= 128:
                check(L.msrl_flash_attn_varlen_fwd(
                    ptr(q), ptr(k), ptr(v), spec, ptr(out), c_ll(h * lay.vp), ptr(lse), ptr(cu_q), ptr(cu_k), c_int(batch),
                    c_int(max_q), c_int(h), c_int(g), c_ll(t), c_int(lay.qp), c_float(scale), c_int(1), win, *form.args(),
                    stream()), "flash_attn_varlen_fwd")
                return out
        lds = (ctypes.c_longlong * 4)(ld, kld, vld, h * lay.vp)
        ints = (ctypes.c_int * 8)(lay.qp, lay.qp, lay.vp, lay.vp, lay.qp, lay.vp, h // g, window or 0)
        check(L.msrl_attn_simt(ptr(q), ptr(k), ptr(v), ptr(out), lds, ints, ptr(cu_q), ptr(cu_k), c_int(batch), c_int(max_q),
                               c_int(h), c_float(scale), *form.args(), _is_f32(proj), stream()), "attn_simt")
        return out
    q, k, v = lay.split(proj)
    if kv is not None:
        k, v = kv
    q, k, v = (x.float() for x in (q, k, v))
    k, v = (x.repeat_interleave(h // g, dim=1) for x in (k, v))
    out = torch.zeros(t, h, lay.vp)
    cq, ck = cu_q.tolist(), cu_k.tolist()
    for b in range(batch):
        qi, ki, vi = q[cq[b]:cq[b + 1]], k[ck[b]:ck[b + 1]], v[ck[b]:ck[b + 1]]
        back = torch.arange(qi.shape[0])[:, None] + (ki.shape[0] - qi.shape[0]) - torch.arange(ki.shape[0])
        hide = (back < 0) | (back >= (window or back.shape[1] + 1))
        p = form.weights(torch.einsum("qhd,khd->hqk", qi, ki) * scale, hide)
        out[cq[b]:cq[b + 1]] = torch.einsum("hqk,khd->qhd", p, vi)
    return form.gated(out).view(t, h * lay.vp).to(proj.dtype)


def window_decode_attention(proj: torch.Tensor, lay: GroupedHeads, k_cache: torch.Tensor, v_cache: torch.Tensor,
                            block_tables: torch.Tensor, context_lens: torch.Tensor, max_context: int, scale: float,
                            window: Optional[int], nsplit: Optional[int] = None, chunk: Optional[int] = None,
                            form: ScoreForm = PLAIN) -> torch.Tensor:
    """One query per sequence (prepared rows; the cache holds their own keys too) over the last ``window`` cached tokens,
    or those of its ``chunk`` -> ``[B, heads * vp]``.  ``nsplit``: key ranges per sequence (default: what fills the machine)."""
    b, h, g = proj.shape[0], lay.heads, lay.kv_heads
    bs = k_cache.shape[1]
    if _lib.use_kernels(proj, k_cache, v_cache, block_tables, context_lens):
        L = _lib.load()
        out = guard.empty(b, h * lay.vp, device=proj.device, dtype=proj.dtype)
        q = proj.view(-1)[lay.q_col:]
        if proj.dtype == torch.bfloat16 and (lay.qp, lay.vp) in TENSOR_CORE_HEADS:
            longest = min(int(max_context), window or chunk or int(max_context))
            n = nsplit or int(L.msrl_paged_decode_nsplit(c_int(b), c_int(g * ((h // g + 15) // 16)), c_int(longest)))
            part_o = _workspace("decode_part_o", b * h * n * lay.vp, proj.device)
            part_ml = _workspace("decode_part_ml", b * h * n * 2, proj.device)
            spec = (ctypes.c_longlong * 4)(proj.stride(0), 0, h, lay.qp)
            check(L.msrl_paged_decode_window(
                ptr(q), spec, ptr(k_cache), ptr(v_cache), ptr(block_tables), c_int(block_tables.shape[1]), ptr(context_lens),
                ptr(out), c_ll(h * lay.vp), ptr(part_o), ptr(part_ml), c_int(b), c_int(h), c_int(g), c_int(lay.qp), c_int(lay.vp),
                c_int(bs), c_float(scale), c_int(window or 0), c_int(chunk or 0), *form.args(), c_int(n), stream()),
                "paged_decode_window")
            return out
        ints = (ctypes.c_int * 9)(h, g, lay.qp, lay.vp, bs, block_tables.shape[1], window or 0, lay.qp, chunk or 0)
        check(L.msrl_paged_decode_simt(ptr(q), c_ll(proj.stride(0)), ptr(k_cache), ptr(v_cache), ptr(block_tables),
                                       ptr(context_lens), ptr(out), ints, c_int(b), c_float(scale), *form.args(), _is_f32(proj),
                                       stream()), "paged_decode_simt")
        return out
    q = lay.split(proj)[0].float()
    out = torch.zeros(b, h, lay.vp)
    for i in range(b):
        n = int(context_lens[i])
        pos = torch.arange(max(n - 1, 0) // chunk * chunk if chunk else max(0, n - (window or n)), n)
        at = block_tables[i, (pos // bs).long()].long() * bs + pos % bs
        k, v = (c.view(-1, *c.shape[2:])[at].float().repeat_interleave(h // g, dim=1) for c in (k_cache, v_cache))
        p = form.weights(torch.einsum("hd,jhd->hj", q[i], k) * scale)
        out[i] = torch.einsum("hj,jhd->hd", p, v)
    return form.gated(out).view(b, h * lay.vp).to(proj.dtype)
