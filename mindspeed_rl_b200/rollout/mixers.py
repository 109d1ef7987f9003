"""Token mixers of layer-by-layer decoders (``models.hybrid_config``) in the rollout engine.

A mixer owns the fused weights of one layer and reads / writes the carried state of one layer run through the
:class:`StepMeta` of the step.  ``prefill`` takes packed prompt portions, ``decode`` one token per sequence; both
return the mixer's output before the residual add.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, NamedTuple, Optional

import torch

from .. import ops
from ..models.hybrid_config import (ChannelDeltaSpec, Chunk, ConvAttentionSpec, HeadDeltaSpec, KeyRange, LatentAttentionSpec,
                                    MatrixMemorySpec, ParallelSpec, RetentionSpec, WKVSpec, WindowAttentionSpec)
from ..ops.conv_qkv import ConvHeads, ConvNormWeights
from ..ops.delta import DeltaLayout, DeltaWeights
from ..ops.gemm import linear_f32, linear_fwd
from ..ops.latent import LatentLayout, pad16
from ..ops.matrix_memory import MemoryLayout, MemoryWeights, constant_decay
from ..ops.min_gru import GRULayout
from ..ops.window import GroupedHeads, ValueSource
from ..ops.wkv import WKVWeights


class KeySpan(NamedTuple):
    """Queries and keys of a prompt step as packed sequences of one attention call (a layer that sees chunks has a
    sequence per chunk)."""
    cu_q: torch.Tensor
    cu_k: torch.Tensor
    max_q: int
    cached: Optional[dict] = None           # block_tables, token_seq, token_pos of the keys; None: the step's own rows


@dataclass
class StepMeta:
    """Where the tokens of a step sit: shared by all layers of the step."""
    ids: torch.Tensor                       # [T] int64
    positions: torch.Tensor                 # [T] int32
    slots: torch.Tensor                     # [T] int64 cache row of every token (-1: none)
    state_slots: torch.Tensor               # [B] int64 recurrent-state slot of every sequence (-1: none)
    max_model_len: int
    # prompt portions
    cu_q: Optional[torch.Tensor] = None     # [B + 1] int32
    max_q: int = 0
    tok_seq: Optional[torch.Tensor] = None  # [T] int32
    start_pos: Optional[torch.Tensor] = None  # [B] int32 position of a portion's first token
    spans: Optional[Dict[KeyRange, KeySpan]] = None     # where a key range needs more than the packed portions
    # decode steps
    block_tables: Optional[torch.Tensor] = None
    context_lens: Optional[torch.Tensor] = None
    max_context: int = 0
    # values of the first layer that mixes values, kept for the later ones of the step
    first_values: Optional[ValueSource] = None

    def span_of(self, keys: KeyRange) -> KeySpan:
        span = None if self.spans is None else self.spans.get(keys)
        return span or KeySpan(self.cu_q, self.cu_q, self.max_q)

    @property
    def is_decode(self) -> bool:
        return self.block_tables is not None


def _pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    if w.shape[0] == rows:
        return w
    return torch.cat([w, w.new_zeros(rows - w.shape[0], *w.shape[1:])])


def _pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    if w.shape[-1] == cols:
        return w
    return torch.cat([w, w.new_zeros(*w.shape[:-1], cols - w.shape[-1])], dim=-1)


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad_heads(w: torch.Tensor, heads: int, dim: int, to: int) -> torch.Tensor:
    """Rows (or entries) of ``heads`` heads of ``dim``, each head zero padded to ``to``."""
    if dim == to:
        return w
    x = w.reshape(heads, dim, *w.shape[1:])
    return torch.cat([x, x.new_zeros(heads, to - dim, *w.shape[1:])], dim=1).reshape(heads * to, *w.shape[1:])


def _table_rows(meta: StepMeta) -> int:
    """Length of rotation tables: whole powers of two, so that engines with different length limits share them."""
    return 1 << max(meta.max_model_len - 1, 1).bit_length()


def stack_sections(parts: List[torch.Tensor]):
    """Rows of several projections of one input as one weight; every section starts on a multiple of eight
    columns of the product (zero rows in between).  Returns the weight and the section starts."""
    cols, start, padded = [], 0, []
    for p in parts:
        cols.append(start)
        padded.append(_pad_rows(p, _pad8(p.shape[0])))
        start += padded[-1].shape[0]
    return torch.cat(padded).contiguous(), cols


class LatentAttention:
    """Heads are padded to a size the tensor-core attention kernels serve (zero rows and columns in the weights,
    so that the products are unchanged); other sizes and fp32 run unpadded on the CUDA cores."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        h, dn, dr, dv, r = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
        qp, vp = dn + dr, dv
        if dtype == torch.bfloat16 and vp <= 128 and qp <= 192:
            vp = 64 if max(qp, vp) <= 64 else 128
            qp = 192 if qp > 128 else vp

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        q = w["uq" if spec.q_rank else "q"]
        q = _pad_cols(q.view(h, dn + dr, -1).transpose(1, 2), qp).transpose(1, 2).reshape(h * qp, -1)
        fused, cols = stack_sections([w["dq"] if spec.q_rank else q, w["dkv"]] + ([w["g"]] if spec.head_gate else []))
        self.lay = lay = LatentLayout(h, dn, dr, dv, r, qp, vp, cols[1], spec.rot.dims, spec.rot.halves, spec.q_rank or 0, cols[0])
        if spec.q_rank:
            self.w_uq = put(_pad_cols(q, lay.QP))
            self.q_norm = put(w["dq.norm"], torch.float32)
        self.g_cols = slice(cols[2], cols[2] + h) if spec.head_gate else None
        self.sink = put(w["sink"].reshape(-1), torch.float32) if spec.sink else None
        uk = _pad_cols(w["uk"], lay.RP).view(h, dn, lay.RP)
        uv = _pad_cols(w["uv"], lay.RP).view(h, dv, lay.RP)
        k_rows = torch.cat([uk, uk.new_zeros(h, qp - dn, lay.RP)], dim=1)
        v_rows = torch.cat([uv, uv.new_zeros(h, vp - dv, lay.RP)], dim=1)
        self.w_in = put(fused)
        self.w_kv = put(torch.cat([k_rows.reshape(h * qp, lay.RP), v_rows.reshape(h * vp, lay.RP)]))
        self.w_k = self.w_kv[:h * qp].view(h, qp, lay.RP)[:, :dn]       # [H, dn, RP]: folds W_uk into the query
        self.w_v = self.w_kv[h * qp:].view(h, vp, lay.RP)               # [H, vp, RP]
        self.w_o = put(_pad_cols(w["o"].view(-1, h, dv), vp).reshape(-1, h * vp))
        self.norm = put(w["dkv.norm"], torch.float32)

    def _form(self, proj: torch.Tensor) -> ops.ScoreForm:
        return ops.ScoreForm(0.0, None if self.g_cols is None else proj[:, self.g_cols], self.sink)

    def _queries(self, proj: torch.Tensor, meta: StepMeta, stored: torch.Tensor, want_rows: bool, decode_q=None):
        """Rows that begin with the prepared query heads, and the step's cache rows."""
        lay, rot = self.lay, self.spec.rot
        table = ops.rope_table(_table_rows(meta), rot.dims, rot.base, self.w_in.device)
        args = (proj, lay, self.norm, self.eps, table, meta.positions, meta.slots, stored, want_rows)
        if not lay.q_rank:
            return proj, ops.latent_prep(*args, decode_q=decode_q)
        rows, cq = ops.latent_prep(*args, q_norm=self.q_norm)
        q = linear_fwd(cq, self.w_uq)
        ops.latent_rotate_queries(q, lay, table, meta.positions, decode_q)
        return q, rows

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        lay, spec, span, stored = self.lay, self.spec, meta.span_of(self.spec.keys), cache.rows[run]["latent"]
        proj = linear_fwd(x, self.w_in)
        q, rows = self._queries(proj, meta, stored, want_rows=span.cached is None)
        if span.cached is not None:
            rows = ops.latent_gather(stored, **span.cached)
        kv = linear_fwd(rows[:, :lay.RP], self.w_kv)
        ops.latent_spread_(kv, rows, lay)
        attn = ops.latent_prefill_attention(q, kv, lay, span.cu_q, span.cu_k, span.max_q, spec.scale, spec.window, self._form(proj))
        return linear_fwd(attn, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        lay, b, stored = self.lay, x.shape[0], cache.rows[run]["latent"]
        proj = linear_fwd(x, self.w_in)
        q = torch.empty(b, lay.heads, lay.CP, dtype=x.dtype, device=x.device)
        heads, _ = self._queries(proj, meta, stored, want_rows=False, decode_q=q)
        heads = heads[:, :lay.heads * lay.qp].view(b, lay.heads, lay.qp)
        torch.bmm(heads[..., :lay.dn].transpose(0, 1), self.w_k, out=q[..., :lay.RP].transpose(0, 1))
        lat = ops.latent_decode_attention(q, stored, lay, meta.block_tables, meta.context_lens, meta.max_context, self.spec.scale,
                                          window=self.spec.window, form=self._form(proj))
        attn = torch.empty(b, lay.heads, lay.vp, dtype=x.dtype, device=x.device)
        torch.bmm(lat.transpose(0, 1), self.w_v.transpose(1, 2), out=attn.transpose(0, 1))
        return linear_fwd(attn.view(b, lay.heads * lay.vp), self.w_o)


class ChannelDelta:
    """Decays and the output gate come through bottlenecks of two products."""
    head_decay = silu_gate = False

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        decay, gate = self._inputs(w)
        fused, cols = stack_sections([w["q"], w["k"], w["v"], w["b"], decay, gate])
        self.lay = DeltaLayout(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.conv, *cols[:4], unit_eps=spec.unit_eps,
                               head_decay=self.head_decay, silu_gate=self.silu_gate)
        self.a_cols, self.g_cols = (slice(c, c + _pad8(p.shape[0])) for c, p in ((cols[4], decay), (cols[5], gate)))

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        f32 = torch.float32
        self.w_in = put(fused)
        self._outputs(w, put)
        self.w_o = put(w["o"])
        self.state = DeltaWeights(conv=put(torch.cat([w["q.conv"], w["k.conv"], w["v.conv"]]), f32),
                                  a_log=put(w["A_log"], f32), dt_bias=put(w["dt_bias"], f32), norm=put(w["norm"], f32))
        if self.state.conv.shape != (self.lay.channels, spec.conv):
            raise ValueError(f"convolution weights {tuple(self.state.conv.shape)} do not fit {spec}")

    def _inputs(self, w):
        return w["a1"], w["g1"]

    def _outputs(self, w, put):
        self.w_a2 = put(_pad_cols(w["a2"], _pad8(w["a1"].shape[0])))
        self.w_g2 = put(_pad_cols(w["g2"], _pad8(w["g1"].shape[0])))

    def _project(self, x: torch.Tensor):
        proj = linear_fwd(x, self.w_in)
        return proj, linear_fwd(proj[:, self.a_cols], self.w_a2), linear_fwd(proj[:, self.g_cols], self.w_g2)

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        proj, a, gate = self._project(x)
        y = ops.delta_prefill(proj, a, gate, self.lay, self.state, cache.slots[run]["ring"], cache.slots[run]["state"], meta.tok_seq,
                              meta.cu_q, meta.start_pos, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        proj, a, gate = self._project(x)
        y = ops.delta_decode(proj, a, gate, self.lay, self.state, cache.slots[run]["ring"], cache.slots[run]["state"], meta.positions,
                             meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)


class HeadDelta(ChannelDelta):
    """One decay per head; decays and the output gate are sections of the fused projection."""
    head_decay = silu_gate = True

    def _inputs(self, w):
        return w["a"], w["g"]

    def _outputs(self, w, put):
        pass

    def _project(self, x: torch.Tensor):
        proj, s = linear_fwd(x, self.w_in), self.spec
        return proj, proj[:, self.a_cols][:, :s.heads], proj[:, self.g_cols][:, :s.heads * s.vdim]


def _cached_kv(rows: Dict[str, torch.Tensor], span: KeySpan):
    """Keys and values that a prompt step looks at, or None where they are its own rows."""
    return None if span.cached is None else tuple(ops.rows_gather(rows[n], **span.cached) for n in ("k", "v"))


class WindowAttention:
    """Grouped-head attention over a window of paged keys and values.  Heads are stored padded (``padded_heads``):
    zero rows and columns in the weights, so that sums of squares and products are unchanged."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        h, g = spec.heads, spec.kv_heads
        qp, vp = spec.padded(dtype)
        f32 = torch.float32

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        def pad(t, heads, dim, to):
            return _pad_heads(t, heads, dim, to)

        parts = [(w["q"], w["q.b"], h, spec.dim, qp), (w["k"], w["k.b"], g, spec.dim, qp), (w["v"], w["v.b"], g, spec.vdim, vp)]
        fused, cols = stack_sections([pad(t, n, d, p) for t, _, n, d, p in parts])
        bias = torch.zeros(fused.shape[0], dtype=w["q.b"].dtype)
        for c, (_, b, n, d, p) in zip(cols, parts):
            bias[c:c + n * p] = pad(b, n, d, p)
        self.lay = GroupedHeads(h, g, spec.dim, spec.vdim, qp, vp, *cols)
        self.w_in, self.b_in = put(fused), put(bias)
        self.q_norm = put(pad(w["q.norm"], h, spec.dim, qp), f32)
        self.k_norm = put(pad(w["k.norm"], g, spec.dim, qp), f32)
        self.mix = put(w["vmix"].reshape(1), f32) if spec.value_mix else None
        if not spec.value_mix and "vmix" in w:
            w["vmix"]                                                   # stored but without a use
        self.w_o = put(_pad_cols(w["o"].reshape(-1, h, spec.vdim), vp).reshape(-1, h * vp))

    def _project(self, x: torch.Tensor, meta: StepMeta, rows: Dict[str, torch.Tensor]) -> torch.Tensor:
        """Normed, rotated and mixed q | k | v rows, written to the cache."""
        lay, spec = self.lay, self.spec
        proj = linear_fwd(x, self.w_in, self.b_in)
        table = ops.angle_table(_table_rows(meta), spec.rot.frequencies(), x.device)
        first = meta.first_values if spec.value_mix else None
        ops.qkv_prep_(proj, lay, self.q_norm, self.k_norm, self.eps, table, meta.positions, meta.slots, rows["k"], rows["v"],
                      first, self.mix)
        if spec.value_mix and first is None:
            meta.first_values = lay.values(proj)
        return proj

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        rows, span, spec = cache.rows[run], meta.span_of(self.spec.keys), self.spec
        proj = self._project(x, meta, rows)
        attn = ops.window_prefill_attention(proj, self.lay, span.cu_q, span.cu_k, span.max_q, spec.scale, spec.window,
                                            _cached_kv(rows, span))
        return linear_fwd(attn, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        rows, spec = cache.rows[run], self.spec
        proj = self._project(x, meta, rows)
        attn = ops.window_decode_attention(proj, self.lay, rows["k"], rows["v"], meta.block_tables, meta.context_lens,
                                           meta.max_context, spec.scale, spec.window)
        return linear_fwd(attn, self.w_o)


class ConvAttention:
    """Short convolutions, per-head norms and rotation between the projection and grouped-head attention.  The projection's
    heads are stored as they are; prepared rows and the cache hold them padded (``padded_heads``)."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        h, g = spec.heads, spec.kv_heads
        qp, vp = spec.padded(dtype)

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        fused, cols = stack_sections([w["q"], w["k"], w["v"], w["g"]])
        self.heads = GroupedHeads(h, g, spec.dim, spec.vdim, qp, vp, 0, h * qp, (h + g) * qp)
        self.lay = ConvHeads(self.heads, spec.conv, *cols[:3])
        self.g_cols = slice(cols[3], cols[3] + h)
        self.w_in = put(fused)
        f32 = torch.float32
        self.prep = ConvNormWeights(put(torch.cat([w["q.conv"], w["k.conv"], w["v.conv"]]), f32), put(w["q.norm"], f32),
                                    put(w["k.norm"], f32))
        if self.prep.conv.shape != (spec.channels, spec.conv):
            raise ValueError(f"convolution weights {tuple(self.prep.conv.shape)} do not fit {spec}")
        self.w_o = put(_pad_cols(w["o"].reshape(-1, h, spec.vdim), vp).reshape(-1, h * vp))

    def _prepare(self, prep, x, meta: StepMeta, cache, run: int, *where):
        proj, rows = linear_fwd(x, self.w_in), cache.rows[run]
        table = ops.angle_table(_table_rows(meta), self.spec.rot.frequencies(), x.device)
        out = prep(proj, self.lay, self.prep, self.eps, table, meta.positions, meta.slots, rows["k"], rows["v"],
                   cache.slots[run]["ring"], meta.state_slots, *where)
        return out, rows, ops.ScoreForm(self.spec.softcap, proj[:, self.g_cols])

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        spec, span = self.spec, meta.span_of(self.spec.keys)
        qkv, rows, form = self._prepare(ops.conv_qkv_prefill, x, meta, cache, run, meta.tok_seq, meta.cu_q, meta.start_pos)
        attn = ops.window_prefill_attention(qkv, self.heads, span.cu_q, span.cu_k, span.max_q, spec.scale,
                                            None if isinstance(spec.keys, Chunk) else spec.keys, _cached_kv(rows, span), form=form)
        return linear_fwd(attn, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        keys = self.spec.keys
        q, rows, form = self._prepare(ops.conv_qkv_decode, x, meta, cache, run)
        attn = ops.window_decode_attention(q, self.heads, rows["k"], rows["v"], meta.block_tables, meta.context_lens,
                                           meta.max_context, self.spec.scale, None if isinstance(keys, Chunk) else keys,
                                           chunk=keys.size if isinstance(keys, Chunk) else None, form=form)
        return linear_fwd(attn, self.w_o)


class MatrixMemory:
    """Head rows are padded to multiples of 16 (zero rows: padded keys and values leave the memory's padding zero);
    gate logits are a product of their own with a 32-bit result."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        h, d, dv = spec.heads, spec.dim, spec.vdim
        dp, vp = pad16(d), pad16(dv)

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        fused, cols = stack_sections([_pad_heads(w["q"], h, d, dp), _pad_heads(w["k"], h, d, dp),
                                      _pad_heads(w["v"], h, dv, vp), _pad_heads(w["g"], h, dv, vp)])
        self.lay = MemoryLayout(h, dp, vp, dv, *cols, scale=d ** -0.5, cap=spec.gate_cap, floor=spec.floor)
        self.w_in, self.w_gates = put(fused), put(torch.cat([w["i"], w["f"]]))
        self.memory = MemoryWeights(bias=put(torch.cat([w["i.b"], w["f.b"]]), torch.float32),
                                    norm=put(_pad_heads(w["norm"], h, dv, vp), torch.float32))
        self.w_o = put(_pad_cols(w["o"].reshape(-1, h, dv), vp).reshape(-1, h * vp))

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        y = ops.memory_prefill(linear_fwd(x, self.w_in), linear_f32(x, self.w_gates), self.lay, self.memory, cache.slots[run],
                               meta.cu_q, meta.max_q, meta.start_pos, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        y = ops.memory_decode(linear_fwd(x, self.w_in), linear_f32(x, self.w_gates), self.lay, self.memory, cache.slots[run],
                              meta.positions, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)


class Retention:
    """The matrix memory with a constant decay per head in place of its gates, no denominator and a silu output gate."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        h, d, dv = spec.heads, spec.dim, spec.vdim
        dp, vp = pad16(d), pad16(dv)

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        fused, cols = stack_sections([_pad_heads(w["q"], h, d, dp), _pad_heads(w["k"], h, d, dp),
                                      _pad_heads(w["v"], h, dv, vp), _pad_heads(w["g"], h, dv, vp)])
        self.lay = MemoryLayout(h, dp, vp, dv, *cols, scale=d ** -0.5, silu_gate=True)
        self.w_in = put(fused)
        self.memory = MemoryWeights(bias=None, norm=torch.ones(h * vp, device=device),
                                    decay=put(constant_decay(spec.decay), torch.float32))
        self.w_o = put(_pad_cols(w["o"].reshape(-1, h, dv), vp).reshape(-1, h * vp))

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        y = ops.memory_prefill(linear_fwd(x, self.w_in), None, self.lay, self.memory, cache.slots[run], meta.cu_q, meta.max_q,
                               meta.start_pos, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        y = ops.memory_decode(linear_fwd(x, self.w_in), None, self.lay, self.memory, cache.slots[run], meta.positions,
                              meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)


class ParallelMixer:
    """Attention with turned values and a minimal gated recurrence on one input.  All projections are one product; both
    sides write their scaled results next to each other, so that their output projections and the sum are one product too."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps
        s, n = spec.left, spec.right.width
        h, g = s.heads, s.kv_heads
        qp, vp = s.padded(dtype)

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        fused, cols = stack_sections([_pad_heads(w["left.q"], h, s.dim, qp), _pad_heads(w["left.k"], g, s.dim, qp),
                                      _pad_heads(w["left.v"], g, s.vdim, vp), w["right.z"], w["right.x"], w["right.g"]])
        self.heads = GroupedHeads(h, g, s.dim, s.vdim, qp, vp, *cols[:3])
        self.gru = GRULayout(n, _pad8(n), *cols[3:], out_col=h * vp, scale=spec.right_scale)
        self.w_in = put(fused)
        self.z_bias, self.x_bias = (put(w[f"right.{i}.b"].reshape(-1), torch.float32) for i in "zx")
        left = _pad_cols(w["left.o"].reshape(-1, h, s.vdim), vp).reshape(-1, h * vp)
        self.w_o = put(torch.cat([left, _pad_cols(w["right.o"], _pad8(n))], dim=1))

    def _prepare(self, x: torch.Tensor, meta: StepMeta, rows: Dict[str, torch.Tensor]):
        s = self.spec.left
        proj = linear_fwd(x, self.w_in)
        table, values = (ops.angle_table(_table_rows(meta), r.frequencies(), x.device) for r in (s.rot, s.value_rot))
        ops.turned_prep_(proj, self.heads, self.eps, table, values, meta.positions, meta.slots, rows["k"], rows["v"])
        return proj, values

    def _finish(self, attn: torch.Tensor, proj: torch.Tensor, values: torch.Tensor, meta: StepMeta, cache, run: int):
        out = torch.empty(proj.shape[0], self.w_o.shape[1], dtype=proj.dtype, device=proj.device)
        ops.turn_back(attn, self.heads, values, meta.positions, self.spec.left_scale, out)
        args = (proj, self.gru, self.z_bias, self.x_bias, cache.slots[run]["state"], out)
        if meta.is_decode:
            ops.min_gru_decode(*args, meta.positions, meta.state_slots)
        else:
            ops.min_gru_prefill(*args, meta.cu_q, meta.max_q, meta.start_pos, meta.state_slots)
        return linear_fwd(out, self.w_o)

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        rows, span = cache.rows[run], meta.span_of(self.spec.keys)
        proj, values = self._prepare(x, meta, rows)
        attn = ops.window_prefill_attention(proj, self.heads, span.cu_q, span.cu_k, span.max_q, self.spec.left.scale, None,
                                            _cached_kv(rows, span))
        return self._finish(attn, proj, values, meta, cache, run)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        rows = cache.rows[run]
        proj, values = self._prepare(x, meta, rows)
        attn = ops.window_decode_attention(proj, self.heads, rows["k"], rows["v"], meta.block_tables, meta.context_lens,
                                           meta.max_context, self.spec.left.scale, None)
        return self._finish(attn, proj, values, meta, cache, run)


class WKV:
    """Projections read mixes of neighbouring tokens, a row of its own each; those of equal shape are one batched product in
    small steps.  The decay's bottleneck has 32-bit results."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], eps: float, dtype, device):
        self.spec, self.eps = spec, eps

        def put(t, dt=dtype):
            return t.to(device=device, dtype=dt).contiguous()

        f32 = torch.float32
        self.w_in = put(torch.stack([w[n] for n in "rkvg"]))                   # [4, heads * dim, W]
        self.w1 = put(w["w1"])
        self.wkv = WKVWeights(mu=put(torch.stack([w["mu." + n].reshape(-1) for n in "rkvgw"]), f32), w2=put(w["w2"]),
                              w0=put(w["w0"].reshape(-1), f32), u=put(w["u"].reshape(-1), f32), norm=put(w["norm"].reshape(-1), f32),
                              heads=spec.heads, dim=spec.dim)
        self.w_o = put(w["o"])

    def _project(self, mixed: torch.Tensor):
        a = linear_f32(mixed[4], self.w1)
        if mixed.shape[1] > 128:
            return [linear_fwd(x, w) for x, w in zip(mixed, self.w_in)], a
        return torch.bmm(mixed[:4], self.w_in.transpose(1, 2)).unbind(), a

    def prefill(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        slots = cache.slots[run]
        rkvg, a = self._project(ops.wkv_mix_prefill(x, self.wkv.mu, slots["last"], meta.tok_seq, meta.cu_q, meta.start_pos,
                                                    meta.state_slots))
        y = ops.wkv_prefill(*rkvg, a, self.wkv, slots["state"], meta.cu_q, meta.max_q, meta.start_pos, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)

    def decode(self, x: torch.Tensor, meta: StepMeta, cache, run: int) -> torch.Tensor:
        slots = cache.slots[run]
        rkvg, a = self._project(ops.wkv_mix_decode(x, self.wkv.mu, slots["last"], meta.positions, meta.state_slots))
        y = ops.wkv_decode(*rkvg, a, self.wkv, slots["state"], meta.positions, meta.state_slots, self.eps)
        return linear_fwd(y, self.w_o)


MIXERS = {LatentAttentionSpec: LatentAttention, ChannelDeltaSpec: ChannelDelta, HeadDeltaSpec: HeadDelta,
          WindowAttentionSpec: WindowAttention, ConvAttentionSpec: ConvAttention, MatrixMemorySpec: MatrixMemory,
          RetentionSpec: Retention, ParallelSpec: ParallelMixer, WKVSpec: WKV}
