"""Inference forward of the rollout engine over a paged KV cache.

The runner owns no parameters: ``RolloutWeights`` is a set of tensors (views into the reshard
arena, or aliases of the training parameters when the layouts coincide) re-bound before every
rollout phase (reference contract: ``VLLMInferEngine.sync_model_weights``,
``mindspeed_rl/models/rollout/vllm_engine.py:381-405``).

Two entry points: ``prefill`` (packed prompt chunks, varlen attention, KV written to the cache)
and ``decode`` (one token per sequence, paged attention).  Decode steps are replayed from CUDA
graphs captured per batch-size bucket; all graph inputs live in static buffers.

Decoders that are composed layer by layer (``models.hybrid_config``) bind ``HybridWeights`` and a
``HybridCache`` instead; they run through the same two entry points, graphs and buffers, with an
fp32 residual stream and the mixers and feed-forwards of ``rollout.mixers`` / ``rollout.feed_forward``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..models.transformer_config import TransformerConfig
from ..ops import QKVLayout
from ..ops.gemm import linear_fwd
from ..parallel.tp_comm import NO_TP, TPComm
from .layer_cache import HybridCache
from .mixers import StepMeta


@dataclass
class LayerWeights:
    input_norm: torch.Tensor
    qkv_w: torch.Tensor
    qkv_b: Optional[torch.Tensor]
    o_w: torch.Tensor
    post_norm: torch.Tensor
    gate_up_w: Optional[torch.Tensor] = None
    down_w: Optional[torch.Tensor] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    moe: Optional[object] = None      # rollout.moe.MoEWeights for expert layers
    mla: Optional[object] = None      # models.mla.MLASelfAttention of a latent-attention layer (replaces qkv_w)


@dataclass
class RolloutWeights:
    embed: torch.Tensor
    layers: List[LayerWeights]
    final_norm: torch.Tensor
    lm_head: torch.Tensor
    qkv_layout: QKVLayout
    vocab_start: int = 0

    def signature(self):
        """Addresses of what captured graphs read."""
        return (self.embed.data_ptr(), self.lm_head.data_ptr(),
                tuple((l.qkv_w if l.qkv_w is not None else l.o_w).data_ptr() for l in self.layers))


class KVCache:
    def __init__(self, num_layers: int, num_blocks: int, block_size: int, nkv: int, hd: int,
                 dtype, device):
        shape = (num_layers, num_blocks, block_size, nkv, hd)
        # uninitialised on the GPU: a slot is always written before any attention reads it, and
        # zero-filling tens of GB costs ~10 ms per rollout phase.  (The CPU reference path
        # gathers whole blocks, so it keeps the zero fill.)
        alloc = torch.empty if torch.device(device).type == "cuda" else torch.zeros
        self.k = alloc(shape, dtype=dtype, device=device)
        self.v = alloc(shape, dtype=dtype, device=device)
        self.num_blocks, self.block_size = num_blocks, block_size

    @staticmethod
    def bytes_per_block(num_layers, block_size, nkv, hd, dtype) -> int:
        return 2 * num_layers * block_size * nkv * hd * torch.empty(0, dtype=dtype).element_size()

    def copy_block(self, src: int, dst: int) -> None:
        self.k[:, dst].copy_(self.k[:, src])
        self.v[:, dst].copy_(self.v[:, src])


class ModelRunner:
    def __init__(self, cfg: TransformerConfig, device, comm: Optional[TPComm] = None,
                 max_model_len: int = 4096, enforce_eager: bool = True,
                 graph_batch_sizes: Tuple[int, ...] = ()):
        self.cfg = cfg
        self.device = torch.device(device)
        self.comm = comm or NO_TP
        self.max_model_len = max_model_len
        self.enforce_eager = enforce_eager or self.device.type != "cuda"
        self.graph_batch_sizes = tuple(sorted(graph_batch_sizes))
        self.weights: Optional[RolloutWeights] = None
        self.cache: Optional[KVCache] = None
        self._rope = None
        self._graphs: Dict[tuple, dict] = {}
        self._static: Optional[dict] = None
        if cfg.is_hybrid and self.comm.world_size > 1:
            raise NotImplementedError(f"{cfg.architecture} is served on one GPU per replica (tensor parallel size 1)")
        self._side = None         # second stream of captured decode steps
        self.layer_probe = None   # callable(run, residual [T, W] fp32) after every layer run of a hybrid decoder (eager steps)
        self.prefix_tile = 0      # key tile of the tcgen05 shared-prefix kernel (set by the engine; 0 = mma.sync kernel)

    # ------------------------------------------------------------------------------------------
    def bind_weights(self, weights: Optional[RolloutWeights]) -> None:
        """(Re)bind parameters; graphs stay valid as long as the tensors keep their addresses."""
        old = self.weights
        self.weights = weights
        if weights is None or old is None or old.signature() != weights.signature():
            self._graphs.clear()

    def bytes_per_block(self, block_size: int) -> int:
        c = self.cfg
        if c.is_hybrid:
            return HybridCache.bytes_per_block(c, block_size)
        return KVCache.bytes_per_block(c.num_layers, block_size, c.num_query_groups // self.comm.world_size, c.head_dim,
                                       c.params_dtype)

    def make_cache(self, num_blocks: int, block_size: int, num_slots: int):
        """The cache of this model: paged K / V, or what the layers of a hybrid decoder carry (``num_slots``
        sequences at most keep recurrent state)."""
        c = self.cfg
        if c.is_hybrid:
            return HybridCache(c, num_blocks, block_size, num_slots, self.device)
        return KVCache(c.num_layers, num_blocks, block_size, c.num_query_groups // self.comm.world_size, c.head_dim,
                       c.params_dtype, self.device)

    def bind_cache(self, cache: Optional[KVCache]) -> None:
        self.cache = cache
        self._graphs.clear()
        self._static = None

    def rope_table(self) -> torch.Tensor:
        if self._rope is None:
            c = self.cfg
            self._rope = ops.rope_table(max(c.max_position_embeddings, self.max_model_len), c.head_dim,
                                        c.rotary_base, self.device, c.rope_scaling)
        return self._rope

    # ------------------------------------------------------------------------------------------
    def _embed(self, ids: torch.Tensor) -> torch.Tensor:
        w = self.weights
        if self.comm.world_size == 1:
            return w.embed[ids]
        local = ids - w.vocab_start
        mine = (local >= 0) & (local < w.embed.shape[0])
        h = w.embed[local.clamp(0, w.embed.shape[0] - 1)] * mine.unsqueeze(-1).to(w.embed.dtype)
        return self.comm.all_reduce(h)

    def _layer(self, li: int, lw: LayerWeights, resid, delta, positions, attend, rope_tab=None):
        cfg = self.cfg
        x, _, resid = ops.rmsnorm_fwd(delta, lw.input_norm, cfg.norm_epsilon, residual=resid,
                                      want_rstd=False) if resid is not None else \
            (*ops.rmsnorm_fwd(delta, lw.input_norm, cfg.norm_epsilon, want_rstd=False)[:2], delta)
        lay = self.weights.qkv_layout
        if lw.mla is not None:
            # latent attention: full per-head q / k / v (rotary and soft-max scale already applied)
            qkv = lw.mla.rollout_qkv(x, positions)
        else:
            qkv = linear_fwd(x, lw.qkv_w, lw.qkv_b)
            if lw.q_norm is not None:
                ops.headnorm_fwd_(qkv, lay, "q", lw.q_norm, cfg.norm_epsilon)
                ops.headnorm_fwd_(qkv, lay, "k", lw.k_norm, cfg.norm_epsilon)
            ops.rope_(qkv, lay, positions, self.rope_table() if rope_tab is None else rope_tab)
        attn = attend(li, qkv, lay)
        delta = self.comm.all_reduce(linear_fwd(attn, lw.o_w))
        x, _, resid = ops.rmsnorm_fwd(delta, lw.post_norm, cfg.norm_epsilon, residual=resid,
                                      want_rstd=False)
        if lw.moe is not None:
            delta = lw.moe.forward(x, self.comm)
        else:
            y = ops.swiglu_fwd(linear_fwd(x, lw.gate_up_w))
            delta = self.comm.all_reduce(linear_fwd(y, lw.down_w))
        return resid, delta

    @torch.no_grad()
    def idle_forward(self) -> None:
        """The collective part of a forward for a rank that has no tokens this step: every expert
        layer joins its group's token exchange with zero tokens (and serves the other ranks' tokens
        that are routed to its experts)."""
        empty = torch.zeros(0, self.cfg.hidden_size, dtype=self.cfg.params_dtype, device=self.device)
        for lw in self.weights.layers:
            if lw.moe is not None:
                lw.moe.forward(empty, self.comm)

    def _forward(self, ids, positions, attend, mm: Optional[dict] = None) -> torch.Tensor:
        """Returns the final hidden states ``[T, H]`` (after the last norm).  ``mm`` (vision-language
        prompts): ``image_index`` / ``image_embeds`` replace placeholder embeddings, ``rope_table [T, d]``
        is the per-token rotary table of three-axis positions (``positions`` then numbers the tokens)."""
        w = self.weights
        resid, delta = None, self._embed(ids)
        rope_tab = None
        if mm is not None:
            if mm.get("image_index") is not None and mm["image_index"].numel():
                delta = delta.index_copy(0, mm["image_index"], mm["image_embeds"].to(delta.dtype))
            rope_tab = mm.get("rope_table")
        for li, lw in enumerate(w.layers):
            resid, delta = self._layer(li, lw, resid, delta, positions, attend, rope_tab)
        x, _, _ = ops.rmsnorm_fwd(delta, w.final_norm, self.cfg.norm_epsilon, residual=resid,
                                  want_rstd=False)
        return x

    def _forward_hybrid(self, meta: StepMeta) -> torch.Tensor:
        """Final hidden states ``[T, H]`` of a layer-by-layer decoder: the fp32 residual is updated in place by
        kernels that add and take the next norm in one pass."""
        w, c, cache = self.weights, self.cfg, self.cache
        order, parallel = c.run_order, c.design.parallel
        if c.design.post_norm:
            return self._forward_post_norm(meta)
        if c.design.sandwich:
            return self._forward_sandwich(meta)

        def norm(weight):
            return ops.Norm(weight, c.norm_epsilon, c.design.norm_offset, c.design.centered)

        resid, x = ops.embed_norm(meta.ids, w.embed, c.embedding_scale, *norm(w.layers[order[0]].norm1))
        for run, li in enumerate(order):
            lw = w.layers[li]
            after = norm(w.layers[order[run + 1]].norm1 if run + 1 < len(order) else w.final_norm)
            mix = lw.mixer.decode if meta.is_decode else lw.mixer.prefill
            if parallel and lw.ff is not None:
                join = self._beside(meta, lambda: lw.ff.forward(x, meta.ids))
                delta = mix(x, meta, cache, run)
                x = lw.ff.finish_(resid, x, join(), after, delta)
            elif lw.ff is not None:
                x = ops.add_norm_(resid, mix(x, meta, cache, run), *norm(lw.norm2))
                x = lw.ff.finish_(resid, x, lw.ff.forward(x, meta.ids), after)
            else:
                x = ops.add_norm_(resid, mix(x, meta, cache, run), *after)
            if self.layer_probe is not None:
                self.layer_probe(run, resid)
        return x

    def _forward_post_norm(self, meta: StepMeta) -> torch.Tensor:
        """The same for designs that norm what a sublayer gives: sublayers read the residual itself (in the activation
        type), and one kernel norms, scales and adds their output."""
        w, c, cache = self.weights, self.cfg, self.cache
        order = c.run_order
        resid, x = ops.embed(meta.ids, w.embed, c.embedding_scale)
        for run, li in enumerate(order):
            lw = w.layers[li]
            post1, post2 = (None if n is None else ops.PostNorm(n, c.norm_epsilon, c.residual_mult) for n in (lw.norm1, lw.norm2))
            after = ops.Norm(w.final_norm, c.norm_epsilon) if run + 1 == len(order) else None
            mix = lw.mixer.decode if meta.is_decode else lw.mixer.prefill
            x = ops.post_add_(resid, mix(x, meta, cache, run), post1, after if lw.ff is None else None)
            if lw.ff is not None:
                x = lw.ff.finish_post_(resid, lw.ff.forward(x, meta.ids), post2, after)
            if self.layer_probe is not None:
                self.layer_probe(run, resid)
        return x

    def _forward_sandwich(self, meta: StepMeta) -> torch.Tensor:
        """The same for designs with a norm before and one after each sublayer, token inputs behind the layers and inputs of
        a loop's passes: the kernel that adds a layer's last term also adds what the next pass starts with and takes the
        next norm."""
        w, c, cache = self.weights, self.cfg, self.cache
        order, starts = c.run_order, c.pass_starts if c.design.loop_input else {}

        def norm(weight):
            return ops.Norm(weight, c.norm_epsilon)

        def post(weight):
            return ops.PostNorm(weight, c.norm_epsilon)

        resid, first, x = ops.post_embed(meta.ids, w.embed, post(w.embed_norm), norm(w.layers[order[0]].norm1),
                                         keep=len(starts) > 1, step=w.loop_step[starts[0]] if 0 in starts else None)
        for run, li in enumerate(order):
            lw = w.layers[li]
            after = norm(w.layers[order[run + 1]].norm1 if run + 1 < len(order) else w.final_norm)
            entry = None
            if run + 1 in starts:
                t = starts[run + 1]
                entry = ops.PassEntry(first if t else None, w.loop_step[t])
            mix = lw.mixer.decode if meta.is_decode else lw.mixer.prefill
            d, last = mix(x, meta, cache, run), (after, entry)
            nothing = (None, None)
            if lw.ff is not None:
                x = ops.post_add_(resid, d, post(lw.post1), norm(lw.norm2))
                x = lw.ff.finish_post_(resid, lw.ff.forward(x, meta.ids), post(lw.post2), *(nothing if lw.side else last))
            else:
                x = ops.post_add_(resid, d, post(lw.post1), *(nothing if lw.side else last))
            if lw.side is not None:
                x = ops.token_side_(resid, x, meta.ids, lw.side, post(lw.side_norm), *last)
            if self.layer_probe is not None:
                self.layer_probe(run, resid if entry is None else resid - entry.step - (0.0 if entry.again is None else entry.again))
        return x

    def _beside(self, meta: StepMeta, work):
        """Start ``work`` beside what the caller launches next; the returned function waits for it and gives its
        result.  Small decode steps leave most of the machine idle, so there the two run on two streams (inside
        a capture the fork and the join become edges of the graph); elsewhere one after the other."""
        if not (meta.is_decode and meta.ids.is_cuda and torch.cuda.is_current_stream_capturing()):
            return work
        main = torch.cuda.current_stream()
        if self._side is None:
            self._side = torch.cuda.Stream(self.device)
        side = self._side
        side.wait_stream(main)
        with torch.cuda.stream(side):
            out = work()

        def join():
            main.wait_stream(side)
            return out
        return join

    def _logits(self, x: torch.Tensor) -> torch.Tensor:
        y, cap = linear_fwd(x, self.weights.lm_head), getattr(self.cfg, "logit_softcap", 0.0)
        return ops.soft_cap_(y, cap) if cap else y

    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def prefill(self, ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                cu_q: torch.Tensor, max_q: int, last_index: torch.Tensor,
                prefix: Optional[dict] = None, mm: Optional[dict] = None,
                state: Optional[dict] = None) -> torch.Tensor:
        """Run packed prompt chunks. ``last_index`` selects the rows whose logits are needed.

        ``prefix`` (for chunks that start inside a sequence) carries ``block_tables``,
        ``token_seq``, ``token_pos``, ``cu_k``: the K/V of ``[0, chunk_end)`` is gathered from the
        cache after this chunk's K/V has been written.  Hybrid decoders get a ``KeySpan`` per key range of their
        attention layers (``HybridConfig.windows``) that lists only the keys inside the range.

        ``state`` (hybrid decoders): ``token_seq [T]`` and ``start_pos [B]`` (int32), ``slots [B]`` (int64, the
        recurrent-state slot of every sequence).
        """
        cache = self.cache
        if self.cfg.is_hybrid:
            meta = StepMeta(ids, positions, slots, state["slots"], self.max_model_len, cu_q=cu_q, max_q=max_q,
                            tok_seq=state["token_seq"], start_pos=state["start_pos"], spans=prefix)
            return self._logits(self._forward_hybrid(meta)[last_index])

        def attend(li, qkv, lay):
            ops.kv_cache_write(qkv, lay, slots, cache.k[li], cache.v[li])
            if prefix is None:
                out, _ = ops.attn_varlen_fwd(qkv, lay, cu_q, max_q, causal=True)
                return out
            k, v = ops.kv_cache_gather(cache.k[li], cache.v[li], prefix["block_tables"],
                                       prefix["token_seq"], prefix["token_pos"])
            out, _ = ops.attn_varlen_fwd(qkv, lay, cu_q, max_q, causal=True, kv=(k, v),
                                         cu_seqlens_k=prefix["cu_k"])
            return out

        x = self._forward(ids, positions, attend, mm)
        return self._logits(x[last_index])

    # ------------------------------------------------------------------------------------------
    def _decode_eager(self, ids, positions, slots, block_tables, context_lens, max_context, groups=None,
                      state_slots=None):
        cache = self.cache
        if self.cfg.is_hybrid:
            meta = StepMeta(ids, positions, slots, state_slots, self.max_model_len, block_tables=block_tables,
                            context_lens=context_lens, max_context=max_context)
            return self._logits(self._forward_hybrid(meta))

        def attend(li, qkv, lay):
            ops.kv_cache_write(qkv, lay, slots, cache.k[li], cache.v[li])
            return ops.paged_decode_attention(qkv, lay, cache.k[li], cache.v[li], block_tables,
                                              context_lens, max_context, groups=groups,
                                              prefix_tile=self.prefix_tile if groups is not None else 0)

        return self._logits(self._forward(ids, positions, attend))

    def _ensure_static(self, max_blocks: int) -> dict:
        cap = self.graph_batch_sizes[-1]
        st = self._static
        if st is None or st["block_tables"].shape[1] < max_blocks:
            dev = self.device
            st = dict(ids=torch.zeros(cap, dtype=torch.int64, device=dev),
                      positions=torch.zeros(cap, dtype=torch.int32, device=dev),
                      slots=torch.full((cap,), -1, dtype=torch.int64, device=dev),
                      block_tables=torch.zeros(cap, max_blocks, dtype=torch.int32, device=dev),
                      context_lens=torch.zeros(cap, dtype=torch.int32, device=dev),
                      state_slots=torch.full((cap,), -1, dtype=torch.int64, device=dev),
                      key_start=torch.zeros(cap, dtype=torch.int32, device=dev),
                      group_rows=torch.full((cap, 8), -1, dtype=torch.int32, device=dev),
                      group_prefix=torch.zeros(cap, dtype=torch.int32, device=dev))
            self._static = st
            self._graphs.clear()
        return st

    @torch.no_grad()
    def decode(self, ids: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
               block_tables: torch.Tensor, context_lens: torch.Tensor, max_context: int,
               groups=None, state_slots: Optional[torch.Tensor] = None) -> torch.Tensor:
        """One token per sequence -> logits ``[B, V_local]``.  ``groups`` (see
        ``ops.paged_decode_attention``; an optional fourth entry gives the number of groups that have
        members, which come first in the tables) turns on shared-prefix attention for n-sample groups.
        Shared prefixes must be multiples of ``self.prefix_tile`` keys when that is non-zero.  ``state_slots``
        ``[B]``: the recurrent-state slot of every sequence (hybrid decoders)."""
        b = ids.shape[0]
        bucket = next((s for s in self.graph_batch_sizes if s >= b), None)
        n_groups = b
        if groups is not None:
            if len(groups) > 3:
                # the shared pass launches one CTA per listed group: list a power of two that covers the real ones
                n_groups = min(b, 1 << max(0, int(groups[3]) - 1).bit_length())
            groups = tuple(groups[:3])
        if self.enforce_eager or bucket is None:
            if groups is not None:
                groups = (groups[0], groups[1][:n_groups], groups[2][:n_groups])
            return self._decode_eager(ids, positions, slots, block_tables, context_lens, max_context, groups,
                                      state_slots)
        max_blocks = (self.max_model_len + self.cache.block_size - 1) // self.cache.block_size
        st = self._ensure_static(max_blocks)
        st["ids"][:b].copy_(ids)
        st["positions"][:b].copy_(positions)
        st["slots"][:b].copy_(slots)
        st["slots"][b:bucket].fill_(-1)
        st["context_lens"][:b].copy_(context_lens)
        st["context_lens"][b:bucket].zero_()
        st["block_tables"][:b, :block_tables.shape[1]].copy_(block_tables)
        if state_slots is not None:
            st["state_slots"][:b].copy_(state_slots)
            st["state_slots"][b:bucket].fill_(-1)
        grouped = groups is not None
        if grouped:
            st["key_start"][:b].copy_(groups[0])
            st["key_start"][b:bucket].zero_()
            st["group_rows"][:b].copy_(groups[1])
            st["group_rows"][b:bucket].fill_(-1)
            st["group_prefix"][:b].copy_(groups[2])
        n_groups = min(n_groups, bucket) if grouped else 0
        g = self._graphs.get((bucket, grouped, n_groups))
        if g is None:
            g = self._capture(bucket, st, grouped, n_groups)
        g["graph"].replay()
        return g["logits"][:b]

    def _capture(self, bucket: int, st: dict, grouped: bool = False, n_groups: int = 0) -> dict:
        groups = (st["key_start"][:bucket], st["group_rows"][:n_groups], st["group_prefix"][:n_groups]) if grouped else None
        args = (st["ids"][:bucket], st["positions"][:bucket], st["slots"][:bucket],
                st["block_tables"][:bucket], st["context_lens"][:bucket], self.max_model_len, groups,
                st["state_slots"][:bucket])
        # the warm-up runs the step for real: a recurrent state must not advance twice, so it sees no state slots
        live = st["state_slots"].clone()
        st["state_slots"].fill_(-1)
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):       # warm-up: sizes scratch buffers outside the capture
            self._decode_eager(*args)
        torch.cuda.current_stream().wait_stream(side)
        st["state_slots"].copy_(live)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            logits = self._decode_eager(*args)
        rec = dict(graph=graph, logits=logits)
        self._graphs[(bucket, grouped, n_groups)] = rec
        return rec
