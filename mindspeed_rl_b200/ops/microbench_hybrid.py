"""Micro-benchmark cases of the layer-by-layer decoders' kernels, at the layer sizes of a model of some ten billion
parameters (32 heads of 128, latent rank 512, width 2304).  Run through ``ops.microbench --only hybrid_*``.

Roofline of the recurrence: its state arithmetic is fp32 on the CUDA cores (4 multiply-adds per state entry and
token), counted against 128 fp32 multiply-adds per SM and clock at the maximum clock.
"""
from __future__ import annotations

import torch

from . import (ConvHeads, ConvNormWeights, DeltaLayout, DeltaWeights, GroupedHeads, GRULayout, LatentLayout, MemoryLayout,
               MemoryWeights, Norm, PassEntry, PostNorm, ScoreForm, TokenSide, WKVWeights, add_norm_, angle_table,
               conv_qkv_decode, conv_qkv_prefill, delta_decode, delta_prefill, embed_norm, glu_fwd, latent_decode_attention,
               latent_prefill_attention, latent_prep, latent_rotate_queries, latent_spread_, memory_decode, memory_prefill,
               min_gru_decode, min_gru_prefill, moe_combine_norm_, moe_post_add_, post_add_, post_embed, qkv_prep_, rope_table,
               rows_gather, soft_cap_, token_side_, turn_back, turned_prep_, window_decode_attention, window_prefill_attention,
               wkv_decode, wkv_mix_decode, wkv_mix_prefill, wkv_prefill)
from . import moe as K
from .matrix_memory import constant_decay
from .microbench import report, timeit


def fp32_tflops() -> float:
    p = torch.cuda.get_device_properties(0)
    clock = getattr(p, "clock_rate", 1965000) * 1e3
    return p.multi_processor_count * 128 * 2 * clock / 1e12


def _delta(t, heads=32, dim=128, vdim=128, taps=4, head_decay=False):
    kd, hv = heads * dim, heads * vdim
    na = heads if head_decay else kd
    lay = DeltaLayout(heads, heads, dim, vdim, taps, 0, kd, 2 * kd, 2 * kd + hv, head_decay=head_decay, silu_gate=head_decay)
    proj = torch.randn(t, 2 * kd + hv + heads + 256, device="cuda").bfloat16()
    a, gate = torch.randn(t, na, device="cuda").bfloat16(), torch.randn(t, hv, device="cuda").bfloat16()
    w = DeltaWeights(torch.randn(lay.channels, taps, device="cuda"), torch.zeros(heads, device="cuda") - 2,
                     torch.zeros(na, device="cuda"), torch.ones(vdim, device="cuda"))
    return lay, proj, a, gate, w


def case_head_delta(small: bool, iters: int):
    case_delta(small, iters, True)


def case_delta(small: bool, iters: int, head_decay: bool = False):
    kind = " decay per head" if head_decay else ""
    for b, n in ([(1, 2048)] if small else [(1, 8192), (8, 1024), (32, 256)]):
        t = b * n
        lay, proj, a, gate, w = _delta(t, head_decay=head_decay)
        ring = torch.zeros(b, lay.taps, lay.channels, device="cuda").bfloat16()
        state = torch.zeros(b, lay.heads, lay.dim, lay.vdim, device="cuda")
        cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
        seq = torch.arange(b, dtype=torch.int32, device="cuda").repeat_interleave(n)
        start, slots = torch.zeros(b, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda")
        ms = timeit(lambda: delta_prefill(proj, a, gate, lay, w, ring, state, seq, cu, start, slots, 1e-5), iters)
        fma = 4.0 * t * lay.heads * lay.dim * lay.vdim
        report(f"delta_prefill {b}x{n} heads=32 dim=128{kind}", ms, bytes_=2.0 * t * (lay.channels + 3 * lay.heads * lay.vdim),
               note=f"{2 * fma / ms / 1e9:.1f} TFLOP/s fp32 = {2 * fma / ms / 1e9 / fp32_tflops():.3f} of nominal fp32")
    for b in ([32] if small else [1, 32, 256]):
        lay, proj, a, gate, w = _delta(b, head_decay=head_decay)
        ring = torch.zeros(b, lay.taps, lay.channels, device="cuda").bfloat16()
        state = torch.zeros(b, lay.heads, lay.dim, lay.vdim, device="cuda")
        pos = torch.full((b,), 100, dtype=torch.int32, device="cuda")
        slots = torch.randperm(b, device="cuda")
        ms = timeit(lambda: delta_decode(proj, a, gate, lay, w, ring, state, pos, slots, 1e-5), iters)
        report(f"delta_decode B={b} heads=32 dim=128{kind}", ms, bytes_=2.0 * state.numel() * 4 + b * lay.channels * 2 * 8)


def case_latent(small: bool, iters: int):
    for heads in (16, 32, 64, 128):
        lay = LatentLayout(heads, 64, 64, 128, 512, 128, 128, heads * 128, 64)
        for b, ctx in ([(16, 1024)] if small else [(256, 2048), (32, 2048), (1, 8192)]):
            nb = b * ctx // 16
            cache = torch.randn(nb, 16, lay.CP, device="cuda").bfloat16()
            bt = torch.randperm(nb, device="cuda").to(torch.int32).view(b, -1)
            cl = torch.full((b,), ctx, dtype=torch.int32, device="cuda")
            q = torch.randn(b, heads, lay.CP, device="cuda").bfloat16()
            ms = timeit(lambda: latent_decode_attention(q, cache, lay, bt, cl, ctx, 0.05), iters)
            report(f"latent_decode H={heads} B={b} ctx={ctx}", ms, bytes_=2.0 * b * ctx * lay.CP,
                   flops=2.0 * b * ctx * heads * (lay.CP + lay.RP))
    heads, t, n = 32, (2048 if small else 16384), 2048
    for dn, dr, dv, p in ((64, 64, 128, 128), (128, 64, 128, 192)):
        lay = LatentLayout(heads, dn, dr, dv, 512, p, 128, heads * p, dr)
        proj = torch.randn(t, heads * p + 576, device="cuda").bfloat16()
        kv = torch.randn(t, heads * (p + 128), device="cuda").bfloat16()
        cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
        ms = timeit(lambda: latent_prefill_attention(proj, kv, lay, cu, cu, n, 0.08), iters)
        report(f"latent_prefill_attention {t // n}x{n} H=32 qk={dn + dr} v={dv}", ms,
               flops=2.0 * t * (n / 2) * heads * (dn + dr + dv))
        pos = torch.arange(t, dtype=torch.int32, device="cuda") % n
        slots = torch.arange(t, device="cuda")
        cache = torch.empty(t // 16, 16, lay.CP, device="cuda").bfloat16()
        tab = rope_table(4096, dr, 1e4, proj.device)
        nw = torch.ones(512, device="cuda")
        ms = timeit(lambda: latent_prep(proj, lay, nw, 1e-5, tab, pos, slots, cache, True), iters)
        report(f"latent_prep T={t} H=32 rot={dr}", ms, bytes_=2.0 * t * (2 * heads * dr + 3 * lay.CP))
        rows = torch.randn(t, lay.CP, device="cuda").bfloat16()
        ms = timeit(lambda: latent_spread_(kv, rows, lay), iters)
        report(f"latent_spread T={t} H=32 rot={dr}", ms, bytes_=2.0 * t * (heads * dr + dr))


def case_stream(small: bool, iters: int):
    t, h, f = (4096, 2304, 4096) if small else (16384, 3584, 18944)
    resid, w = torch.zeros(t, h, device="cuda"), torch.zeros(h, device="cuda")
    x = torch.randn(t, h, device="cuda").bfloat16()
    ms = timeit(lambda: add_norm_(resid, x, w, 1e-5, 1.0), iters)
    report(f"add_norm {t}x{h} (fp32 residual)", ms, bytes_=t * h * 12.0)
    table, ids = torch.randn(32768, h, device="cuda").bfloat16(), torch.randint(0, 32768, (t,), device="cuda")
    ms = timeit(lambda: embed_norm(ids, table, 1.0, w, 1e-5, 1.0), iters)
    report(f"embed_norm {t}x{h}", ms, bytes_=t * h * 8.0)
    for act in ("gelu_tanh", "clamped_swish"):
        gu = torch.randn(t, 2 * f, device="cuda").bfloat16()
        ms = timeit(lambda: glu_fwd(gu, act, 7.0, 1.702), iters)
        report(f"glu {act} {t}x{f}", ms, bytes_=6.0 * t * f)
        del gu
    e, k, h, f = 64, 8, 2304, 1024
    for t in ([2048] if small else [16384, 256]):
        x = torch.randn(t, h, device="cuda").bfloat16()
        idx = torch.stack([torch.randperm(e, device="cuda")[:k] for _ in range(256)]).repeat((t + 255) // 256, 1)[:t]
        plan = K.moe_plan(idx, e)
        w1, w2 = (torch.randn(e, n, c, device="cuda").bfloat16() for n, c in ((2 * f, h), (h, f)))
        xp = K.moe_permute(x, plan)
        ms = timeit(lambda: K.grouped_gemm_nt(xp, plan, w1), iters)
        report(f"grouped_gemm_nt w1 rows={t * k} E={e}", ms, bytes_=2.0 * w1.numel() + 2.0 * t * k * (h + 2 * f), flops=2.0 * t * k * h * 2 * f)
        gu = K.grouped_gemm_nt(xp, plan, w1)
        ms = timeit(lambda: glu_fwd(gu, "clamped_swish", 7.0, 1.702, plan=plan), iters)
        report(f"glu clamped_swish by expert rows={t * k} F={f}", ms, bytes_=6.0 * t * k * f)
        y = K.grouped_gemm_nt(glu_fwd(gu, "clamped_swish", 7.0, 1.702, plan=plan), plan, w2)
        resid, sh, sg = torch.zeros(t, h, device="cuda"), torch.randn(t, h, device="cuda").bfloat16(), torch.randn(h, device="cuda").bfloat16()
        w = torch.zeros(h, device="cuda")
        ms = timeit(lambda: moe_combine_norm_(resid, y, plan.pos, k, 1.0 / k, x, sh, sg, w, 1e-5, 1.0), iters)
        report(f"moe_combine_norm T={t} k={k} H={h}", ms, bytes_=t * h * (2.0 * k + 4 + 8 + 2))


def _memory(t, slots, heads, dim, vdim, retention=False):
    n = heads * (2 * dim + 2 * vdim)
    lay = MemoryLayout(heads, dim, vdim, vdim, 0, heads * dim, 2 * heads * dim, heads * (2 * dim + vdim), dim ** -0.5, 15.0,
                       silu_gate=retention)
    w = MemoryWeights(torch.zeros(2 * heads, device="cuda"), torch.ones(heads * vdim, device="cuda"),
                      constant_decay([0.99] * heads).cuda() if retention else None)
    state = {"memory": torch.zeros(slots, heads, dim, vdim, device="cuda"), "norm": torch.zeros(slots, heads, dim, device="cuda"),
             "peak": torch.zeros(slots, heads, device="cuda")}
    return lay, torch.randn(t, n, device="cuda").bfloat16(), torch.randn(t, 2 * heads, device="cuda"), w, state


def case_retention(small: bool, iters: int):
    case_memory(small, iters, True)


def case_memory(small: bool, iters: int, retention: bool = False):
    """Roofline of prompts: the rows read and written once (the recurrence's products are far below the tensor peak)."""
    kind = "retention" if retention else "memory"
    for heads, dim, vdim in ((32, 128, 128), (8, 256, 512)):
        for b, n in ([(1, 2048)] if small else [(1, 8192), (8, 1024), (32, 256)]):
            t = b * n
            lay, proj, z, w, state = _memory(t, b, heads, dim, vdim, retention)
            cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
            start, slots = torch.zeros(b, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda")
            ms = timeit(lambda: memory_prefill(proj, z, lay, w, state, cu, n, start, slots, 1e-5), iters)
            report(f"{kind}_prefill {b}x{n} heads={heads} {dim}x{vdim}", ms, bytes_=2.0 * t * heads * (2 * dim + 3 * vdim),
                   flops=4.0 * t * heads * dim * vdim)
        for b in ([32] if small else [1, 32, 256]):
            lay, proj, z, w, state = _memory(b, b, heads, dim, vdim, retention)
            pos, slots = torch.full((b,), 100, dtype=torch.int32, device="cuda"), torch.randperm(b, device="cuda")
            ms = timeit(lambda: memory_decode(proj, z, lay, w, state, pos, slots, 1e-5), iters)
            report(f"{kind}_decode B={b} heads={heads} {dim}x{vdim}", ms, bytes_=8.0 * state["memory"].numel())


def case_window(small: bool, iters: int):
    h, g, d = 32, 8, 128
    lay = GroupedHeads(h, g, d, d, d, d, 0, h * d, (h + g) * d)
    t, n = (2048, 2048) if small else (16384, 8192)
    for window in (None, 4096, 1024):
        proj = torch.randn(t, (h + 2 * g) * d, device="cuda").bfloat16()
        cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
        w = min(window or n, n)
        pairs = t // n * (w * (w + 1) / 2 + (n - w) * w)
        ms = timeit(lambda: window_prefill_attention(proj, lay, cu, cu, n, d ** -0.5, window), iters)
        report(f"window_prefill_attention {t // n}x{n} H={h}/{g} window={window}", ms, flops=4.0 * pairs * h * d)
    pos, slots = torch.arange(t, dtype=torch.int32, device="cuda") % n, torch.arange(t, device="cuda")
    kc, vc = (torch.empty(t // 16, 16, g, d, device="cuda").bfloat16() for _ in range(2))
    tab = angle_table(8192, tuple(1e4 ** (-i / 64) for i in range(64)), proj.device)
    qn, kn, mix = torch.ones(h * d, device="cuda"), torch.ones(g * d, device="cuda"), torch.full((1,), 0.3, device="cuda")
    other = lay.values(torch.randn_like(proj))
    ms = timeit(lambda: qkv_prep_(proj, lay, qn, kn, 1e-5, tab, pos, slots, kc, vc, other, mix), iters)
    report(f"qkv_prep T={t} H={h}/{g} d={d}", ms, bytes_=2.0 * t * d * (2 * h + 4 * g + 3 * g))
    bt = torch.randperm(t // 16, device="cuda").to(torch.int32).view(1, -1)
    seq, at = torch.zeros(t, dtype=torch.int32, device="cuda"), torch.arange(t, dtype=torch.int32, device="cuda")
    ms = timeit(lambda: rows_gather(kc, bt, seq, at), iters)
    report(f"rows_gather T={t} row={g * d}", ms, bytes_=4.0 * t * g * d)
    for b, ctx, window in ([(16, 1024, None)] if small else [(256, 2048, None), (256, 8192, 1024), (32, 8192, 4096), (1, 8192, 4096)]):
        nb = b * ctx // 16
        kc, vc = (torch.randn(nb, 16, g, d, device="cuda").bfloat16() for _ in range(2))
        bt = torch.randperm(nb, device="cuda").to(torch.int32).view(b, -1)
        cl = torch.full((b,), ctx, dtype=torch.int32, device="cuda")
        q = torch.randn(b, (h + 2 * g) * d, device="cuda").bfloat16()
        ms = timeit(lambda: window_decode_attention(q, lay, kc, vc, bt, cl, ctx, d ** -0.5, window), iters)
        report(f"window_decode H={h}/{g} B={b} ctx={ctx} window={window}", ms, bytes_=4.0 * b * min(ctx, window or ctx) * g * d)


def case_routed(small: bool, iters: int):
    """What scored experts in parallel layers add: router, weighted permutation, centred norm with the mixer's output."""
    e, k, h = 64, 8, 2304
    for t in ([2048] if small else [16384, 256]):
        x, z = torch.randn(t, h, device="cuda").bfloat16(), torch.randn(t, e, device="cuda")
        ms = timeit(lambda: K.route_top(z, k), iters)
        report(f"route_top T={t} E={e} k={k}", ms, bytes_=t * (4.0 * e + 12 * k))
        idx, score = K.route_top(z, k)
        plan = K.moe_plan(idx, e)
        ms = timeit(lambda: K.moe_permute(x, plan, score), iters)
        report(f"moe_permute weighted T={t} k={k} H={h}", ms, bytes_=2.0 * t * h * (k + 1))
        y, sh, mixer = torch.randn(plan.max_rows, h, device="cuda").bfloat16(), torch.randn_like(x), torch.randn_like(x)
        resid, w = torch.zeros(t, h, device="cuda"), torch.ones(h, device="cuda")
        ms = timeit(lambda: moe_combine_norm_(resid, y, plan.pos, k, 1.0, x, sh, None, w, 1e-5, 0.0, True, delta=mixer), iters)
        report(f"moe_combine_norm centred + mixer T={t} k={k} H={h}", ms, bytes_=t * h * (2.0 * k + 4 + 8 + 2))
        ms = timeit(lambda: add_norm_(resid, mixer, w, 1e-5, 0.0, True), iters)
        report(f"add_norm centred {t}x{h}", ms, bytes_=t * h * 12.0)


def case_conv(small: bool, iters: int):
    """Convolved attention in chunks: preparation, soft-capped and gated prompt attention, decode over a chunk."""
    h, g, d, size = 32, 8, 128, 1024
    heads = GroupedHeads(h, g, d, d, d, d, 0, h * d, (h + g) * d)
    lay = ConvHeads(heads, 4, 0, h * d, (h + g) * d)
    w = ConvNormWeights(torch.randn(lay.channels, 4, device="cuda"), torch.ones(d, device="cuda"), torch.ones(d, device="cuda"))
    tab = angle_table(8192, tuple(1e4 ** (-i / 32) for i in range(32)), "cuda")
    t, n = (2048, 2048) if small else (16384, 8192)
    b = t // n
    proj = torch.randn(t, lay.row + 32, device="cuda").bfloat16()
    gate = proj[:, lay.row:]
    pos, slots = torch.arange(t, dtype=torch.int32, device="cuda") % n, torch.arange(t, device="cuda")
    kc, vc = (torch.empty(t // 16, 16, g, d, device="cuda").bfloat16() for _ in range(2))
    ring = torch.zeros(256, 4, lay.channels, device="cuda").bfloat16()
    cu, seq = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda"), torch.arange(t, dtype=torch.int32, device="cuda") // n
    start, state = torch.zeros(b, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda")
    ms = timeit(lambda: conv_qkv_prefill(proj, lay, w, 1e-5, tab, pos, slots, kc, vc, ring, state, seq, cu, start), iters)
    report(f"conv_qkv_prefill T={t} H={h}/{g} d={d}", ms, bytes_=2.0 * t * d * (2 * h + 6 * g))
    for name, form, keys in (("plain", ScoreForm(), None), ("gated", ScoreForm(0.0, gate), None), ("capped and gated", ScoreForm(30.0, gate), None),
                             ("capped and gated", ScoreForm(30.0, gate), size)):
        cq = torch.arange(0, t + 1, keys or n, dtype=torch.int32, device="cuda")
        ms = timeit(lambda: window_prefill_attention(proj, heads, cq, cq, keys or n, d ** -0.5, None, form=form), iters)
        pairs = t * ((keys or n) + 1) / 2
        report(f"prompt attention {name} {b}x{n} H={h}/{g} chunk={keys}", ms, flops=4.0 * pairs * h * d,
               note=f"{ms * 1e6 / (pairs * h) * 1e3 * torch.cuda.get_device_properties(0).multi_processor_count:.1f} SM-ps per score")
    for b, ctx in ([(16, 1024)] if small else [(256, 2048), (32, 8192), (1, 8192)]):
        nb = b * ctx // 16
        kc, vc = (torch.randn(nb, 16, g, d, device="cuda").bfloat16() for _ in range(2))
        bt = torch.randperm(nb, device="cuda").to(torch.int32).view(b, -1)
        cl = torch.full((b,), ctx, dtype=torch.int32, device="cuda")
        pos, slots, state = cl - 1, bt[:, -1].long() * 16 + 15, torch.arange(b, device="cuda")
        x = proj[:b]
        ms = timeit(lambda: conv_qkv_decode(x, lay, w, 1e-5, tab, pos, slots, kc, vc, ring, state), iters)
        report(f"conv_qkv_decode B={b} H={h}/{g}", ms, bytes_=2.0 * b * (lay.channels * 6 + lay.row) + 16.0 * lay.channels)
        q = torch.randn(b, h * d, device="cuda").bfloat16()
        for chunk in (None, size):
            ms = timeit(lambda: window_decode_attention(q, heads, kc, vc, bt, cl, ctx, d ** -0.5, None, chunk=chunk,
                                                        form=ScoreForm(30.0, gate[:b])), iters)
            report(f"decode capped and gated H={h}/{g} B={b} ctx={ctx} chunk={chunk}", ms,
                   bytes_=4.0 * b * ((ctx - 1) % chunk + 1 if chunk else ctx) * g * d)


def case_gated_latent(small: bool, iters: int):
    """Latent attention with a query latent, half-split rotation, window, sink and gates."""
    for heads in (16, 32, 64):
        lay = LatentLayout(heads, 64, 64, 128, 512, 128, 128, 768, 64, True, 768, 0)
        for b, ctx, window in ([(16, 1024, None)] if small else [(256, 2048, None), (256, 2048, 1024), (32, 8192, 1024), (1, 8192, 1024)]):
            nb = b * ctx // 16
            cache = torch.randn(nb, 16, lay.CP, device="cuda").bfloat16()
            bt = torch.randperm(nb, device="cuda").to(torch.int32).view(b, -1)
            cl = torch.full((b,), ctx, dtype=torch.int32, device="cuda")
            q, gate = torch.randn(b, heads, lay.CP, device="cuda").bfloat16(), torch.randn(b, heads, device="cuda").bfloat16()
            form = ScoreForm(0.0, gate, torch.zeros(heads, device="cuda"))
            ms = timeit(lambda: latent_decode_attention(q, cache, lay, bt, cl, ctx, 0.05, window=window, form=form), iters)
            report(f"latent_decode gated, sink H={heads} B={b} ctx={ctx} window={window}", ms, bytes_=2.0 * b * min(ctx, window or ctx) * lay.CP)
    heads, t, n = 32, (2048 if small else 16384), 2048
    lay = LatentLayout(heads, 64, 64, 128, 512, 128, 128, 768, 64, True, 768, 0)
    proj = torch.randn(t, 768 + 576 + 32, device="cuda").bfloat16()
    q = torch.randn(t, heads * 128, device="cuda").bfloat16()
    pos, slots = torch.arange(t, dtype=torch.int32, device="cuda") % n, torch.arange(t, device="cuda")
    cache = torch.empty(t // 16, 16, lay.CP, device="cuda").bfloat16()
    tab, nw, qw = rope_table(4096, 64, 1e4, proj.device), torch.ones(512, device="cuda"), torch.ones(768, device="cuda")
    ms = timeit(lambda: latent_prep(proj, lay, nw, 1e-5, tab, pos, slots, cache, True, q_norm=qw), iters)
    report(f"latent_prep with query latent T={t}", ms, bytes_=2.0 * t * (2 * 768 + 3 * lay.CP))
    ms = timeit(lambda: latent_rotate_queries(q, lay, tab, pos), iters)
    report(f"latent_rotate_queries T={t} H={heads} rot=64", ms, bytes_=4.0 * t * heads * 64)
    kv = torch.randn(t, heads * 256, device="cuda").bfloat16()
    cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
    form = ScoreForm(0.0, proj[:, -32:], torch.zeros(heads, device="cuda"))
    for window in (None, 1024):
        ms = timeit(lambda: latent_prefill_attention(q, kv, lay, cu, cu, n, 0.08, window, form), iters)
        w = window or n
        report(f"latent_prefill_attention gated, sink {t // n}x{n} H=32 window={window}", ms,
               flops=4.0 * (t // n) * (w * (w + 1) / 2 + (n - w) * w) * heads * 128)


def case_post_norm(small: bool, iters: int):
    """Post-norm adds and the soft-max router."""
    e, k, h = 64, 8, 2304
    for t in ([2048] if small else [16384, 256]):
        z, corr = torch.randn(t, e + 8, device="cuda"), torch.zeros(e + 8, device="cuda")
        ms = timeit(lambda: K.route_softmax_top(z, corr, k), iters)
        report(f"route_softmax_top T={t} E={e + 8} k={k}", ms, bytes_=t * (4.0 * (e + 8) + 12 * k))
        idx, score = K.route_softmax_top(z, corr, k)
        plan = K.moe_plan(idx, e)
        x, y = torch.randn(t, h, device="cuda").bfloat16(), torch.randn(plan.max_rows, h, device="cuda").bfloat16()
        resid, w = torch.zeros(t, h, device="cuda"), torch.ones(h, device="cuda")
        post = PostNorm(w, 1e-5, 0.5)
        ms = timeit(lambda: K.moe_permute(x, plan), iters)
        report(f"moe_permute T={t} k={k} of {e} + 8 H={h}", ms, bytes_=2.0 * t * h * (k * e / (e + 8) + 1))
        ms = timeit(lambda: moe_post_add_(resid, y, plan.pos, score, post), iters)
        report(f"moe_post_add T={t} k={k} H={h}", ms, bytes_=t * h * (2.0 * k * e / (e + 8) + 8 + 2))
        ms = timeit(lambda: post_add_(resid, x, post), iters)
        report(f"post_add {t}x{h}", ms, bytes_=t * h * 12.0)


def case_wkv(small: bool, iters: int):
    """State arithmetic in fp32: three multiply-adds per state entry and token (decayed state, added product, output)."""
    heads, dim, rank, width = 64, 64, 64, 2304
    hd = heads * dim
    g = torch.Generator(device="cuda").manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    w = WKVWeights(torch.rand(5, width, device="cuda"), rnd(hd, rank).bfloat16() * 0.1, rnd(hd) - 3, rnd(hd), torch.ones(hd, device="cuda"), heads, dim)
    for b, n in ([(1, 2048)] if small else [(1, 8192), (8, 1024), (32, 256), (8, 2048)]):
        t = b * n
        r, k, v, gate = (rnd(t, hd).bfloat16() for _ in range(4))
        a, h = rnd(t, rank), rnd(t, width).bfloat16()
        state, last = torch.zeros(b, heads, dim, dim, device="cuda"), torch.zeros(b, width, device="cuda")
        cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
        seq = torch.arange(b, dtype=torch.int32, device="cuda").repeat_interleave(n)
        start, slots = torch.zeros(b, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda")
        ms = timeit(lambda: wkv_prefill(r, k, v, gate, a, w, state, cu, n, start, slots, 1e-5), iters)
        flops = 6.0 * t * heads * dim * dim
        report(f"wkv_prefill {b}x{n} heads={heads} dim={dim}", ms, bytes_=10.0 * t * hd + 4.0 * t * rank,
               note=f"{flops / ms / 1e9:.1f} TFLOP/s fp32 = {flops / ms / 1e9 / fp32_tflops():.3f} of nominal fp32")
        ms = timeit(lambda: wkv_mix_prefill(h, w.mu, last, seq, cu, start, slots), iters)
        report(f"wkv_mix T={t} W={width}", ms, bytes_=12.0 * t * width)
    for b in ([32] if small else [1, 32, 256]):
        r, k, v, gate = (rnd(b, hd).bfloat16() for _ in range(4))
        a, h = rnd(b, rank), rnd(b, width).bfloat16()
        state, last = torch.zeros(b, heads, dim, dim, device="cuda"), torch.zeros(b, width, device="cuda")
        pos, slots = torch.full((b,), 100, dtype=torch.int32, device="cuda"), torch.randperm(b, device="cuda")
        ms = timeit(lambda: wkv_decode(r, k, v, gate, a, w, state, pos, slots, 1e-5), iters)
        report(f"wkv_decode B={b} heads={heads} dim={dim}", ms, bytes_=8.0 * state.numel() + 10.0 * b * hd + 2.0 * hd * rank)
        ms = timeit(lambda: wkv_mix_decode(h, w.mu, last, pos, slots), iters)
        report(f"wkv_mix decode B={b} W={width}", ms, bytes_=20.0 * b * width)


def case_parallel(small: bool, iters: int):
    """Around the attention with turned values, and the gated recurrence beside it."""
    h, g, d, width = 32, 8, 128, 2304
    lay = GroupedHeads(h, g, d, d, d, d, 0, h * d, (h + g) * d)
    c0 = (h + 2 * g) * d
    gru = GRULayout(width, width, c0, c0 + width, c0 + 2 * width, h * d, 0.7)
    tab, vtab = (angle_table(8192, tuple(1e4 ** (-i / n) for i in range(n)), "cuda") for n in (32, 64))
    zb, xb = torch.zeros(width, device="cuda"), torch.zeros(width, device="cuda")
    for b, n in ([(1, 2048)] if small else [(1, 8192), (8, 2048)]):
        t = b * n
        proj = torch.randn(t, c0 + 3 * width, device="cuda").bfloat16()
        pos, slots = torch.arange(t, dtype=torch.int32, device="cuda") % n, torch.arange(t, device="cuda")
        kc, vc = (torch.empty(t // 16, 16, g, d, device="cuda").bfloat16() for _ in range(2))
        ms = timeit(lambda: turned_prep_(proj, lay, 1e-5, tab, vtab, pos, slots, kc, vc), iters)
        report(f"turned_prep T={t} H={h}/{g} d={d} rot=64", ms, bytes_=2.0 * t * (2 * (h + g) * 64 + 2 * g * d + g * 64 + 2 * g * d))
        attn, out = torch.randn(t, h * d, device="cuda").bfloat16(), torch.empty(t, h * d + width, device="cuda").bfloat16()
        ms = timeit(lambda: turn_back(attn, lay, vtab, pos, 0.7, out), iters)
        report(f"turn_back T={t} H={h} d={d}", ms, bytes_=4.0 * t * h * d)
        cu = torch.arange(0, t + 1, n, dtype=torch.int32, device="cuda")
        start, own, state = torch.zeros(b, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda"), torch.zeros(b, width, device="cuda")
        ms = timeit(lambda: min_gru_prefill(proj, gru, zb, xb, state, out, cu, n, start, own), iters)
        report(f"min_gru_prefill {b}x{n} width={width}", ms, bytes_=8.0 * t * width)
    for b in ([32] if small else [1, 256]):
        proj, out = torch.randn(b, c0 + 3 * width, device="cuda").bfloat16(), torch.empty(b, h * d + width, device="cuda").bfloat16()
        pos, own, state = torch.full((b,), 100, dtype=torch.int32, device="cuda"), torch.arange(b, device="cuda"), torch.zeros(b, width, device="cuda")
        slots, kc, vc = own * 16, *(torch.empty(b, 16, g, d, device="cuda").bfloat16() for _ in range(2))
        ms = timeit(lambda: turned_prep_(proj, lay, 1e-5, tab, vtab, pos, slots, kc, vc), iters)
        report(f"turned_prep decode B={b} H={h}/{g}", ms, bytes_=2.0 * b * (2 * (h + g) * 64 + 5 * g * d + g * 64))
        attn = torch.randn(b, h * d, device="cuda").bfloat16()
        ms = timeit(lambda: turn_back(attn, lay, vtab, pos, 0.7, out), iters)
        report(f"turn_back decode B={b} H={h}", ms, bytes_=4.0 * b * h * d)
        ms = timeit(lambda: min_gru_decode(proj, gru, zb, xb, state, out, pos, own), iters)
        report(f"min_gru_decode B={b} width={width}", ms, bytes_=16.0 * b * width)


def case_sandwich(small: bool, iters: int):
    """Norms around sublayers, token inputs, pass inputs, the router over the chosen and capped logits."""
    e, k, h, dim = 64, 8, 2304, 64
    table, rows = (torch.randn(32768, n, device="cuda").bfloat16() for n in (h, 4 * dim))
    w, step = torch.ones(h, device="cuda"), torch.ones(h, device="cuda")
    post, after = PostNorm(w, 1e-5), Norm(w, 1e-5)
    side = TokenSide(torch.randn(dim, h, device="cuda").bfloat16(), torch.randn(h, dim, device="cuda").bfloat16(), rows, dim, dim)
    for t in ([2048] if small else [16384, 256, 32, 1]):
        ids = torch.randint(0, 32768, (t,), device="cuda")
        x, resid, again = torch.randn(t, h, device="cuda").bfloat16(), torch.zeros(t, h, device="cuda"), torch.zeros(t, h, device="cuda")
        ms = timeit(lambda: post_embed(ids, table, post, after, True, step), iters)
        report(f"post_embed {t}x{h}", ms, bytes_=t * h * 12.0)
        ms = timeit(lambda: post_add_(resid, x, post, after), iters)
        report(f"post_add + norm {t}x{h}", ms, bytes_=t * h * 12.0)
        ms = timeit(lambda: post_add_(resid, x, post, after, PassEntry(again, step)), iters)
        report(f"post_add + pass input + norm {t}x{h}", ms, bytes_=t * h * 16.0)
        z = torch.randn(t, e, device="cuda")
        ms = timeit(lambda: K.route_top(z, k, True), iters)
        report(f"route_top over the chosen T={t} E={e} k={k}", ms, bytes_=t * (4.0 * e + 12 * k))
        idx, score = K.route_top(z, k, True)
        plan = K.moe_plan(idx, e)
        y = torch.randn(plan.max_rows, h, device="cuda").bfloat16()
        ms = timeit(lambda: moe_post_add_(resid, y, plan.pos, score, post), iters)
        report(f"moe_post_add T={t} k={k} H={h}", ms, bytes_=t * h * (2.0 * k + 8 + 2))
        for fused in ((0,) if t > 256 else (0, t)):
            ms = timeit(lambda: token_side_(resid, x, ids, side, post, after, fused_tokens=fused), iters)
            report(f"token_side{' gate in one kernel' if fused else ''} {t}x{h} dim={dim}", ms, bytes_=t * h * 16.0 + 4.0 * h * dim)
    logits = torch.randn(32 if small else 256, 151936, device="cuda").bfloat16()
    ms = timeit(lambda: soft_cap_(logits, 30.0), iters)
    report(f"soft_cap {logits.shape[0]}x151936", ms, bytes_=4.0 * logits.numel())


CASES = {"hybrid_retention": case_retention, "hybrid_wkv": case_wkv, "hybrid_parallel": case_parallel, "hybrid_sandwich": case_sandwich,
         "hybrid_conv": case_conv, "hybrid_gated_latent": case_gated_latent, "hybrid_head_delta": case_head_delta,
         "hybrid_post_norm": case_post_norm, "hybrid_memory": case_memory, "hybrid_window": case_window, "hybrid_routed": case_routed,
         "hybrid_delta": case_delta, "hybrid_latent": case_latent, "hybrid_stream": case_stream}
