"""Gapevik decoders through the rollout engine against the plain restatement in ``gapevik_oracle`` (fp64).

Every test runs on the CPU formulation; the same tests run on the CUDA kernels on a GPU machine, in true 32-bit and,
where it makes sense, in bf16 with a tolerance of bf16 rounding.
"""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gapevik_models as M
import gapevik_oracle as O
from hybrid_helpers import TOL, close, dtypes, make_engine, run_schedule
from mindspeed_rl_b200 import ops
from mindspeed_rl_b200.models import registry
from mindspeed_rl_b200.models.hybrid_config import Chunk, HybridConfig, first_key
from mindspeed_rl_b200.ops import moe as K
from mindspeed_rl_b200.rollout.engine import LLMEngine
from mindspeed_rl_b200.rollout.hybrid_weights import build_hybrid_weights
from mindspeed_rl_b200.rollout.scheduler import SamplingParams

CUDA = pytest.param("cuda", marks=pytest.mark.gpu)
DEVICES = ["cpu", CUDA]


@functools.lru_cache(maxsize=None)
def _weights(name, seed=0):
    return M.weights(M.ZOO[name], seed)


@functools.lru_cache(maxsize=None)
def _expected(name, n, seed=0):
    """Oracle logits of the first ``n`` tokens of a fixed sequence."""
    return O.forward(M.ZOO[name], _weights(name), M.tokens(n, M.ZOO[name]["vocab"], seed))


def engine(name, device, dtype=torch.float32, **kw):
    return make_engine(M.ZOO[name], _weights(name), device, dtype, **kw)


def close_routed(got, want, dtype=torch.float32, share=0.85):
    """bf16 may turn close calls of a router with random weights, so most positions count, not the worst one."""
    if dtype == torch.float32:
        return close(got, want)
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float((err < TOL[dtype]).double().mean()) >= share, err.sort().values[-8:]


def _pad(x, to):
    return torch.nn.functional.pad(x, (0, to - x.shape[-1]))


# ---- norms of what a sublayer gives -----------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [40, 42, 1100, 9000])
@pytest.mark.parametrize("last", [False, True])
def test_post_norm_adds(device, width, last):
    g = torch.Generator().manual_seed(3)
    t, top = 5, 3
    for dtype in dtypes(device):
        tol = 2e-6 if dtype == torch.float32 else 6e-3
        x, d = torch.randn(t, width, generator=g) * 3, torch.randn(t, width, generator=g).to(dtype) * 0.2
        w, aw = (1.0 + 0.3 * torch.randn(width, generator=g) for _ in range(2))
        rows, score = torch.randn(7, width, generator=g).to(dtype), torch.rand(t, top, generator=g)
        pos = torch.tensor([[0, 3, -1], [6, -1, 2], [-1, -1, -1], [5, 4, 1], [-1, 0, 6]], dtype=torch.int32)
        post, after = ops.PostNorm(w.to(device), 1e-2, 0.3), ops.Norm(aw.to(device), 1e-3) if last else None
        mixed = sum(score[:, j:j + 1].double() * torch.where((pos[:, j] < 0)[:, None], x.double(), rows[pos[:, j].clamp(min=0).long()].double())
                    for j in range(top))
        for what, sub in (("rows", d.double()), ("experts", mixed)):
            resid = x.clone().to(device)
            if what == "rows":
                y = ops.post_add_(resid, d.to(device), post, after)
            else:
                y = ops.moe_post_add_(resid, rows.to(device), pos.reshape(-1).to(device), score.to(device), post, after)
            want = x.double() + 0.3 * O.rms(sub, 1e-2) * w.double()
            close(resid, want, tol=2e-6)
            close(y, O.rms(want, 1e-3) * aw.double() if last else want, tol=tol)
            assert y.dtype == dtype and y.data_ptr() != resid.data_ptr()
        table, ids = torch.randn(9, width, generator=g).to(dtype), torch.tensor([3, 0, 8, 8, 1])
        resid, y = ops.embed(ids.to(device), table.to(device), 2.5)
        close(resid, table[ids].double() * 2.5, tol=1e-6)
        close(y, table[ids].double() * 2.5, tol=tol)
    tiny = torch.full((1, width), 1e-3)                    # eps inside the root
    resid = torch.zeros(1, width, device=device)
    ops.post_add_(resid, tiny.to(device), ops.PostNorm(torch.ones(width, device=device), 1e-4, 1.0))
    close(resid, tiny.double() / (1e-6 + 1e-4) ** 0.5, tol=1e-5)


# ---- experts ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,identity,top", [(1, 0, 1), (3, 4, 7), (29, 4, 4), (200, 7, 8), (700, 1, 3)])
def test_router_and_identity_rows(device, experts, identity, top):
    g = torch.Generator().manual_seed(experts)
    t, n = 19, experts + identity
    z, corr = torch.randn(t, n, generator=g) * 2, torch.randn(n, generator=g) * 0.3
    z[3] += 80.0                                           # the soft-max does not see a common offset
    idx, score = K.route_softmax_top(z.to(device), corr.to(device), top)
    changed = 0
    for i in range(t):
        s = torch.softmax(z[i].double(), -1)
        want = O.choose(s, corr.double(), top)
        assert idx[i].cpu().tolist() == want
        assert torch.allclose(score[i].cpu().double(), s[want], rtol=1e-5)         # the correction is not in the weights
        changed += want != O.choose(s, torch.zeros(n), top)
    assert changed > 0 or n == 1
    same = torch.zeros(2, n)
    idx0, _ = K.route_softmax_top(same.to(device), torch.zeros(n, device=device), top)
    assert idx0.cpu().tolist() == [list(range(top))] * 2   # equal ones: the lower first
    plan = K.moe_plan(idx, experts)
    pos = plan.pos.cpu().view(t, top)
    real = idx.cpu() < experts
    assert bool(((pos >= 0) == real).all())
    assert plan.counts.cpu().tolist() == [int((idx == e).sum()) for e in range(experts)]
    assert len(set(pos[real].tolist())) == int(real.sum())
    for dtype in dtypes(device):
        for h in (16, 12, 7):
            x = torch.randn(t, h, generator=g).to(device, dtype)
            rows = K.moe_permute(x, plan)
            got = rows[plan.pos.long().clamp(min=0)].view(t, top, h).cpu()
            assert torch.equal(got[real], x.cpu()[:, None].expand(t, top, h)[real])


# ---- convolution, head norms, rotation, cache write ---------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,d,dv,taps,qp,vp,rot", [(4, 2, 12, 8, 3, 12, 8, 8), (3, 3, 7, 5, 4, 8, 8, 6), (5, 1, 72, 100, 2, 128, 128, 40),
                                                     (2, 2, 40, 24, 1, 64, 64, 40), (2, 1, 136, 20, 5, 192, 128, 2), (9, 3, 64, 64, 4, 64, 64, 64)])
def test_convolution_norm_rotation_and_cache(device, h, g, d, dv, taps, qp, vp, rot):
    """Two sequences in portions around the number of taps, then token by token, in slots that held something else."""
    n, gen = 31, torch.Generator().manual_seed(d)
    rots = {"dims": rot, "base": 60.0}
    lay = ops.ConvHeads(ops.GroupedHeads(h, g, d, dv, qp, vp, 0, h * qp, (h + g) * qp), taps, 8, 8 + h * d + 3, 16 + (h + g) * d)
    if d % 4 == 0:
        lay = ops.ConvHeads(lay.out, taps, 8, 8 + h * d + 4, 16 + (h + g) * d)
    table = ops.angle_table(64, tuple(60.0 ** (-2 * i / rot) for i in range(rot // 2)), "cpu").to(device)
    wide = -(-(lay.v_col + g * dv + 5) // 8) * 8
    for dtype in dtypes(device):
        proj = torch.randn(2 * n, wide, generator=gen).to(dtype)
        conv = torch.randn(lay.channels, taps, generator=gen)
        qn, kn = torch.rand(d, generator=gen) + 0.5, torch.rand(d, generator=gen) + 0.5
        w = ops.ConvNormWeights(conv.to(device), qn.to(device), kn.to(device))
        want = []
        for s in range(2):
            x = proj[s * n:(s + 1) * n].double()
            q, k, v = (x[:, c:c + m * e] for c, m, e in ((lay.q_col, h, d), (lay.k_col, g, d), (lay.v_col, g, dv)))
            cw = conv.double().split([h * d, g * d, g * dv])
            q, k, v = (O.short_conv(u, c).view(n, -1, e) for u, c, e in zip((q, k, v), cw, (d, d, dv)))
            want.append((O.rotate_pairs(O.rms(q, 1e-2) * qn.double(), rots), O.rotate_pairs(O.rms(k, 1e-2) * kn.double(), rots), v))
        fill = float("nan") if device == "cuda" else 7.0
        ring = torch.full((4, taps, lay.channels), fill, device=device, dtype=dtype)
        kc, vc = (torch.zeros(2 * n // 4 + 1, 4, g, p, device=device, dtype=dtype) for p in (qp, vp))
        tol = 2e-6 if dtype == torch.float32 else 6e-3
        owner, at = [2, 0], [0, 0]

        def check(y, s, pos, whole=True):
            q = y[:h * qp].view(h, qp).float().cpu()
            close(q[:, :d], want[s][0][pos], tol=tol)
            if whole:
                kk, vv = y[h * qp:(h + g) * qp].view(g, qp).float().cpu(), y[(h + g) * qp:].view(g, vp).float().cpu()
                close(kk[:, :d], want[s][1][pos], tol=tol)
                close(vv[:, :dv], want[s][2][pos], tol=tol)
                assert float(q[:, d:].abs().sum() + kk[:, d:].abs().sum() + vv[:, dv:].abs().sum()) == 0

        for cut in ([taps - 1, 1], [1, taps], [2, 3], [taps + 1, 2], [9, 1]):
            rows = torch.cat([torch.arange(s * n + at[s], s * n + at[s] + cut[s]) for s in range(2)])
            pos = torch.cat([torch.arange(at[s], at[s] + cut[s]) for s in range(2)]).to(torch.int32)
            y = ops.conv_qkv_prefill(proj[rows].to(device), lay, w, 1e-2, table, pos.to(device), rows.to(device), kc, vc, ring,
                                     torch.tensor(owner, device=device), torch.tensor([0] * cut[0] + [1] * cut[1], dtype=torch.int32, device=device),
                                     torch.tensor([0, cut[0], sum(cut)], dtype=torch.int32, device=device),
                                     torch.tensor(at, dtype=torch.int32, device=device))
            for i, r in enumerate(rows.tolist()):
                check(y[i], r // n, r % n)
            at = [a + c for a, c in zip(at, cut)]
        while min(at) < n:                                 # one row of every step is not in use
            live = [s for s in range(2) if at[s] < n]
            rows = torch.tensor([s * n + at[s] for s in live] + [0])
            pos = torch.tensor([at[s] for s in live] + [5], dtype=torch.int32, device=device)
            y = ops.conv_qkv_decode(proj[rows].to(device), lay, w, 1e-2, table, pos, torch.tensor(rows.tolist()[:-1] + [-1], device=device),
                                    kc, vc, ring, torch.tensor([owner[s] for s in live] + [-1], device=device))
            for i, s in enumerate(live):
                check(y[i], s, at[s], whole=False)
                at[s] += 1
        flat_k, flat_v = kc.float().cpu().view(-1, g, qp), vc.float().cpu().view(-1, g, vp)
        for s in range(2):
            for p in range(n):
                close(flat_k[s * n + p, :, :d], want[s][1][p], tol=tol)
                close(flat_v[s * n + p, :, :dv], want[s][2][p], tol=tol)
        assert float(flat_k[..., d:].abs().sum() + flat_v[..., dv:].abs().sum() + flat_k[2 * n:].abs().sum()) == 0


# ---- latents -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,dn,dr,rank,qr,qp", [(3, 12, 8, 24, 20, 20), (2, 5, 6, 19, 13, 11), (4, 64, 64, 80, 48, 128), (2, 8, 4, 16, 12, 12)])
def test_latents_and_half_split_rotation(device, h, dn, dr, rank, qr, qp):
    t, gen = 9, torch.Generator().manual_seed(rank)
    dkv, dq = -(-qr // 8) * 8, 0
    lay = ops.LatentLayout(h, dn, dr, 8, rank, qp, 8, dkv, dr, True, qr, dq)
    rot, pos = {"dims": dr, "base": 30.0}, torch.tensor([0, 1, 2, 9, 40, 41, 7, 3, 63], dtype=torch.int32)
    table = ops.rope_table(64, dr, 30.0, "cpu").to(device)
    slots = torch.tensor([5, -1, 0, 7, 12, 3, 2, 1, 4])
    for dtype in dtypes(device):
        tol = 2e-5 if dtype == torch.float32 else 6e-3
        proj = torch.randn(t, dkv + -(-(rank + dr) // 8) * 8, generator=gen).to(dtype)
        nw, qw = torch.rand(rank, generator=gen) + 0.5, torch.rand(qr, generator=gen) + 0.5
        cache = torch.zeros(4, 4, lay.CP, device=device, dtype=dtype)
        rows, cq = ops.latent_prep(proj.to(device), lay, nw.to(device), 1e-2, table, pos.to(device), slots.to(device), cache, True,
                                   q_norm=qw.to(device))
        x = proj.double()

        def turn(y, i):                                    # rotation of one row at its position
            full = torch.zeros(int(pos[i]) + 1, *y.shape, dtype=torch.float64)
            full[-1] = y
            return O.rotate_halves(full, rot)[-1]

        close(cq[:, :qr], O.rms(x[:, :qr], 1e-2) * qw.double(), tol=tol)
        assert cq.shape[1] % 8 == 0 and float(cq[:, qr:].abs().sum()) == 0
        close(rows[:, :rank], O.rms(x[:, dkv:dkv + rank], 1e-2) * nw.double(), tol=tol)
        for i in range(t):
            close(rows[i:i + 1, lay.RP:lay.RP + dr], turn(x[i:i + 1, dkv + rank:dkv + rank + dr], i), tol=tol)
        flat = cache.view(16, -1)
        for i, s in enumerate(slots.tolist()):
            if s >= 0:
                assert torch.equal(flat[s], rows[i])
        q = torch.randn(t, h * qp, generator=gen).to(dtype)
        qd = torch.full((t, h, lay.CP), 3.0, device=device, dtype=dtype)
        ops.latent_rotate_queries(q.to(device), lay, table, pos.to(device), qd)
        turned = q.clone().to(device)
        ops.latent_rotate_queries(turned, lay, table, pos.to(device))
        for i in range(t):
            want = turn(q[i].double().view(h, qp)[:, dn:dn + dr], i)
            close(turned[i].view(h, qp)[:, dn:dn + dr], want, tol=tol)
            close(qd[i, :, lay.RP:lay.RP + dr], want, tol=tol)
        assert torch.equal(turned.cpu().view(t, h, qp)[..., :dn], q.view(t, h, qp)[..., :dn])
        assert bool((qd[..., :lay.RP] == 3).all()) and float(qd[..., lay.RP + dr:].abs().sum()) == 0


# ---- key ranges ------------------------------------------------------------------------------------------
def test_key_ranges_and_packed_chunks():
    for size in (1, 2, 5, 7):
        for pos in range(30):
            assert first_key(Chunk(size), pos) == O.chunk_start(pos, size) and first_key(size, pos) == O.window_start(pos, size)
            assert first_key(None, pos) == 0

    class Item:
        def __init__(self, start, length):
            self.start, self.length = start, length

    eng = engine("mixed", "cpu")
    items = [Item(0, 20), Item(13, 1), Item(14, 9), Item(17, 2), Item(9, 9)]
    tables = torch.zeros(5, 4, dtype=torch.int32)
    span = eng._key_span(items, tables, Chunk(9))
    q, k = np.diff(span.cu_q.tolist()).tolist(), np.diff(span.cu_k.tolist()).tolist()
    assert q == [9, 9, 2, 1, 4, 5, 1, 1, 9] and k == [9, 9, 2, 5, 9, 5, 9, 1, 9] and span.max_q == 9
    pos = span.cached["token_pos"].tolist()
    assert pos == [*range(20), *range(9, 14), *range(9, 23), *range(9, 19), *range(9, 18)]
    fresh = eng._key_span(items[:1], None, Chunk(9))
    assert fresh.cached is None and fresh.cu_q.tolist() == fresh.cu_k.tolist() == [0, 9, 18, 20]
    span = eng._key_span(items, tables, 11)
    assert np.diff(span.cu_k.tolist()).tolist() == [20, 11, 19, 12, 18] and np.diff(span.cu_q.tolist()).tolist() == [20, 1, 9, 2, 9]


# ---- attention: keys at borders, capped scores, sinks, gates ---------------------------------------------
def _ask(pos, lo, k, scale, i):
    """A query whose score stands out at one key of the range [lo, pos]; the keys just outside would win if they were seen."""
    ts = [t for t in (lo, pos, pos - 1, lo + 1, (lo + pos) // 2, 15, 16, 63, 64, 127, 128) if lo <= t <= pos]
    q = k[ts[i % len(ts)]] * (9.0 / scale / k.shape[-1])
    for out in (lo - 1, pos + 1):
        if 0 <= out < k.shape[0]:
            q = q + k[out] * (18.0 / scale / k.shape[-1])
    return q


FORMS = {"plain": (0.0, False, False), "capped": (7.0, False, True), "sink": (0.0, True, False), "all": (12.0, True, True)}


def _form(name, t, h, gen, device, dtype):
    cap, sink, gate = FORMS[name]
    wide = torch.randn(t, h + 5, generator=gen).to(dtype) * 2
    s = torch.randn(h, generator=gen) * 2 + 6
    s[0] = 40.0 if sink else s[0]                          # a sink that takes nearly all
    form = ops.ScoreForm(cap, wide.to(device)[:, 3:3 + h] if gate else None, s.to(device) if sink else None)
    return form, cap, s.double() if sink else None, torch.sigmoid(wide[:, 3:3 + h].double()) if gate else torch.ones(t, h).double()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("form", sorted(FORMS))
@pytest.mark.parametrize("h,g,qp,vp,keys", [(4, 2, 12, 8, Chunk(21)), (2, 1, 64, 64, Chunk(64)), (4, 1, 128, 128, Chunk(65)), (2, 2, 128, 128, 50),
                                            (2, 1, 192, 128, Chunk(33)), (2, 1, 64, 64, Chunk(1)), (3, 3, 208, 136, 40), (2, 1, 192, 128, None)])
def test_prompt_attention(device, form, h, g, qp, vp, keys):
    scale = 0.4
    lay = ops.GroupedHeads(h, g, qp, vp, qp, vp, 0, h * qp, h * qp + g * qp)

    class Item:
        def __init__(self, start, length):
            self.start, self.length = start, length

    eng = engine("mixed", device)
    for dtype in dtypes(device):
        for lens, starts in (([140, 1, 33], [0, 0, 0]), ([40, 2, 71], [90, 0, 49])):
            gen = torch.Generator().manual_seed(7)
            tq = sum(lens)
            items = [Item(s, n) for s, n in zip(starts, lens)]
            span = eng._key_span(items, None, keys)
            f, cap, sink, gate = _form(form, tq, h, gen, device, dtype)
            q, ks, vs = torch.zeros(tq, h, qp), [], []
            want, q0 = torch.zeros(tq, h, vp, dtype=torch.float64), 0
            for it in items:
                total, low = it.start + it.length, int(first_key(keys, it.start))
                k, v = (torch.randn(total, g, n, generator=gen).to(dtype).float() for n in (qp, vp))
                for i in range(it.length):
                    pos = it.start + i
                    lo = int(first_key(keys, pos))
                    for x in range(h):
                        q[q0 + i, x] = _ask(pos, lo, k[:, x // (h // g)], scale, i + x).to(dtype).float()
                    kk, vv = (y[lo:pos + 1].double().repeat_interleave(h // g, 1) for y in (k, v))
                    s = O.capped(torch.einsum("hd,jhd->hj", q[q0 + i].double(), kk) * scale, cap)
                    want[q0 + i] = torch.einsum("hj,jhd->hd", O.weights_of_scores(s, sink), vv)
                ks.append(k[low:])
                vs.append(v[low:])
                q0 += it.length
            want = want * gate[..., None]
            k, v = torch.cat(ks), torch.cat(vs)
            proj = torch.zeros(tq, (h + g) * qp + g * vp)
            proj[:, :h * qp] = q.reshape(tq, -1)
            kv = (k.to(device, dtype), v.to(device, dtype))
            if not any(starts):                            # keys from the same rows
                proj[:, lay.k_col:lay.v_col], proj[:, lay.v_col:] = k.reshape(tq, -1), v.reshape(tq, -1)
                kv = None
            for t5 in ((True, False) if device == "cuda" and qp == 128 else (True,)):
                got = ops.window_prefill_attention(proj.to(device, dtype), lay, span.cu_q, span.cu_k, span.max_q, scale,
                                                   None if isinstance(keys, Chunk) else keys, kv, use_tcgen05=t5, form=f)
                close(got.view(tq, -1), want.view(tq, -1), dtype, tol=2e-5 if dtype == torch.float32 else 2e-2)


def _paged(lens, bs, rows, gen, device, dtype):
    """Random rows of sequences in scattered pages; what else the pages hold must not matter."""
    b, blocks = len(lens), -(-max(lens) // bs)
    perm = torch.randperm(b * blocks, generator=gen).view(b, blocks)
    fill = float("nan") if device == "cuda" else 7.0
    caches, data = [torch.full((b * blocks, bs, *r), fill) for r in rows], []
    for i, m in enumerate(lens):
        data.append([torch.randn(m, *r, generator=gen).to(dtype).float() for r in rows])
        for c, x in zip(caches, data[-1]):
            for p in range(m):
                c[perm[i, p // bs], p % bs] = x[p]
    return perm.to(device, torch.int32), [c.to(device, dtype) for c in caches], data


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("form", sorted(FORMS))
@pytest.mark.parametrize("h,g,qp,vp,bs,keys", [(4, 2, 12, 8, 4, Chunk(21)), (4, 2, 64, 64, 16, Chunk(64)), (20, 1, 128, 128, 16, Chunk(65)),
                                               (4, 4, 128, 128, 8, Chunk(300)), (6, 2, 192, 128, 32, Chunk(33)), (3, 3, 208, 136, 16, Chunk(40)),
                                               (2, 1, 64, 64, 16, Chunk(1)), (4, 4, 128, 128, 64, None)])
def test_decode_attention_in_chunks(device, form, h, g, qp, vp, bs, keys):
    n, scale = 333, 0.5
    size = keys.size if keys else n
    lay = ops.GroupedHeads(h, g, qp, vp, qp, vp, 0, h * qp, h * qp + g * qp)
    lens = sorted({m for m in (n, 1, 2, bs, bs + 1, size, size + 1, 2 * size - 1, 2 * size, 2 * size + 1, 64, 65, 0) if m <= n})
    for dtype in dtypes(device):
        gen = torch.Generator().manual_seed(1)
        perm, (kc, vc), data = _paged(lens, bs, [(g, qp), (g, vp)], gen, device, dtype)
        b = len(lens)
        f, cap, sink, gate = _form(form, b, h, gen, device, dtype)
        proj, want = torch.zeros(b, (h + g) * qp + g * vp), torch.zeros(b, h, vp, dtype=torch.float64)
        for i, m in enumerate(lens):
            if m == 0:
                continue
            k, v = data[i]
            lo = int(first_key(keys, m - 1))
            q = torch.stack([_ask(m - 1, lo, k[:, x // (h // g)], scale, i + x) for x in range(h)]).to(dtype).float()
            proj[i, :h * qp] = q.reshape(-1)
            kk, vv = (y[lo:].double().repeat_interleave(h // g, 1) for y in (k, v))
            s = O.capped(torch.einsum("hd,jhd->hj", q.double(), kk) * scale, cap)
            want[i] = torch.einsum("hj,jhd->hd", O.weights_of_scores(s, sink), vv) * gate[i][:, None]
        for nsplit in (None, 1, 3):
            got = ops.window_decode_attention(proj.to(device, dtype), lay, kc, vc, perm, torch.tensor(lens, dtype=torch.int32, device=device), n,
                                              scale, None, nsplit=nsplit, chunk=keys.size if keys else None, form=f)
            close(got.reshape(b * h, -1), want.reshape(b * h, -1), dtype, tol=2e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("form", ["plain", "sink", "gate", "both"])
@pytest.mark.parametrize("h,rank,dr,bs,window", [(4, 24, 8, 4, 21), (3, 128, 32, 16, 64), (20, 80, 64, 16, 65), (40, 512, 64, 16, 130), (70, 32, 16, 32, 33),
                                                 (2, 256, 64, 64, 1), (6, 16, 16, 8, 300), (5, 48, 16, 16, None)])
def test_latent_decode_attention(device, form, h, rank, dr, bs, window):
    n, scale = 333, 0.5
    lay = ops.LatentLayout(h, 8, dr, 8, rank, 8 + dr, 8, 0, dr, True)
    win = window or n
    lens = sorted({m for m in (n, 1, 2, bs, bs + 1, win, win + 1, win + 2, win + bs - 1, 64, 65, 0) if m <= n})
    for dtype in dtypes(device):
        gen = torch.Generator().manual_seed(2)
        perm, (cache,), data = _paged(lens, bs, [(lay.CP,)], gen, device, dtype)
        b = len(lens)
        f, _, sink, gate = _form({"plain": "plain", "sink": "sink", "gate": "capped", "both": "all"}[form], b, h, gen, device, dtype)
        f = f._replace(softcap=0.0)
        q, want = torch.zeros(b, h, lay.CP), torch.zeros(b, h, lay.RP, dtype=torch.float64)
        for i, m in enumerate(lens):
            if m == 0:
                continue
            rows = data[i][0]
            lo = int(first_key(window, m - 1))
            q[i] = torch.stack([_ask(m - 1, lo, rows, scale, i + x) for x in range(h)]).to(dtype).float()
            p = O.weights_of_scores(q[i].double() @ rows[lo:].double().t() * scale, sink)
            want[i] = (p @ rows[lo:, :lay.RP].double()) * gate[i][:, None]
        for nsplit in (None, 1, 3):
            for t5 in ((True, False) if device == "cuda" and dtype == torch.bfloat16 else (True,)):
                got = ops.latent_decode_attention(q.to(device, dtype), cache, lay, perm, torch.tensor(lens, dtype=torch.int32, device=device), n,
                                                  scale, nsplit=nsplit, use_tcgen05=t5, window=window, form=f)
                close(got.reshape(b * h, -1), want.reshape(b * h, -1), dtype, tol=2e-5 if dtype == torch.float32 else 1.5e-2)


# ---- delta rule ----------------------------------------------------------------------------------------
def _delta_case(t, h, kvh, d, dv, taps, gen):
    kd, hv = kvh * d, h * dv
    up = lambda n: -(-n // 8) * 8
    cols = [0, up(kd), 2 * up(kd), 2 * up(kd) + up(hv)]
    a_col = cols[3] + up(h)
    lay = ops.DeltaLayout(h, kvh, d, dv, taps, *cols, head_decay=True, silu_gate=True)
    proj = torch.randn(t, a_col + up(h) + up(hv), generator=gen)
    w = ops.DeltaWeights(torch.randn(lay.channels, taps, generator=gen) * 0.7, torch.rand(h, generator=gen) * 5 - 4,
                         torch.randn(h, generator=gen), torch.rand(dv, generator=gen) + 0.5)
    return lay, proj, slice(a_col, a_col + h), slice(a_col + up(h), a_col + up(h) + hv), w


def _delta_want(lay, x, a, g, w, eps):
    t, h, kvh, d, dv = x.shape[0], lay.heads, lay.kv_heads, lay.dim, lay.vdim
    x, of = x.double(), torch.arange(h) // (h // kvh)
    cw = w.conv.double().split([kvh * d, kvh * d, h * dv])
    q, k, v = (O.silu(O.short_conv(x[:, c:c + cc.shape[0]], cc)) for c, cc in zip((lay.q_col, lay.k_col, lay.v_col), cw))
    q, k = O.unit(q.view(t, kvh, d))[:, of] * d ** -0.5, O.unit(k.view(t, kvh, d))[:, of]
    decay = torch.exp(-torch.exp(w.a_log.double()) * O.softplus(x[:, a] + w.dt_bias.double()))
    o, _ = O.delta_recurrence(q, k, v.view(t, h, dv), decay, torch.sigmoid(x[:, lay.b_col:lay.b_col + h]))
    return (O.rms(o, eps) * w.norm.double() * O.silu(x[:, g]).view(t, h, dv)).reshape(t, -1)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,kvh,d,dv,taps", [(4, 2, 12, 8, 3), (3, 1, 10, 7, 5), (2, 2, 64, 128, 4), (6, 3, 100, 36, 2), (2, 1, 200, 40, 1)])
def test_delta_rule_portions_and_decode(device, h, kvh, d, dv, taps):
    n, gen = 60, torch.Generator().manual_seed(d)
    lay, proj, a, g, w = _delta_case(2 * n, h, kvh, d, dv, taps, gen)
    for dtype in dtypes(device):
        x = proj.to(dtype)
        want = torch.stack([_delta_want(lay, x[i * n:(i + 1) * n].float(), a, g, w, 1e-4) for i in range(2)])
        bad = float("nan") if device == "cuda" else 7.0
        dev = dict(device=device)
        ring, state = torch.full((4, taps, lay.channels), bad, dtype=dtype, **dev), torch.full((4, h, d, dv), bad, **dev)
        wd = ops.DeltaWeights(*(t.to(**dev) for t in (w.conv, w.a_log, w.dt_bias, w.norm)))
        got, at, owner = torch.zeros_like(want), [0, 0], torch.tensor([2, 0], **dev)
        for cut in ([7, 1], [1, 6], [2, 3], [17, 5]):
            rows = torch.cat([torch.arange(i * n + at[i], i * n + at[i] + cut[i]) for i in range(2)])
            p = x[rows].to(**dev)
            y = ops.delta_prefill(p, p[:, a], p[:, g], lay, wd, ring, state, torch.tensor([0] * cut[0] + [1] * cut[1], dtype=torch.int32, **dev),
                                  torch.tensor([0, cut[0], sum(cut)], dtype=torch.int32, **dev), torch.tensor(at, dtype=torch.int32, **dev),
                                  owner, 1e-4).double().cpu()
            for i in range(2):
                got[i, at[i]:at[i] + cut[i]] = y[:cut[0]] if i == 0 else y[cut[0]:]
                at[i] += cut[i]
        while min(at) < n:
            live = [i for i in range(2) if at[i] < n]
            p = x[torch.tensor([i * n + at[i] for i in live] + [0])].to(**dev)
            y = ops.delta_decode(p, p[:, a], p[:, g], lay, wd, ring, state, torch.tensor([at[i] for i in live] + [5], dtype=torch.int32, **dev),
                                 torch.cat([owner[live], torch.tensor([-1], **dev)]), 1e-4).double().cpu()
            for j, i in enumerate(live):
                got[i, at[i]] = y[j]
                at[i] += 1
        close(got.flatten(0, 1), want.flatten(0, 1), tol=5e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rate,keeps", [(-20.0, True), (1.5, False)])
def test_delta_rule_far_write(device, rate, keeps):
    """A value written under a key of its own comes back many tokens later when nothing decays, and is gone otherwise."""
    n, far, d = 333, 6, 16
    lay = ops.DeltaLayout(1, 1, d, d, 1, 0, d, 2 * d, 3 * d, head_decay=True, silu_gate=True)
    proj = torch.zeros(n, 4 * d + 16 + d)
    proj[:, lay.k_col + 1] = 4.0                           # all other tokens write under entry 1
    proj[:, lay.v_col] = 0.5
    proj[far, lay.k_col:lay.k_col + d] = torch.eye(d)[4] * 4
    proj[far, lay.v_col:lay.v_col + d] = torch.arange(1.0, 17.0)
    proj[-1, lay.q_col + 4] = 4.0
    proj[-1, lay.k_col:lay.k_col + d] = torch.eye(d)[1] * 4
    proj[:, lay.b_col] = 20.0
    gate = slice(4 * d + 16, 5 * d + 16)
    proj[:, gate] = 30.0                                   # silu(30) = 30
    for dtype in dtypes(device):
        dev = dict(device=device)
        w = ops.DeltaWeights(torch.ones(lay.channels, 1, **dev), torch.full((1,), rate, **dev), torch.zeros(1, **dev), torch.ones(d, **dev))
        p = proj.to(device, dtype)
        y = ops.delta_prefill(p, p[:, 4 * d + 8:4 * d + 9], p[:, gate], lay, w, torch.zeros(1, 1, lay.channels, dtype=dtype, **dev),
                              torch.zeros(1, 1, d, d, **dev), torch.zeros(n, dtype=torch.int32, **dev), torch.tensor([0, n], dtype=torch.int32, **dev),
                              torch.zeros(1, dtype=torch.int32, **dev), torch.zeros(1, dtype=torch.int64, **dev), 1e-6)
        got = y[-1].double().cpu() / 30.0
        v = O.silu(torch.arange(1.0, 17.0).double())
        want = v / v.pow(2).mean().sqrt()
        if keeps:                                          # what is read beside it: small components of the unit key vectors
            close(got[None], want[None], tol=2e-2)
        else:
            assert float((got * want).mean().abs()) < 0.5


# ---- layers alone ----------------------------------------------------------------------------------------
def _layer(device, mixer, mlp, n, seed, **kw):
    cfg = M.config([(mixer, mlp)], **kw)
    w, seq, trace = M.weights(cfg, seed), M.tokens(n, cfg["vocab"], 2), []
    O.forward(cfg, w, seq, trace=trace)
    for dtype in dtypes(device):
        eng = make_engine(cfg, w, device, dtype)
        seen = []
        eng.runner.layer_probe = lambda run, r: seen.append(r.float().cpu().clone())
        eng.replay([("a", seq, [])], ["a"])
        (close if mlp is None else close_routed)(seen[0], trace[0], dtype)


MIXER_CASES = {
    "attention": M.attention(), "one_token_chunk": M.attention(chunk=1), "no_chunk": M.attention(chunk=None), "one_head": M.attention(1, 1, 4, 3, 2, 6, rot_dims=2),
    "all_rotated": M.attention(6, 2, 10, 12, 4, 8, rot_dims=10), "tight_cap": M.attention(softcap=0.5), "wide": M.attention(3, 1, 130, 100, 4, 12, 0.06, rot_dims=66),
    "wider_than_tensor_cores": M.attention(2, 1, 200, 132, 3, 12, 0.06), "six_taps": M.attention(conv=6), "bf16_tiles": M.attention(2, 2, 128, 128, 4, 17, 0.1, rot_dims=64),
    "latent": M.latent(), "latent_no_window": M.latent(window=None), "latent_one_token": M.latent(window=1), "latent_one_head": M.latent(1, 4, 2, 3, 5, 6, 4),
    "latent_wide": M.latent(2, 150, 60, 140, 90, 70, 12, 0.06), "latent_tiles": M.latent(4, 64, 64, 128, 64, 48, 20, 0.1),
    "delta": M.delta(), "delta_one_head": M.delta(1, 1, 4, 3, 2), "delta_wide": M.delta(2, 1, 140, 60, 3), "delta_tiles": M.delta(2, 2, 128, 128, 4),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", sorted(MIXER_CASES))
def test_mixer_alone(device, case):
    _layer(device, MIXER_CASES[case], None, 37, 5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("mlp", ["moe", "all_outputs", "no_identity", "one_expert", "mostly_identity", "many"])
def test_experts_in_a_layer(device, mlp):
    f = {"moe": M.moe(), "all_outputs": M.moe(3, 2, 5, 8), "no_identity": M.moe(4, 0, 2, 40), "one_expert": M.moe(1, 0, 1, 64),
         "mostly_identity": M.moe(1, 6, 3, 16), "many": M.moe(65, 10, 7, 16)}[mlp]
    _layer(device, M.attention(1, 1, 4, 3, 2, 5, rot_dims=2), f, 50, 6, width=64)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case,size", [("attention", 9), ("latent", 11)])
def test_a_token_is_seen_up_to_the_edge(device, case, size):
    """Two sequences that differ in one token: a later position changes exactly where the token is inside its range (or
    reaches a key of the range through the convolution), whole and token by token."""
    mixer = MIXER_CASES[case]
    cfg = M.config([(mixer, None)])
    w, n, at = M.weights(cfg, 11), 40, 13
    a = M.tokens(n, cfg["vocab"], 4)
    b = list(a)
    b[at] = (b[at] + 7) % cfg["vocab"]
    reach = mixer["mixer"].get("conv", 1) - 1
    seen = [at <= i and at + reach >= first_key(Chunk(size) if case == "attention" else size, i) for i in range(n)]
    want = O.forward(cfg, w, a), O.forward(cfg, w, b)
    assert [bool((x - y).abs().max() > 1e-12) for x, y in zip(*want)] == seen
    assert any(seen[at + 2:]) and not all(seen[at:])
    for cuts in ([n], [7, 1], [3]):
        got = [run_schedule(make_engine(cfg, w, device), s, cuts) for s in (a, b)]
        for x, y in zip(got, want):
            close(x, y)
        assert [bool((x != y).any()) for x, y in zip(*got)] == seen


# ---- schedules --------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_whole_prompt_then_decode(device, name):
    n = 70
    seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
    for dtype in dtypes(device):
        eng = engine(name, device, dtype)
        close_routed(run_schedule(eng, seq, [n]), want, dtype, 0.6)
        close_routed(run_schedule(eng, seq, [30, 1]), want, dtype, 0.6)
        assert eng.bm.num_free_blocks == 64 and eng.state_slots.num_free == 8


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [5, 2], [16], [17, 1, 1, 2], [33, 4, 1], [9, 18, 9]], ids=str)
def test_portions(device, cuts):
    n = 50
    for name in ("mixed", "odd_sizes", "one_tap"):
        seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
        close(run_schedule(engine(name, device, block=4), seq, cuts), want)
    if device == "cuda":
        close_routed(run_schedule(engine("mixed", device, torch.bfloat16), M.tokens(n, M.ZOO["mixed"]["vocab"]), cuts),
                     _expected("mixed", n), torch.bfloat16, 0.6)


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[1], [2], [40, 7], [129, 1]], ids=str)
def test_bf16_does_not_depend_on_the_cut(cuts):
    """The same bf16 model whole and in portions: without close calls of a router the two differ by rounding only."""
    cfg = M.config([(M.attention(8, 2, 64, 64, 4, 40, 0.12, rot_dims=32), M.moe(3, 1, 4, 64)), (M.delta(2, 2, 48, 80, 3), M.moe(2, 1, 3, 64)),
                    (M.attention(4, 1, 96, 128, 3, 50, 0.1, rot_dims=96), None), (M.latent(4, 32, 32, 64, 48, 40, 30, 0.15), M.moe(2, 0, 2, 32))], width=128)
    w, seq = M.weights(cfg, 3), M.tokens(140, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    close(run_schedule(make_engine(cfg, w, "cuda", torch.bfloat16), seq, [140]), want, torch.bfloat16)
    close(run_schedule(make_engine(cfg, w, "cuda", torch.bfloat16), seq, cuts), want, torch.bfloat16)


@pytest.mark.parametrize("device", DEVICES)
def test_token_budget_cuts_a_step_without_effect(device):
    seq, want = M.tokens(70, M.ZOO["mixed"]["vocab"]), _expected("mixed", 70)
    eng = engine("mixed", device, budget=9)
    got = eng.replay([("a", seq[:40], list(range(40))), ("b", seq[:11], [0, 10]), ("c", seq[:1], [0])])
    close(got, torch.cat([want[:40], want[[0, 10]], want[:1]]))


@pytest.mark.parametrize("device", DEVICES)
def test_unequal_batches_match_each_alone(device):
    vocab = M.ZOO["mixed"]["vocab"]
    lens, total = [1, 2, 17, 40, 5], 46
    seqs = [M.tokens(total, vocab, s) for s in range(len(lens))]
    want = [_expected("mixed", total, s) for s in range(len(lens))]
    eng = engine("mixed", device, graphs=(8,) if device == "cuda" else ())
    got = eng.replay([(str(i), s[:n], list(range(n))) for i, (s, n) in enumerate(zip(seqs, lens))])
    close(got, torch.cat([w[:n] for w, n in zip(want, lens)]))
    at = list(lens)
    for step in range(6):           # decode together; shorter ones leave on the way, order changes
        live = [i for i in range(5) if step < 6 - i][::-1 if step % 2 else 1]
        got = eng.replay([(str(i), [seqs[i][at[i]]], [0]) for i in live], [str(i) for i in live if step == 5 - i])
        close(got, torch.stack([want[i][at[i]] for i in live]))
        for i in live:
            at[i] += 1
    assert eng.state_slots.num_free == 8 and eng.bm.num_free_blocks == 64
    # a new prompt, a portion of a running one and single tokens in one step
    eng.replay([("x", seqs[0][:9], []), ("y", seqs[1][:4], [])])
    got = eng.replay([("z", seqs[2][:3], [2]), ("x", seqs[0][9:10], [0]), ("y", seqs[1][4:10], [0, 5])])
    close(got, torch.stack([want[2][2], want[0][9], want[1][4], want[1][9]]))


@pytest.mark.parametrize("device", DEVICES)
def test_pages_and_slots_are_used_again(device):
    vocab = M.ZOO["mixed"]["vocab"]
    eng = engine("mixed", device, blocks=13, block=4, seqs=2)
    seqs = [M.tokens(46, vocab, s) for s in range(3)]
    want = [_expected("mixed", 46, s) for s in range(3)]
    for s in (0, 1, 2, 1):
        close(run_schedule(eng, seqs[s], [20, 1, 1, 3, 1]), want[s])
        assert eng.bm.num_free_blocks == 13 and eng.state_slots.num_free == 2
    # interleaved lifetimes: pages and slots of a finished request go to the next one while another runs
    eng.replay([("keep", seqs[0][:6], [])])
    for s in (1, 2):
        close(run_schedule(eng, seqs[s][:20], [7, 1], rid=f"t{s}"), want[s][:20])
        close(eng.replay([("keep", [seqs[0][5 + s]], [0])]), want[0][5 + s:6 + s])


@pytest.mark.parametrize("device", DEVICES)
def test_single_tokens_from_the_start(device):
    """Decoding right after a first portion of one token: convolutions, windows and chunks that are not full yet."""
    for name in sorted(M.ZOO):
        close(run_schedule(engine(name, device), M.tokens(12, M.ZOO[name]["vocab"]), [1]), _expected(name, 12))


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    n = 220
    eng = engine("mixed", device, graphs=(1, 2) if device == "cuda" else ())
    close(run_schedule(eng, M.tokens(n, M.ZOO["mixed"]["vocab"]), [10, 1]), _expected("mixed", n))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["attention", "latent", "delta"])
def test_one_kind_of_layer_only(device, case):
    """Latent attention alone takes no state slots, the delta rule alone no cache memory; attention takes both."""
    cfg = M.config([(MIXER_CASES[case], M.moe()), (MIXER_CASES[case], None)])
    w, seq = M.weights(cfg, 8), M.tokens(40, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = make_engine(cfg, w, device, graphs=(1,) if device == "cuda" else ())
    assert (eng.state_slots is None) == (case == "latent") and (eng.kv_bytes_per_block() == 0) == (case == "delta")
    close(run_schedule(eng, seq, [11, 6, 1]), want)
    out = eng.generate([seq[:9]], SamplingParams(n=2, temperature=0.0, max_tokens=5))[0].outputs
    assert out[0].token_ids == out[1].token_ids and out[0].token_ids[0] == int(want[8].argmax())


@pytest.mark.parametrize("device", DEVICES)
def test_a_far_token_reaches_through_the_recurrence_only(device):
    """Two sequences that differ in their first token: past every window and chunk the logits still differ, as the oracle's
    do in both."""
    vocab, n = M.ZOO["mixed"]["vocab"], 60
    a = M.tokens(n, vocab, 4)
    b = [(a[0] + 7) % vocab] + a[1:]
    want = [O.forward(M.ZOO["mixed"], _weights("mixed"), s) for s in (a, b)]
    assert float((want[0][-1] - want[1][-1]).abs().max()) > 1e-5
    for s, w in zip((a, b), want):
        close(run_schedule(engine("mixed", device), s, [7, 1])[-1:], w[-1:])


# ---- generation through the scheduler -----------------------------------------------------------------
def _greedy(name, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        lg = O.forward(M.ZOO[name], _weights(name), ids)[-1]
        top = lg.topk(2).values
        if float(top[0] - top[1]) < 1e-3:
            break                       # too close to call in 32-bit: compare up to here
        ids.append(int(lg.argmax()))
    return ids[len(prompt):]


@functools.lru_cache(maxsize=None)
def _greedy_cases():
    vocab = M.ZOO["mixed"]["vocab"]
    prompts = [M.tokens(n, vocab, 10 + n) for n in (3, 19, 1, 8)]
    return prompts, [_greedy("mixed", p, 9) for p in prompts]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("setting", ["plain", "small_budget", "two_at_a_time", "few_pages"])
def test_greedy_generation(device, setting):
    prompts, want = _greedy_cases()
    kw = {"plain": {}, "small_budget": dict(budget=5), "two_at_a_time": dict(seqs=2),
          "few_pages": dict(blocks=12, block=4)}[setting]
    eng = engine("mixed", device, graphs=(2, 4) if device == "cuda" else (), **kw)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9))
    for o, w in zip(outs, want):
        assert o.outputs[0].token_ids[:len(w)] == w
        assert len(o.outputs[0].token_ids) == 9
    if setting == "few_pages":
        assert eng.stats["preemptions"] > 0            # recomputed from the first token, in another slot
    assert eng.state_slots.num_free == eng.max_num_seqs and eng.bm.num_free_blocks == eng.bm.num_blocks


@pytest.mark.parametrize("device", DEVICES)
def test_samples_of_a_prompt_fork_state_and_pages(device):
    prompts, want = _greedy_cases()
    eng = engine("mixed", device, block=4, budget=7, seqs=6, graphs=(8,) if device == "cuda" else ())
    for o, w in zip(eng.generate(prompts, SamplingParams(n=3, temperature=0.0, max_tokens=9)), want):
        for c in o.outputs:
            assert c.token_ids[:len(w)] == w
    a = eng.generate(prompts[:2], SamplingParams(n=4, temperature=1.0, max_tokens=12, seed=5))
    b = engine("mixed", device).generate(prompts[:2], SamplingParams(n=4, temperature=1.0, max_tokens=12, seed=5))
    for x, y in zip(a, b):               # sampled: the same draws whatever the batch, the pages and the slots
        assert [c.token_ids for c in x.outputs] == [c.token_ids for c in y.outputs]
        c = x.outputs[0]                 # what was sampled has the log-probability the oracle gives it
        lp = torch.log_softmax(O.forward(M.ZOO["mixed"], _weights("mixed"), x.prompt_token_ids + c.token_ids), -1)
        for j, (tok, got) in enumerate(zip(c.token_ids, c.logprobs)):
            assert abs(float(lp[len(x.prompt_token_ids) - 1 + j, tok]) - got) < 1e-3


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["many_heads", "odd_sizes", "wide_heads", "one_tap"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_graph_decode_is_the_eager_decode(dtype, name):
    """A captured step advances every state exactly once, also the step whose capture it is."""
    seqs = [M.tokens(40, M.ZOO[name]["vocab"], s) for s in range(3)]
    got = []
    for graphs in ((), (4,)):
        eng = engine(name, "cuda", dtype, graphs=graphs)
        eng.replay([(str(i), s[:20 + i], []) for i, s in enumerate(seqs)])
        steps = [eng.replay([(str(i), [s[20 + i + k]], [0]) for i, s in enumerate(seqs)]).float().cpu() for k in range(10)]
        got.append(torch.stack(steps))
    if dtype == torch.float32:
        close(got[1].flatten(0, 1), got[0].flatten(0, 1), tol=1e-5)
    else:
        close_routed(got[1].flatten(0, 1), got[0].flatten(0, 1), dtype, 0.9)


# ---- framework ------------------------------------------------------------------------------------------
def test_configuration_and_loading_errors(tmp_path):
    cfg = M.ZOO["mixed"]
    folder = M.save(cfg, _weights("mixed"), str(tmp_path / "m"))
    c, w = registry.load_model(folder, torch.float32, "cpu")
    assert c.architecture == "Gapevik" and len(w.layers) == 4 and c.is_moe and c.is_recurrent
    assert c.windows == (Chunk(9), 11) and c.residual_mult == 0.6
    assert w.layers[3] is w.layers[0] and w.lm_head is w.embed
    for change, message in (({"l0.mix.stray": torch.zeros(3)}, "stray"), ({"l3.norm1": torch.zeros(48)}, "l3.norm1"),
                            ({"l0.mlp.router": torch.zeros(3, 48)}, "outputs"), ({"l0.mix.q.conv": torch.zeros(48, 2)}, "convolution|size")):
        with pytest.raises((ValueError, RuntimeError), match=message):
            build_hybrid_weights(c, {**_weights("mixed"), **change}, "cpu")
    with pytest.raises(KeyError, match="sink"):
        build_hybrid_weights(c, {k: v for k, v in _weights("mixed").items() if k != "l1.mix.sink"}, "cpu")
    for layers, message in (([(M.attention(5, 2), None)], "divide"), ([(M.attention(rot_dims=7), None)], "even"), ([(M.delta(5, 2), None)], "divide"),
                            ([(M.attention(), M.moe(2, 1, 4))], "top 4"), ([({"type": "mlstm", "mixer": {}}, None)], "mixer type"),
                            ([(M.latent(rot_dim=7), None)], "even"), ([(M.latent(window=-3), None)], "window"), ([(M.attention(chunk=-3), None)], "chunk"),
                            ([(M.attention(softcap=-1.0), None)], "capped")):
        with pytest.raises(ValueError, match=message):
            HybridConfig.from_json(M.config(layers))
    for of, message in ((1, "has none"), (2, "has none"), (0, "differs")):
        bad = M.config([(M.attention(), None), (M.latent(), None)])
        bad["layers"][1]["weights_of"] = of
        with pytest.raises(ValueError, match=message):
            HybridConfig.from_json(bad)
    with pytest.raises(ValueError, match="prefix caching"):
        LLMEngine(c, "cpu", enable_prefix_caching=True)


def test_layers_that_share_tensors_have_caches_of_their_own():
    eng = engine("odd_sizes", "cpu")
    cache, w = eng.runner.cache, eng.runner.weights
    assert w.layers[4] is w.layers[1]
    assert [sorted(r) for r in cache.rows] == [[], ["latent"], ["k", "v"], [], ["latent"]]
    assert [sorted(s) for s in cache.slots] == [["ring", "state"], [], ["ring"], ["ring", "state"], []]
    assert cache.rows[1]["latent"].data_ptr() != cache.rows[4]["latent"].data_ptr()
    chain = M.config([(M.attention(), None)] * 3, weights_of=[(1, 0), (2, 1)])       # through another one that shares
    seq, wt = M.tokens(30, chain["vocab"]), M.weights(chain, 4)
    close(run_schedule(make_engine(chain, wt, "cpu"), seq, [13, 1]), O.forward(chain, wt, seq))


def test_prefix_caching_without_carried_state():
    cfg = M.config([(M.latent(), M.moe()), (M.latent(window=5), None)])
    w, seq = M.weights(cfg, 2), M.tokens(30, cfg["vocab"])
    eng = LLMEngine(HybridConfig.from_json(cfg, torch.float32), "cpu", max_num_seqs=2, max_model_len=64, block_size=4, enable_prefix_caching=True)
    eng.runner.bind_weights(build_hybrid_weights(eng.cfg, w, "cpu"))
    eng.init_cache(32)
    want = O.forward(cfg, w, seq)
    for _ in range(2):
        out = eng.generate([seq], SamplingParams(temperature=0.0, max_tokens=1))
        assert out[0].outputs[0].token_ids[0] == int(want[-1].argmax())
    assert eng.bm.stats()["prefix_hits"] > 0


@pytest.mark.parametrize("device", DEVICES)
def test_trace_runner_and_generate_command_lines(device, tmp_path):
    root = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))
    folder = M.save(M.ZOO["mixed"], _weights("mixed"), str(tmp_path / "m"))
    seq, want = M.tokens(30, M.ZOO["mixed"]["vocab"]), _expected("mixed", 30)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seq[:9], "want": [8, 0]}, {"id": "b", "tokens": seq[:4], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [seq[9]], "want": []}], "end": ["b"]},
             {"step": 7, "entries": [{"id": "a", "tokens": [seq[10]], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "20", "--device", device], input="\n".join(map(json.dumps, steps)) + "\n", text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 7"]
    v = M.ZOO["mixed"]["vocab"]
    read = lambda n: torch.frombuffer(bytearray((out / n).read_bytes()), dtype=torch.float32).view(-1, v)
    close(read("0.f32"), want[[8, 0, 1]])
    close(read("7.f32"), want[[10]])
    prompts, greedy = _greedy_cases()
    r = subprocess.run([sys.executable, os.path.join(root, "cli", "generate.py"), "--model", folder, "--dtype", "float32",
                        "--device", device, "--temperature", "0", "--max-tokens", "6", "--prompt-ids",
                        " ".join(map(str, prompts[1]))], text=True, capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr
    ids = json.loads(r.stdout.splitlines()[-1])["outputs"][0]["token_ids"]
    assert ids[:len(greedy[1])] == greedy[1][:6] and len(ids) == 6
