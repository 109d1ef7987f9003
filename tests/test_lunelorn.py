"""Lunelorn decoders through the rollout engine against the plain restatement in ``lunelorn_oracle`` (fp64).

Every test runs on the CPU formulation; the same tests run on the CUDA kernels on a GPU machine, in true 32-bit and,
where it makes sense, in bf16 with a tolerance of bf16 rounding.
"""
import functools
import json
import os
import subprocess
import sys

import pytest
import torch

import lunelorn_models as M
import lunelorn_oracle as O
from hybrid_helpers import TOL, close, dtypes, make_engine, run_schedule
from mindspeed_rl_b200 import ops
from mindspeed_rl_b200.models import registry
from mindspeed_rl_b200.models.hybrid_config import HybridConfig
from mindspeed_rl_b200.ops import moe as K
from mindspeed_rl_b200.ops import wkv as W
from mindspeed_rl_b200.ops.matrix_memory import constant_decay
from mindspeed_rl_b200.rollout.engine import LLMEngine
from mindspeed_rl_b200.rollout.hybrid_weights import build_hybrid_weights
from mindspeed_rl_b200.rollout.scheduler import SamplingParams

CUDA = pytest.param("cuda", marks=pytest.mark.gpu)
DEVICES = ["cpu", CUDA]
F64 = torch.float64


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


def i32(x, device):
    return torch.tensor(x, dtype=torch.int32, device=device)


def i64(x, device):
    return torch.tensor(x, dtype=torch.int64, device=device)


# ---- mechanisms alone: residual stream -----------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [42, 48, 1100, 9000])
def test_sandwich_adds_and_pass_inputs(device, width):
    g = torch.Generator().manual_seed(3)
    t, dev = 5, dict(device=device)
    w1, w2, step = (torch.randn(width, generator=g) * 0.3 + 1.0 for _ in range(3))
    post, after = ops.PostNorm(w1.to(**dev), 1e-2), ops.Norm(w2.to(**dev), 1e-3)
    table, ids = torch.randn(9, width, generator=g) * 0.1, torch.tensor([3, 0, 8, 8, 1])
    d1, d2 = w1.double(), w2.double()
    e0 = O.rms(table[ids].double(), 1e-2) * d1
    for keep, s in ((False, None), (True, step)):
        resid, first, y = ops.post_embed(ids.to(**dev), table.to(**dev), post, after, keep, None if s is None else s.to(**dev))
        x = e0 if s is None else e0 + s.double()
        close(resid, x, tol=1e-6)
        close(y, O.rms(x, 1e-3) * d2, tol=1e-5)
        assert (first is None) == (not keep)
        if keep:
            close(first, e0, tol=1e-6)
    r0, d, rows = torch.randn(t, width, generator=g), torch.randn(t, width, generator=g) * 0.02, torch.randn(11, width, generator=g)
    pos, wt = torch.tensor([[0, 3], [9, 10], [4, 1], [2, 2], [8, 7]]), torch.rand(t, 2, generator=g)
    mixed = (rows[pos].double() * wt[..., None].double()).sum(1)
    for entry in (None, ops.PassEntry(None, step), ops.PassEntry(r0 * 2, step)):
        more = 0.0 if entry is None else step.double() + (0.0 if entry.again is None else entry.again.double())
        e = entry and ops.PassEntry(None if entry.again is None else entry.again.to(**dev), entry.step.to(**dev))
        for norm in (None, after):
            resid = r0.to(**dev).clone()
            y = ops.post_add_(resid, d.to(**dev), post, norm, e)
            x = r0.double() + O.rms(d.double(), 1e-2) * d1 + more
            close(resid, x, tol=1e-6)
            close(y, x if norm is None else O.rms(x, 1e-3) * d2, tol=1e-5)
            resid = r0.to(**dev).clone()
            y = ops.moe_post_add_(resid, rows.to(**dev), pos.reshape(-1).to(torch.int32).to(**dev), wt.to(**dev), post, norm, entry=e)
            x = r0.double() + O.rms(mixed, 1e-2) * d1 + more
            close(resid, x, tol=1e-6)
            close(y, x if norm is None else O.rms(x, 1e-3) * d2, tol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width,dim", [(42, 5), (48, 8), (64, 16), (1100, 12), (2048, 40)])
def test_token_side(device, width, dim):
    g = torch.Generator().manual_seed(dim)
    t, layers, li, pad = 7, 3, 1, (dim + 7) // 8 * 8
    for dtype in dtypes(device):
        x = torch.randn(t, width, generator=g)
        gate, proj, table = (torch.randn(*s, generator=g).to(dtype) for s in ((dim, width), (width, dim), (9, layers * dim)))
        norm, nxt = (torch.randn(width, generator=g) * 0.3 + 1.0 for _ in range(2))
        ids = torch.tensor([3, 0, 8, 8, 1, 2, 5])
        gate = (gate.float() * 1.5 / width ** 0.5).to(dtype)
        want = x.double() + O.token_side(x.double(), table[ids, li * dim:(li + 1) * dim].double(),
                                         {"gate": gate.double(), "proj": proj.double(), "norm": norm.double()}, 1e-3)
        side = ops.TokenSide(torch.nn.functional.pad(gate, (0, 0, 0, pad - dim)).to(device),
                             torch.nn.functional.pad(proj, (0, pad - dim)).contiguous().to(device), table.to(device), li * dim, dim)
        post, after = ops.PostNorm(norm.to(device), 1e-3), ops.Norm(nxt.to(device), 1e-2)
        for fused in (None, 0):            # the gate's product in its kernel, and as a matrix product
            for entry in (None, ops.PassEntry(x.to(device) * 3, nxt.to(device))):
                resid = x.to(device).clone()
                y = ops.token_side_(resid, x.to(device, dtype), ids.to(device), side, post, after, entry, fused_tokens=fused)
                w = want if entry is None else want + 3 * x.double() + nxt.double()
                close(resid, w, tol=1e-5 if dtype == torch.float32 else 2e-2)
                close(y, O.rms(w, 1e-2) * nxt.double(), tol=1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
def test_soft_cap(device):
    for n in (3 * 40, 3 * 41):
        x = torch.linspace(-90, 90, n).view(3, -1)
        for dtype in dtypes(device):
            y = ops.soft_cap_(x.to(device, dtype).clone(), 7.0)
            close(y, 7.0 * torch.tanh(x.to(dtype).double() / 7.0), tol=1e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,top", [(1, 1), (5, 5), (33, 4), (200, 40), (700, 3)])
def test_router_weights_over_the_chosen(device, experts, top):
    z = torch.randn(19, experts, generator=torch.Generator().manual_seed(experts)) * 4
    z[3] += 300.0
    z[4] -= 300.0
    idx, score = K.route_top(z.to(device), top, chosen_softmax=True)
    for t in range(19):
        want = O.choose(z[t].double(), top)
        assert idx[t].cpu().tolist() == want
        assert torch.allclose(score[t].cpu().double(), torch.softmax(z[t, want].double(), -1), atol=1e-6)


# ---- attention with turned values ------------------------------------------------------------------------
TURNED = [(4, 2, 12, 10, 16, 12, 8), (3, 3, 6, 4, 6, 4, 6), (8, 2, 96, 64, 128, 128, 64), (6, 2, 40, 24, 64, 64, 16), (2, 1, 12, 14, 64, 64, 2)]


def _pad(x, to):
    return torch.nn.functional.pad(x, (0, to - x.shape[-1]))


def _turn_at(x, pos, dims, base, sign=1.0):
    """Rows ``x [T, heads, n]`` turned by their positions, one by one."""
    out = torch.empty_like(x)
    for i, p in enumerate(pos):
        full = torch.zeros(p + 1, *x.shape[1:], dtype=x.dtype)
        full[-1] = x[i]
        out[i] = O.turn(full, dims, base, sign)[-1]
    return out


def _turned_layout(h, g, d, dv, qp, vp):
    return ops.GroupedHeads(h, g, d, dv, qp, vp, 0, h * qp, (h + g) * qp)


def _tables(rot, dv, base, n=512):
    f = lambda dims: tuple(base ** (-2.0 * i / dims) for i in range(dims // 2))
    return ops.angle_table(n, f(rot), "cpu"), ops.angle_table(n, f(dv), "cpu")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,d,dv,qp,vp,rot", TURNED)
def test_rotation_and_turned_values(device, h, g, d, dv, qp, vp, rot):
    t, gen, base = 11, torch.Generator().manual_seed(5), 50.0
    lay = _turned_layout(h, g, d, dv, qp, vp)
    pos = [0, 1, 5, 30, 31, 2, 9, 17, 3, 300, 8]
    slots = torch.tensor([3, -1, 0, 7, 12, 20, 31, 1, 2, 4, 5])
    table, vtable = _tables(rot, dv, base)
    for dtype in dtypes(device):
        q, k, v = (torch.randn(t, n, x, generator=gen).to(dtype) for n, x in ((h, d), (g, d), (g, dv)))
        proj = torch.cat([_pad(q, qp).reshape(t, -1), _pad(k, qp).reshape(t, -1), _pad(v, vp).reshape(t, -1)], 1).to(device)
        kc, vc = torch.zeros(8, 4, g, qp, device=device, dtype=dtype), torch.zeros(8, 4, g, vp, device=device, dtype=dtype)
        ops.turned_prep_(proj, lay, 1e-2, table.to(device), vtable.to(device), i32(pos, device), slots.to(device), kc, vc)
        tol = 1e-6 if dtype == torch.float32 else 6e-3
        got = lay.split(proj.cpu().float())
        want = (_turn_at(q.double(), pos, rot, base), _turn_at(k.double(), pos, rot, base),
                _turn_at(O.rms(v.double(), 1e-2), pos, dv, base))
        for x, y, n in zip(got, want, (d, d, dv)):
            close(x[..., :n].reshape(t, -1), y.reshape(t, -1), tol=tol)
            assert float(x[..., n:].abs().sum()) == 0
        flat_k, flat_v = kc.cpu().float().view(-1, g, qp), vc.cpu().float().view(-1, g, vp)
        for i, s in enumerate(slots.tolist()):
            if s >= 0:
                assert torch.equal(flat_k[s], got[1][i]) and torch.equal(flat_v[s], got[2][i])
        unused = [s for s in range(32) if s not in slots.tolist()]
        assert float(flat_k[unused].abs().sum() + flat_v[unused].abs().sum()) == 0
        attn = _pad(torch.randn(t, h, dv, generator=gen).to(dtype), vp)
        out = torch.full((t, h * vp + 8), 5.0, dtype=dtype, device=device)
        ops.turn_back(attn.reshape(t, -1).to(device), lay, vtable.to(device), i32(pos, device), 0.6, out)
        back = out.cpu().double()[:, :h * vp].view(t, h, vp)
        close(back[..., :dv].reshape(t, -1), 0.6 * _turn_at(attn[..., :dv].double(), pos, dv, base, -1.0).reshape(t, -1), tol=tol)
        assert float(back[..., dv:].abs().sum()) == 0 and bool((out[:, h * vp:] == 5.0).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,d,dv,qp,vp,rot,bs", [(4, 2, 12, 10, 12, 12, 8, 4), (4, 1, 48, 64, 64, 64, 48, 16), (6, 2, 96, 80, 128, 128, 30, 16),
                                                   (2, 1, 160, 96, 192, 128, 40, 32), (2, 2, 200, 132, 200, 136, 66, 16)])
def test_attention_finds_far_keys(device, h, g, d, dv, qp, vp, rot, bs):
    """Queries whose score stands out at one key (first tokens, page and tile borders, far and near ones) get that key's
    value with the turn of the distance between the two; prompts, portions and decode steps."""
    n, base, scale, eps = 270, 50.0, 0.4, 1e-3
    lay = _turned_layout(h, g, d, dv, qp, vp)
    table, vtable = _tables(rot, dv, base)
    for dtype in dtypes(device):
        gen = torch.Generator().manual_seed(7)
        k, v = (torch.randn(n, g, x, generator=gen).to(dtype).double() for x in (d, dv))
        kr = O.turn(k, rot, base)
        qr = torch.empty(n, h, d, dtype=F64)
        for i in range(n):
            ts = [t for t in (0, 1, i, i - 1, i // 2, bs - 1, bs, 2 * bs, 63, 64, 127, 128, 255, 256) if 0 <= t <= i]
            for x in range(h):
                qr[i, x] = kr[ts[(i + x) % len(ts)], x // (h // g)] * (14.0 / scale / d)
        q = O.turn(qr, rot, base, -1.0).to(dtype).double()
        vn = O.turn(O.rms(v, eps), dv, base)
        want = (0.8 * O.turn(O.attend(O.turn(q, rot, base), kr, vn, scale), dv, base, -1.0)).reshape(n, -1)
        rows = torch.cat([_pad(q, qp).reshape(n, -1), _pad(k, qp).reshape(n, -1), _pad(v, vp).reshape(n, -1)], 1).to(dtype)
        blocks = (n + bs - 1) // bs
        perm = torch.randperm(blocks, generator=gen)
        fill = float("nan") if device == "cuda" else 7.0
        kc, vc = (torch.full((blocks, bs, g, x), fill, device=device, dtype=dtype) for x in (qp, vp))
        at = perm[torch.arange(n) // bs] * bs + torch.arange(n) % bs
        got, bt = torch.zeros(n, h * dv, dtype=F64), perm[None].to(device, torch.int32)
        tol = 3e-5 if dtype == torch.float32 else 4e-2

        def run(lo, hi, attend):
            proj, pos = rows[lo:hi].to(device, copy=True), i32(list(range(lo, hi)), device)
            ops.turned_prep_(proj, lay, eps, table.to(device), vtable.to(device), pos, at[lo:hi].to(device), kc, vc)
            out = torch.empty(hi - lo, h * vp, dtype=dtype, device=device)
            ops.turn_back(attend(proj), lay, vtable.to(device), pos, 0.8, out)
            got[lo:hi] = out.double().cpu().view(hi - lo, h, vp)[..., :dv].reshape(hi - lo, -1)

        run(0, n, lambda p: ops.window_prefill_attention(p, lay, i32([0, n], device), i32([0, n], device), n, scale, None))
        close(got, want, dtype, tol=tol)
        whole = got.clone()
        for lo, hi in ((0, 129), (129, 131), (131, 250)):              # portions over the cache
            def attend(p):
                where = dict(block_tables=bt, token_seq=i32([0] * hi, device), token_pos=i32(list(range(hi)), device))
                kv = tuple(ops.rows_gather(c, **where) for c in (kc, vc))
                return ops.window_prefill_attention(p, lay, i32([0, hi - lo], device), i32([0, hi], device), hi - lo, scale, None, kv)
            run(lo, hi, attend)
        for i in range(250, n):
            run(i, i + 1, lambda p: ops.window_decode_attention(p, lay, kc, vc, bt, i32([i + 1], device), i + 1, scale, None))
        close(got, want, dtype, tol=tol)
        close(got, whole, dtype, tol=tol)


# ---- recurrences: portions, decode, reuse of slots ------------------------------------------------------------
def _walk(n, device, prefill, decode, cuts=([127, 1], [1, 130], [2, 3], [65, 64])):
    """Two sequences of n tokens in portions that straddle segment borders, then token by token beside a row without a
    slot.  ``prefill(rows, cu, longest, starts, owner)`` and ``decode(rows, positions, owner)`` -> outputs."""
    got, at, owner = {}, [0, 0], torch.tensor([2, 0], device=device)
    for cut in cuts:
        cut = [min(c, n - a - 3) for c, a in zip(cut, at)]
        rows = torch.cat([torch.arange(i * n + at[i], i * n + at[i] + cut[i]) for i in range(2)])
        y = prefill(rows, i32([0, cut[0], sum(cut)], device), max(cut), i32(at, device), owner, i32([0] * cut[0] + [1] * cut[1], device))
        got.update(zip(rows.tolist(), y.double().cpu()))
        at = [a + c for a, c in zip(at, cut)]
    while min(at) < n:
        live = [i for i in range(2) if at[i] < n]
        rows = torch.tensor([i * n + at[i] for i in live] + [0])
        y = decode(rows, i32([at[i] for i in live] + [5], device), torch.cat([owner[live], torch.tensor([-1], device=device)]))
        got.update(zip(rows.tolist()[:-1], y.double().cpu()))
        at = [a + 1 if i in live else a for i, a in enumerate(at)]
    return torch.stack([got[i] for i in range(2 * n)])


def _filled(device, *shape):
    """State of slots before use: what it holds must not matter to a sequence's first token."""
    return torch.full(shape, float("nan") if device == "cuda" else 7.0, device=device)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,d,dv", [(4, 12, 20), (3, 64, 32), (1, 128, 128), (2, 40, 130), (1, 200, 300)])
@pytest.mark.parametrize("chunked", [False, True])
def test_retention_portions_and_decode(device, h, d, dv, chunked):
    if device == "cpu" and chunked:
        pytest.skip("one CPU formulation")
    n, gen, eps = 210, torch.Generator().manual_seed(1), 1e-5
    dp, vp = (d + 15) // 16 * 16, (dv + 15) // 16 * 16
    lay = ops.MemoryLayout(h, dp, vp, dv, 0, h * dp, 2 * h * dp, 2 * h * dp + h * vp, d ** -0.5, silu_gate=True)
    decay = [0.999, 0.6, 0.0, 1.0][:h]
    for dtype in dtypes(device):
        if dtype == torch.float32 and chunked:
            continue
        q, k, v, gate = (torch.randn(2 * n, h, x, generator=gen).to(dtype) for x in (d, d, dv, dv))
        proj = torch.cat([_pad(x, p).reshape(2 * n, -1) for x, p in ((q, dp), (k, dp), (v, vp), (gate, vp))], 1)
        want = []
        for i in range(2):
            s = slice(i * n, (i + 1) * n)
            o, _ = O.retention_recurrence(q[s].double(), k[s].double() * d ** -0.5, v[s].double(), torch.tensor(decay, dtype=F64))
            want.append(_pad(O.rms(o, eps) * O.silu(gate[s].double()), vp).reshape(n, -1))
        want = torch.cat(want)
        w = ops.MemoryWeights(None, torch.ones(h * vp, device=device), constant_decay(decay).to(device))
        slots = {"memory": _filled(device, 4, h, dp, vp)}
        got = _walk(n, device,
                    lambda r, cu, m, st, own, _: ops.memory_prefill(proj[r].to(device), None, lay, w, slots, cu, m, st, own, eps, chunked=chunked),
                    lambda r, pos, own: ops.memory_decode(proj[r].to(device), None, lay, w, slots, pos, own, eps))
        close(got, want, tol=2e-5 if dtype == torch.float32 else 2e-2)
        if dtype == torch.bfloat16:                        # inputs are exact: only the result is rounded
            assert float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) < 3e-3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("decay", [1.0, 0.9])
def test_retention_far_write(device, decay):
    """A value written under a key of its own comes back hundreds of tokens later as far as the decay lets it."""
    n, far, d = 333, 6, 16
    lay = ops.MemoryLayout(1, d, d, d, 0, d, 2 * d, 3 * d, 1.0, silu_gate=True)
    proj = torch.zeros(n, 4 * d)
    proj[:, d + 1] = 4.0                                   # all other tokens write zeros under entry 1
    proj[far, d:2 * d], proj[far, 2 * d:3 * d] = torch.eye(d)[4] * 4, torch.arange(1.0, 17.0)
    proj[-1, :d] = torch.eye(d)[4] * 4
    proj[:, 3 * d:] = 1.0
    v = torch.arange(1.0, 17.0).double() * 16 * decay ** (n - 1 - far)
    want = O.rms(v[None], 1e-6)[0] * O.silu(torch.ones(16).double())
    assert (float(want.abs().max()) > 1) == (decay == 1.0)
    for dtype in dtypes(device):
        w = ops.MemoryWeights(None, torch.ones(d, device=device), constant_decay([decay]).to(device))
        y = ops.memory_prefill(proj.to(device, dtype), None, lay, w, {"memory": _filled(device, 1, 1, d, d)}, i32([0, n], device), n,
                               i32([0], device), i64([0], device), 1e-6)
        assert torch.allclose(y[-1].double().cpu(), want, atol=1e-4 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [20, 7, 136, 515])
def test_min_gru_portions_and_decode(device, width):
    n, gen, padded = 200, torch.Generator().manual_seed(width), (width + 7) // 8 * 8
    lay = ops.GRULayout(width, padded, 8, 8 + padded, 8 + 2 * padded, out_col=16, scale=1.7)
    for dtype in dtypes(device):
        zb, xb = torch.randn(width, generator=gen) * 2 - 2, torch.randn(width, generator=gen)
        zb[0], zb[1] = -14.0, 9.0                          # a long memory, and none
        proj = torch.randn(2 * n, 8 + 3 * padded, generator=gen).to(dtype)
        z, x, g = (proj[:, c:c + width].double() for c in (lay.z_col, lay.x_col, lay.g_col))
        z, u = torch.sigmoid(z + zb.double()), x + xb.double()
        cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        s = torch.cat([O.min_gru_scan(z[i:i + n], cand[i:i + n]) for i in (0, n)])
        want = s * O.silu(g) * lay.scale
        state, args = _filled(device, 4, width), (zb.to(device), xb.to(device))

        def run(f, r, *rest):
            out = torch.full((len(r), 16 + padded), 3.0, dtype=dtype, device=device)
            f(proj[r].to(device), lay, *args, state, out, *rest)
            assert bool((out[:, :16] == 3.0).all()) and not bool(out[:, 16 + width:].any())
            return out[:, 16:16 + width]

        got = _walk(n, device, lambda r, cu, m, st, own, _: run(ops.min_gru_prefill, r, cu, m, st, own),
                    lambda r, pos, own: run(ops.min_gru_decode, r, pos, own))
        close(got, want, tol=1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [24, 21, 1100])
def test_wkv_mixes_of_neighbours(device, width):
    n, gen = 40, torch.Generator().manual_seed(width)
    mu = torch.rand(5, width, generator=gen)
    for dtype in dtypes(device):
        h = torch.randn(2 * n, width, generator=gen).to(dtype)
        x = h.double().view(2, n, width)
        before = torch.stack([O.shifted(s) for s in x])
        want = (x[None] + (before - x)[None] * mu.double()[:, None, None]).view(5, 2 * n, width)
        last, m = _filled(device, 4, width), mu.to(device)
        flat = lambda y: y.transpose(0, 1).reshape(y.shape[1], -1)
        got = _walk(n, device,
                    lambda r, cu, _, st, own, seq: flat(ops.wkv_mix_prefill(h[r].to(device), m, last, seq, cu, st, own)),
                    lambda r, pos, own: flat(ops.wkv_mix_decode(h[r].to(device), m, last, pos, own)), cuts=([1, 3], [2, 1], [9, 20], [2, 2]))
        close(got, flat(want), tol=1e-6 if dtype == torch.float32 else 1e-2)
        close(last[torch.tensor([2, 0], device=device)], x[:, -1], tol=1e-7)


def _wkv_case(t, h, d, rank, dtype, seed=0):
    g = torch.Generator().manual_seed(seed)
    r, k, v, gate = (torch.randn(t, h * d, generator=g).to(dtype) for _ in range(4))
    a = torch.randn(t, rank, generator=g) * 2
    w2 = (torch.randn(h * d, rank, generator=g) * 1.5 / rank ** 0.5).to(dtype)
    w0 = torch.randn(h * d, generator=g) * 3 - 3           # decays from nothing to almost one
    u, norm = torch.randn(h * d, generator=g), torch.rand(h * d, generator=g) + 0.5
    return (r, k, v, gate), a, ops.WKVWeights(None, w2, w0, u, norm, h, d)


def _wkv_want(rows, a, w, eps):
    t, h, d = a.shape[0], w.heads, w.dim
    decay = torch.exp(-torch.exp(torch.tanh(a.double()) @ w.w2.double().t() + w.w0.double()))
    r, k, v = (x.double().view(t, h, d) for x in rows[:3])
    o, _ = O.wkv_recurrence(r, k, v, decay.view(t, h, d), w.u.double().view(h, d))
    return O.rms(o, eps).reshape(t, -1) * w.norm.double() * O.silu(rows[3].double())


def _to(w, device):
    return ops.WKVWeights(None, *(x.to(device) for x in (w.w2, w.w0, w.u, w.norm)), w.heads, w.dim)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,d,rank", [(3, 12, 5), (2, 10, 1), (3, 16, 4), (2, 32, 16), (2, 40, 6), (3, 64, 20), (1, 100, 8), (1, 104, 12),
                                       (2, 128, 64), (1, 200, 3)])
@pytest.mark.parametrize("segment,chunked", [(0, True), (0, False), (16, True), (48, True), (48, False)])
def test_wkv_portions_and_decode(device, h, d, rank, segment, chunked, monkeypatch):
    """Sequences from end to end and cut into segments, on the tensor cores and token by token; decays computed ahead of a
    decode step and inside it."""
    if device == "cpu" and (segment or not chunked):
        pytest.skip("one CPU formulation")
    n, eps = 200, 1e-4
    monkeypatch.setattr(W, "DECAY_IN_DECODE", 0 if segment else 8)
    for dtype in dtypes(device):
        if dtype == torch.float32 and not chunked:
            continue
        rows, a, w = _wkv_case(2 * n, h, d, rank, dtype)
        want = torch.cat([_wkv_want([x[i:i + n] for x in rows], a[i:i + n], w, eps) for i in (0, n)])
        wd, state = _to(w, device), _filled(device, 4, h, d, d)
        pick = lambda r: [x[r].to(device) for x in (*rows, a)]
        got = _walk(n, device,
                    lambda r, cu, m, st, own, _: ops.wkv_prefill(*pick(r), wd, state, cu, m, st, own, eps, segment=segment, chunked=chunked),
                    lambda r, pos, own: ops.wkv_decode(*pick(r), wd, state, pos, own, eps))
        close(got, want, tol=5e-5 if dtype == torch.float32 else 2e-2)
        if dtype == torch.bfloat16:
            assert float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) < 3e-3


@pytest.mark.parametrize("device", DEVICES)
def test_wkv_far_write_and_bonus(device):
    """A value written under a channel that keeps comes back far later, one under a channel that forgets does not; the bonus
    counts for the current token only."""
    n, d, far = 300, 16, 5
    rows, a, w = _wkv_case(n, 1, d, 4, torch.float32)
    r, k, v, gate = rows
    for x in (r, k, v):
        x.zero_()
    gate.fill_(1.0)
    w.w2.zero_()
    w.w0.fill_(2.0)                                        # forgets at once, but for entry 3
    w.w0[3] = -30.0
    w.u.fill_(0.0)
    w.u[7] = 2.0
    k[far, 3], k[far, 4], v[far] = 1.0, 1.0, torch.arange(1.0, 17.0)
    r[n - 3, 3], r[n - 2, 4] = 1.0, 1.0
    r[n - 1, 7], k[n - 1, 7], v[n - 1] = 1.0, 1.0, torch.arange(16.0, 0.0, -1.0)
    want = _wkv_want(rows, a, w, 1e-6)
    assert float(want[n - 3].abs().max()) > 1 and float(want[n - 2].abs().max()) < 1e-3 and float(want[n - 1].abs().max()) > 1
    for dtype in dtypes(device):
        wd = _to(ops.WKVWeights(None, w.w2.to(dtype), w.w0, w.u, w.norm, 1, d), device)
        for segment in (0, 32):
            y = ops.wkv_prefill(*(x.to(device, dtype) for x in rows), a.to(device), wd, _filled(device, 1, 1, d, d), i32([0, n], device), n,
                                i32([0], device), i64([0], device), 1e-6, segment=segment)
            assert torch.allclose(y.double().cpu(), want, atol=1e-4 if dtype == torch.float32 else 2e-2)


# ---- layers alone ------------------------------------------------------------------------------------------
def _layer(device, mixer, mlp, n, seed, **kw):
    cfg = M.config([(mixer, mlp)], **kw)
    w, seq, trace = M.weights(cfg, seed), M.tokens(n, cfg["vocab"], 2), []
    O.forward(cfg, w, seq, trace=trace)
    for dtype in dtypes(device):
        eng = make_engine(cfg, w, device, dtype)
        seen = []
        eng.runner.layer_probe = lambda run, r: seen.append(r.float().cpu().clone())
        eng.replay([("a", seq, [])], ["a"])
        if mlp is None:
            close(seen[0], trace[0], dtype)
        else:
            close_routed(seen[0], trace[0], dtype)


MIXER_CASES = {
    "retention": M.retention(), "retention_one_head": M.retention(1, 4, 3, (0.97,)), "retention_wide_values": M.retention(2, 20, 150, (0.9, 0.99)),
    "retention_wide_keys": M.retention(1, 260, 17, (0.98,)),
    "parallel": M.parallel(), "parallel_one_head": M.parallel(1, 1, 4, 6, rot_dims=2, width=3), "all_rotated": M.parallel(6, 2, 10, 12, rot_dims=10, width=50),
    "parallel_wide": M.parallel(3, 1, 130, 100, 0.1, rot_dims=66, width=9), "wider_than_tensor_cores": M.parallel(2, 1, 200, 132, 0.1, rot_dims=8),
    "unit_scales": M.parallel(2, 2, 8, 8, 1.0, rot_dims=8, width=8, left=1.0, right=1.0),
    "wkv": M.wkv(), "wkv_one_head": M.wkv(1, 3, 2), "wkv_wide": M.wkv(2, 132, 40),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", sorted(MIXER_CASES))
def test_mixer_alone(device, case):
    _layer(device, MIXER_CASES[case], None, 37, 5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("mlp", [(5, 2, 24), (3, 3, 8), (1, 1, 64), (65, 7, 16)], ids=str)
def test_feed_forward(device, mlp):
    _layer(device, M.retention(1, 4, 3, (0.9,)), M.moe(*mlp), 50, 6, width=64)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 1, 3), (1, 3, 2), (0, 3, 2), (2, 3, 4)], ids=str)
def test_residual_stream_of_every_pass(device, loop):
    """The stream after every layer run, each pass with a state of its own and its inputs, none of them inside the probe."""
    cfg = M.config([(M.wkv(2, 6, 3), None), (M.retention(), None), (M.parallel(), None)], loop=loop)
    w, seq, trace = M.weights(cfg, 4), M.tokens(23, cfg["vocab"]), []
    want = O.forward(cfg, w, seq, trace=trace)
    eng = make_engine(cfg, w, device)
    seen = []
    eng.runner.layer_probe = lambda run, r: seen.append((run, r.float().cpu().clone()))
    close(eng.replay([("a", seq, list(range(23)))], ["a"]), want)
    assert [r for r, _ in seen] == list(range(len(trace)))
    for (_, got), t in zip(seen, trace):
        close(got, t)


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
@pytest.mark.parametrize("cuts", [[1], [2], [3], [5, 2], [16], [17, 1, 1, 2], [33, 4, 1]], ids=str)
def test_portions(device, cuts):
    n = 50
    for name in ("mixed", "late_loop", "once"):
        seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
        close(run_schedule(engine(name, device, block=4), seq, cuts), want)
    if device == "cuda":
        close_routed(run_schedule(engine("mixed", device, torch.bfloat16), M.tokens(n, M.ZOO["mixed"]["vocab"]), cuts),
                     _expected("mixed", n), torch.bfloat16, 0.7)


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[1], [2], [40, 7], [129, 1]], ids=str)
def test_bf16_does_not_depend_on_the_cut(cuts):
    """The same bf16 model whole and in portions: without close calls of a router the two differ by rounding only."""
    cfg = M.config([(M.wkv(2, 64, 24), M.moe(4, 4, 64)), (M.parallel(8, 2, 64, 64, 0.3, rot_dims=32, width=96), M.moe(3, 3, 64)),
                    (M.retention(2, 48, 80, (0.99, 0.9)), None)], width=128, loop=(0, 2, 2))
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
    for name in ("mixed", "late_loop", "no_loop"):
        close(run_schedule(engine(name, device), M.tokens(12, M.ZOO[name]["vocab"]), [1]), _expected(name, 12))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["retention", "parallel", "wkv"])
def test_one_kind_of_layer_only(device, case):
    cfg = M.config([(MIXER_CASES[case], M.moe()), (MIXER_CASES[case], None)], loop=(0, 2, 2))
    w, seq = M.weights(cfg, 8), M.tokens(40, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = make_engine(cfg, w, device, graphs=(1,) if device == "cuda" else ())
    assert (eng.kv_bytes_per_block() == 0) == (case != "parallel")
    close(run_schedule(eng, seq, [11, 6, 1]), want)
    out = eng.generate([seq[:9]], SamplingParams(n=2, temperature=0.0, max_tokens=5))[0].outputs
    assert out[0].token_ids == out[1].token_ids and out[0].token_ids[0] == int(want[8].argmax())


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    n = 220
    eng = engine("mixed", device, graphs=(1, 2) if device == "cuda" else ())
    close(run_schedule(eng, M.tokens(n, M.ZOO["mixed"]["vocab"]), [10, 1]), _expected("mixed", n))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "late_loop"])
def test_a_far_token_is_remembered(device, name):
    """Two sequences that differ in their first token have different logits at the end, the oracle's in both."""
    vocab, n = M.ZOO[name]["vocab"], 60
    a = M.tokens(n, vocab, 4)
    b = [(a[0] + 7) % vocab] + a[1:]
    want = [O.forward(M.ZOO[name], _weights(name), s) for s in (a, b)]
    assert float((want[0][-1] - want[1][-1]).abs().max()) > 1e-3
    for s, w in zip((a, b), want):
        close(run_schedule(engine(name, device), s, [7, 1])[-1:], w[-1:])


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
@pytest.mark.parametrize("name", ["many_heads", "mixed", "wide_heads"])
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
    close(got[1].flatten(0, 1), got[0].flatten(0, 1), dtype, tol=1e-5 if dtype == torch.float32 else 1e-2)


# ---- framework ------------------------------------------------------------------------------------------
def test_configuration_and_loading_errors(tmp_path):
    cfg = M.ZOO["mixed"]
    folder = M.save(cfg, _weights("mixed"), str(tmp_path / "m"))
    c, w = registry.load_model(folder, torch.float32, "cpu")
    assert c.architecture == "Lunelorn" and len(w.layers) == 3 and c.is_moe and c.is_recurrent and c.windows == (None,)
    assert w.lm_head.data_ptr() != w.embed.data_ptr() and c.pass_starts == {0: 0, 2: 1}
    assert HybridConfig.from_json(M.ZOO["late_loop"]).pass_starts == {1: 0, 3: 1, 5: 2}
    for change, message in (({"l0.mix.stray": torch.zeros(3)}, "stray"), ({"head": torch.zeros(3, 3)}, "head"),
                            ({"side.embed": torch.zeros(61, 3)}, "side.embed"), ({"loop.step": torch.zeros(3, 48)}, "loop.step")):
        with pytest.raises(ValueError, match=message):
            build_hybrid_weights(c, {**_weights("mixed"), **change}, "cpu")
    with pytest.raises(KeyError, match="z.b"):
        build_hybrid_weights(c, {k: v for k, v in _weights("mixed").items() if k != "l1.mix.right.z.b"}, "cpu")
    for layers, message in (([(M.parallel(5, 2), None)], "divide"), ([(M.parallel(rot_dims=7), None)], "even"),
                            ([(M.parallel(vdim=9), None)], "even"), ([(M.retention(2), None)], "decays"),
                            ([(M.retention(), M.moe(3, 4))], "top 4"), ([({"type": "attention", "mixer": {}}, None)], "mixer type")):
        with pytest.raises(ValueError, match=message):
            HybridConfig.from_json(M.config(layers))
    with pytest.raises(ValueError, match="prefix caching"):
        LLMEngine(c, "cpu", enable_prefix_caching=True)


def test_cache_follows_the_layers():
    eng = engine("late_loop", "cpu")
    cache = eng.runner.cache
    assert [sorted(r) for r in cache.rows] == [["k", "v"]] + [[]] * 6
    assert [sorted(s) for s in cache.slots] == [["state"]] + [["memory"], ["last", "state"]] * 3
    assert eng.kv_bytes_per_block() == 16 * 4 * 3 * (12 + 16)
    assert eng.state_bytes() == 8 * 4 * (24 + 3 * (2 * 16 * 32 + 42 + 2 * 10 * 10))


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
