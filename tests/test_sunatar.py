"""Sunatar decoders through the rollout engine against the plain restatement in ``sunatar_oracle`` (fp64).

Every test runs on the CPU formulation; the same tests run on the CUDA kernels on a GPU machine, in true 32-bit and,
where it makes sense, in bf16 with a tolerance of bf16 rounding.
"""
import functools
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import sunatar_models as M
import sunatar_oracle as O
from hybrid_helpers import TOL, close, dtypes, make_engine, run_schedule
from mindspeed_rl_b200 import ops
from mindspeed_rl_b200.models import registry
from mindspeed_rl_b200.models.hybrid_config import HybridConfig, Rotary, WavelengthScaling
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


# ---- mechanisms alone -------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [40, 42, 1100, 9000])
def test_centered_norm_and_sums(device, width):
    g = torch.Generator().manual_seed(3)
    x, w, d, d2 = (torch.randn(5, width, generator=g) for _ in range(4))
    x, w = x + 30.0, w[0] * 0.3 + 1.0                      # a mean far above the spread
    dev = dict(device=device)
    resid = x.clone().to(**dev)
    y = ops.add_norm_(resid, d.to(**dev), w.to(**dev), 1e-2, 0.0, True, delta2=d2.to(**dev))
    s = x.double() + d + d2
    close(resid, s, tol=1e-6)
    close(y, O.layer_norm(s, w.double(), 1e-2), tol=1e-5)
    table, ids = torch.randn(9, width, generator=g) - 2.0, torch.tensor([3, 0, 8, 8, 1])
    resid, y = ops.embed_norm(ids.to(**dev), table.to(**dev), 2.5, w.to(**dev), 1e-3, 0.0, True)
    close(y, O.layer_norm(table[ids].double() * 2.5, w.double(), 1e-3), tol=1e-5)
    tiny = torch.tensor([[1e-3, -1e-3]]).repeat(1, width // 2)     # eps inside the root
    y = ops.add_norm_(tiny.clone().to(**dev), torch.zeros(1, width, **dev), torch.ones(width, **dev), 1e-4, 0.0, True)
    close(y, tiny.double() / (1e-6 + 1e-4) ** 0.5, tol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,top", [(1, 1), (5, 5), (33, 4), (200, 8), (700, 3)])
def test_router_and_input_weights(device, experts, top):
    g = torch.Generator().manual_seed(experts)
    z = torch.randn(19, experts, generator=g) * 4
    z[3] += 60.0                                           # saturated scores are still told apart by their logits
    idx, score = K.route_top(z.to(device), top)
    for t in range(19):
        want = z[t].topk(top).indices
        assert idx[t].cpu().tolist() == want.tolist()
        assert torch.allclose(score[t].cpu(), torch.sigmoid(z[t, want]), atol=1e-6)
    for dtype in dtypes(device):
        for h in (16, 12, 7):
            x = torch.randn(19, h, generator=g).to(device, dtype)
            plan = K.moe_plan(idx, experts)
            rows = K.moe_permute(x, plan, score)[plan.pos.long()].float().cpu().view(19, top, h)
            want = score.cpu()[:, :, None] * x.float().cpu()[:, None]
            assert torch.allclose(rows, want, rtol=1e-6 if dtype == torch.float32 else 1e-2, atol=1e-6)


@pytest.mark.parametrize("scaling", [None, M.SCALING, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 700}])
def test_frequencies(scaling):
    rot = {"dims": 20, "base": 5000.0, "scaling": scaling}
    got = Rotary(20, 5000.0, True, WavelengthScaling(**scaling) if scaling else None).frequencies()
    want = O.frequencies(rot)
    assert all(abs(a - b) <= 1e-12 * b for a, b in zip(got, want))
    if scaling:                                            # all three ranges occur
        plain = O.frequencies({"dims": 20, "base": 5000.0})
        kinds = {"kept" if math.isclose(a, b) else "divided" if math.isclose(a * scaling["factor"], b) else "blended"
                 for a, b in zip(got, plain)}
        assert kinds == {"kept", "divided", "blended"}
    table = ops.angle_table(64, got, "cpu")
    assert torch.allclose(table[37, 3], torch.tensor(math.cos(37 * want[3])), atol=1e-6)
    assert torch.allclose(table[37, 13], torch.tensor(math.sin(37 * want[3])), atol=1e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,d,dv,qp,vp,rot,other", [(4, 2, 12, 10, 16, 12, 8, None), (3, 3, 6, 5, 6, 5, 6, (5, 7)),
                                                      (8, 2, 96, 64, 128, 128, 64, (64, 128)), (6, 2, 40, 24, 64, 64, 16, (16, 64))])
def test_norm_rotation_and_value_mixing(device, h, g, d, dv, qp, vp, rot, other):
    t, gen = 11, torch.Generator().manual_seed(5)
    lay = ops.GroupedHeads(h, g, d, dv, qp, vp, 0, h * qp, h * qp + g * qp)
    pos = torch.tensor([0, 1, 5, 30, 31, 2, 9, 17, 3, 3, 8], dtype=torch.int32)
    slots = torch.tensor([3, -1, 0, 7, 12, 20, 31, 1, 2, 4, 5])
    rots = {"dims": rot, "base": 50.0, "scaling": M.SCALING}
    table = ops.angle_table(64, tuple(O.frequencies(rots)), "cpu")
    q, k, v = torch.randn(t, h, d, generator=gen) * 3, torch.randn(t, g, d, generator=gen), torch.randn(t, g, dv, generator=gen)
    qn, kn = torch.rand(h, d, generator=gen) + 0.5, torch.rand(g, d, generator=gen) + 0.5
    od, op = other or (dv, vp)
    first = torch.randn(t, g * dv // od if other else g, od, generator=gen) if g * dv % od == 0 else None
    mix = torch.tensor([0.3])

    def pad(x, to):
        return torch.nn.functional.pad(x, (0, to - x.shape[-1]))

    for dtype in dtypes(device):
        q, k, v = (x.to(dtype).float() for x in (q, k, v))
        proj = torch.cat([pad(q, qp).reshape(t, -1), pad(k, qp).reshape(t, -1), pad(v, vp).reshape(t, -1)], 1).to(device, dtype)
        kc, vc = torch.zeros(8, 4, g, qp, device=device, dtype=dtype), torch.zeros(8, 4, g, vp, device=device, dtype=dtype)
        src = None if other is None else ops.ValueSource(pad(first, op).reshape(t, -1).to(device, dtype), od, op)
        ops.qkv_prep_(proj, lay, pad(qn, qp).reshape(-1).to(device), pad(kn, qp).reshape(-1).to(device), 1e-2, table.to(device),
                      pos.to(device), slots.to(device), kc, vc, src, mix.to(device))
        tol = 1e-6 if dtype == torch.float32 else 6e-3
        full = torch.zeros(64, h, d, dtype=torch.float64)
        got = lay.split(proj.cpu().float())
        for x, w, n, y in ((q, qn, h, got[0]), (k, kn, g, got[1])):
            x = (O.rms(x.double().reshape(t, -1), 1e-2) * w.double().reshape(-1)).view(t, n, d)
            for i in range(t):                             # the rotation of one row at its position
                full = torch.zeros(int(pos[i]) + 1, n, d, dtype=torch.float64)
                full[-1] = x[i]
                close(y[i, :, :d], O.rotate_halves(full, rots)[-1], tol=tol)
            assert float(y[..., d:].abs().sum()) == 0
        want = v.double() if other is None else O.mix_values(v.double(), first.to(dtype).double().reshape(t, g, dv), 0.3)
        close(got[2][..., :dv].reshape(t, -1), want.reshape(t, -1), tol=tol)
        flat_k, flat_v = kc.cpu().float().view(-1, g, qp), vc.cpu().float().view(-1, g, vp)
        for i, s in enumerate(slots.tolist()):
            if s >= 0:
                assert torch.equal(flat_k[s], got[1][i]) and torch.equal(flat_v[s], got[2][i])
        unused = [s for s in range(32) if s not in slots.tolist()]
        assert float(flat_k[unused].abs().sum() + flat_v[unused].abs().sum()) == 0


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
    "attention": M.attention(), "one_token_window": M.attention(window=1), "no_window": M.attention(window=None),
    "one_head": M.attention(1, 1, 4, 3, 6, rot_dims=2), "all_rotated": M.attention(6, 2, 10, 12, 8, rot_dims=10, scaling=None),
    "wide": M.attention(3, 1, 130, 100, 12, 0.1, rot_dims=66), "wider_than_tensor_cores": M.attention(2, 1, 200, 132, 12, 0.1),
    "mlstm": M.mlstm(), "mlstm_one_head": M.mlstm(1, 4, 3, 2.0), "mlstm_wide_values": M.mlstm(2, 20, 150),
    "mlstm_wide_keys": M.mlstm(1, 260, 17),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", sorted(MIXER_CASES))
def test_mixer_alone(device, case):
    _layer(device, MIXER_CASES[case], None, 37, 5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("mlp", ["moe", "all_experts", "no_shared", "one_expert", "many"])
def test_parallel_feed_forward(device, mlp):
    f = {"moe": M.moe(), "all_experts": M.moe(3, 3, 8), "no_shared": M.moe(4, 2, 40, shared_ff=0), "one_expert": M.moe(1, 1, 64, 5),
         "many": M.moe(65, 7, 16)}[mlp]
    _layer(device, M.attention(1, 1, 4, 3, 5, rot_dims=2), f, 50, 6, width=64)


# ---- matrix memory --------------------------------------------------------------------------------------
def _memory_case(t, h, d, dv, seed=0, forget=3.0):
    g = torch.Generator().manual_seed(seed)
    dp, vp = (d + 15) // 16 * 16, (dv + 15) // 16 * 16
    lay = ops.MemoryLayout(h, dp, vp, dv, 0, h * dp, 2 * h * dp, 2 * h * dp + h * vp, d ** -0.5, 11.0)
    proj = torch.zeros(t, 2 * h * (dp + vp))
    q, k = (proj[:, c:c + h * dp].view(t, h, dp) for c in (lay.q_col, lay.k_col))
    v, gate = (proj[:, c:c + h * vp].view(t, h, vp) for c in (lay.v_col, lay.g_col))
    q[..., :d], k[..., :d] = torch.randn(t, h, d, generator=g) * 2, torch.randn(t, h, d, generator=g) * 2
    v[..., :dv], gate[..., :dv] = torch.randn(t, h, dv, generator=g), torch.randn(t, h, dv, generator=g)
    z = torch.cat([torch.randn(t, h, generator=g) * 4, torch.randn(t, h, generator=g) * 3 + forget], 1)
    norm = torch.zeros(h, vp)
    norm[:, :dv] = torch.rand(h, dv, generator=g) + 0.5
    return lay, proj, z, ops.MemoryWeights(torch.randn(2 * h, generator=g), norm.reshape(-1))


def _memory_want(lay, proj, z, w, d, eps=1e-5):
    """Oracle output of one sequence, padded as the op pads."""
    t, h, dv = proj.shape[0], lay.heads, lay.rms_dim
    x = proj.double()
    q, k = (x[:, c:c + h * lay.dim].view(t, h, lay.dim)[..., :d] for c in (lay.q_col, lay.k_col))
    v, g = (x[:, c:c + h * lay.vdim].view(t, h, lay.vdim)[..., :dv] for c in (lay.v_col, lay.g_col))
    zz = lay.cap * torch.tanh((z.double() + w.bias.double()) / lay.cap)
    o = O.matrix_memory(q * lay.scale, k, v, zz[:, :h], O.logsigmoid(zz[:, h:]))
    y = O.rms(o, eps) * w.norm.double().view(h, lay.vdim)[:, :dv] * torch.sigmoid(g)
    return torch.nn.functional.pad(y, (0, lay.vdim - dv)).reshape(t, -1)


def _slots(lay, n, device):
    bad = float("nan") if device == "cuda" else 7.0        # what a slot holds before a sequence's first token does not matter
    return {"memory": torch.full((n, lay.heads, lay.dim, lay.vdim), bad, device=device),
            "norm": torch.full((n, lay.heads, lay.dim), bad, device=device), "peak": torch.full((n, lay.heads), bad, device=device)}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,d,dv", [(2, 12, 20), (3, 64, 64), (1, 128, 128), (2, 40, 130), (1, 200, 300)])
@pytest.mark.parametrize("chunked", [False, True])
def test_matrix_memory_portions_and_decode(device, h, d, dv, chunked):
    """Two sequences in portions around the chunk size, then token by token, against the recurrence."""
    if device == "cpu" and chunked:
        pytest.skip("one CPU formulation")
    n = 300 if d * dv < 2e4 else 200
    lay, proj, z, w = _memory_case(2 * n, h, d, dv)
    for dtype in dtypes(device):
        if dtype == torch.float32 and chunked:
            continue
        proj = proj.to(dtype).float()
        want = torch.stack([_memory_want(lay, proj[i * n:(i + 1) * n], z[i * n:(i + 1) * n], w, d) for i in range(2)])
        slots, dev = _slots(lay, 4, device), dict(device=device)
        wd = ops.MemoryWeights(w.bias.to(**dev), w.norm.to(**dev))
        got = torch.zeros_like(want)
        at, owner = [0, 0], torch.tensor([2, 0], **dev)
        for cut in ([127, 1], [1, 130], [2, 3], [130, 60]):
            cut = [min(c, n - a - 3) for c, a in zip(cut, at)]
            rows = torch.cat([torch.arange(i * n + at[i], i * n + at[i] + cut[i]) for i in range(2)])
            y = ops.memory_prefill(proj[rows].to(device, dtype), z[rows].to(**dev), lay, wd, slots,
                                   torch.tensor([0, cut[0], sum(cut)], dtype=torch.int32, **dev), max(cut),
                                   torch.tensor(at, dtype=torch.int32, **dev), owner, 1e-5, chunked=chunked).double().cpu()
            for i in range(2):
                got[i, at[i]:at[i] + cut[i]] = y[:cut[0]] if i == 0 else y[cut[0]:]
                at[i] += cut[i]
        while min(at) < n:
            live = [i for i in range(2) if at[i] < n]
            rows = torch.tensor([i * n + at[i] for i in live] + [0])
            y = ops.memory_decode(proj[rows].to(device, dtype), z[rows].to(**dev), lay, wd, slots,
                                  torch.tensor([at[i] for i in live] + [5], dtype=torch.int32, **dev),
                                  torch.cat([owner[live], torch.tensor([-1], **dev)]), 1e-5).double().cpu()
            for x, i in enumerate(live):
                got[i, at[i]] = y[x]
                at[i] += 1
        close(got.flatten(0, 1), want.flatten(0, 1), tol=2e-5 if dtype == torch.float32 else 2e-2)
        if dtype == torch.bfloat16:                        # inputs are exact: only the result is rounded
            assert float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) < 3e-3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("forget,keeps", [(40.0, True), (-2.0, False)])
def test_matrix_memory_far_write(device, forget, keeps):
    """A value written under a key of its own comes back many tokens later when nothing is forgotten."""
    n, far = 333, 6
    lay, proj, z, w = _memory_case(n, 1, 16, 16)
    w = ops.MemoryWeights(torch.zeros(2), torch.ones(16))
    proj.zero_()
    proj[:, lay.k_col + 1] = 4.0                           # all other tokens write zeros under entry 1
    proj[far, lay.k_col:lay.k_col + 16] = torch.eye(16)[4] * 4
    proj[far, lay.v_col:lay.v_col + 16] = torch.arange(1.0, 17.0)
    proj[-1, lay.q_col:lay.q_col + 16] = torch.eye(16)[4] * 4
    z[:, 0], z[:, 1] = 0.0, forget
    for dtype in dtypes(device):
        dev = dict(device=device)
        y = ops.memory_prefill(proj.to(device, dtype), z.to(**dev), lay, ops.MemoryWeights(w.bias.to(**dev), w.norm.to(**dev)),
                               _slots(lay, 1, device), torch.tensor([0, n], dtype=torch.int32, **dev), n,
                               torch.zeros(1, dtype=torch.int32, **dev), torch.zeros(1, dtype=torch.int64, **dev), 1e-6)
        v = torch.arange(1.0, 17.0).double()
        want = 0.5 * v / v.pow(2).mean().sqrt() if keeps else torch.zeros(16).double()
        assert torch.allclose(y[-1].double().cpu(), want, atol=1e-3 if dtype == torch.float32 else 1e-2), (dtype, y[-1])


def test_running_maximum_starts_at_zero():
    """With small gates from the first token on, the floor exp(-m) and the state carry the scale that a maximum
    started at zero gives."""
    lay, proj, z, w = _memory_case(3, 1, 4, 4, forget=0.0)
    z[:, 0] = -9.0
    y = ops.memory_prefill(proj, z, lay, w, _slots(lay, 1, "cpu"), torch.tensor([0, 3], dtype=torch.int32), 3,
                           torch.zeros(1, dtype=torch.int32), torch.zeros(1, dtype=torch.int64), 1e-5)
    close(y, _memory_want(lay, proj, z, w, 4), tol=1e-5)


# ---- attention: keys at window and page borders ----------------------------------------------------------
def _targets(pos, window):
    """Keys worth asking for from ``pos``: the window's two ends, its neighbours outside, page and tile borders."""
    lo = pos - window + 1
    return [t for t in (lo, lo - 1, pos, pos - 1, lo + 1, pos // 2, 0, 15, 16, 63, 64, 127, 128) if 0 <= t <= pos]


def _peaked(pos, k, window, scale, i):
    """A query whose score stands out at one target; the keys just outside the window would win if they were seen."""
    ts = _targets(pos, window)
    target = ts[i % len(ts)]
    q = k[target] * (14.0 / scale / k.shape[-1])
    for out in (pos - window, pos + 1):
        if 0 <= out < k.shape[0] and out != target:
            q = q + k[out] * (26.0 / scale / k.shape[-1])
    return q


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,qp,vp,window", [(4, 2, 12, 8, 21), (2, 1, 64, 64, 64), (4, 1, 128, 128, 65), (2, 2, 128, 128, 200),
                                              (2, 1, 192, 128, 33), (2, 1, 64, 64, 1), (3, 3, 208, 136, 40)])
def test_prompt_attention_keys_at_window_borders(device, h, g, qp, vp, window):
    scale = 0.4
    lay = ops.GroupedHeads(h, g, qp, vp, qp, vp, 0, h * qp, h * qp + g * qp)
    for dtype in dtypes(device):
        for lens_q, lens_k in (([250, 1, 33], [250, 1, 33]), ([40, 2, 131], [270, 2, 180])):
            gen = torch.Generator().manual_seed(7)
            tq, tk = sum(lens_q), sum(lens_k)
            k, v = (torch.randn(tk, g, n, generator=gen).to(dtype).float() for n in (qp, vp))
            q = torch.zeros(tq, h, qp)
            want = torch.zeros(tq, h, vp, dtype=torch.float64)
            q0 = k0 = hits = 0
            for lq, lk in zip(lens_q, lens_k):
                for i in range(lq):
                    pos = lk - lq + i
                    for x in range(h):
                        q[q0 + i, x] = _peaked(pos, k[k0:k0 + lk, x // (h // g)], window, scale, i + x).to(dtype).float()
                    lo = max(0, pos - window + 1)
                    kk, vv = (y[k0 + lo:k0 + pos + 1].double().repeat_interleave(h // g, 1) for y in (k, v))
                    p = torch.softmax(torch.einsum("hd,jhd->hj", q[q0 + i].double(), kk) * scale, -1)
                    hits += int((p.max() > 0.9))
                    want[q0 + i] = torch.einsum("hj,jhd->hd", p, vv)
                q0, k0 = q0 + lq, k0 + lk
            assert hits > tq // 2                          # keys do stand out
            cu = [torch.tensor([0] + list(torch.tensor(x).cumsum(0)), dtype=torch.int32, device=device) for x in (lens_q, lens_k)]
            proj = torch.zeros(tq, (h + g) * qp + g * vp)
            proj[:, :h * qp] = q.reshape(tq, -1)
            kv = (k.to(device, dtype), v.to(device, dtype))
            if lens_q == lens_k:                           # keys from the same rows
                proj[:, lay.k_col:lay.v_col], proj[:, lay.v_col:] = k.reshape(tk, -1), v.reshape(tk, -1)
                kv = None
            for t5 in ((True, False) if device == "cuda" and qp == 128 else (True,)):
                got = ops.window_prefill_attention(proj.to(device, dtype), lay, cu[0], cu[1], max(lens_q), scale, window, kv,
                                                   use_tcgen05=t5)
                close(got.view(tq, -1), want.view(tq, -1), dtype, tol=1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("h,g,qp,vp,bs,window", [(4, 2, 12, 8, 4, 21), (4, 2, 64, 64, 16, 64), (20, 1, 128, 128, 16, 65),
                                                 (6, 2, 128, 128, 8, 300), (40, 2, 192, 128, 32, 33), (3, 3, 208, 136, 16, 40),
                                                 (2, 1, 64, 64, 16, 1), (4, 4, 128, 128, 64, None)])
def test_decode_attention_keys_at_window_and_page_borders(device, h, g, qp, vp, bs, window):
    n, scale = 333, 0.5
    lay = ops.GroupedHeads(h, g, qp, vp, qp, vp, 0, h * qp, h * qp + g * qp)
    blocks = (n + bs - 1) // bs
    win = window or 10 ** 6
    for dtype in dtypes(device):
        lens = [n] * 7 + [1, 2, bs, bs + 1, min(win, n), min(win + 1, n), min(win + 2, n), 64, 65, 0]
        b = len(lens)
        gen = torch.Generator().manual_seed(1)
        perm = torch.randperm(b * blocks, generator=gen).view(b, blocks)
        fill = float("nan") if device == "cuda" else 7.0   # what freed pages hold must not matter
        kc, vc = torch.full((b * blocks, bs, g, qp), fill), torch.full((b * blocks, bs, g, vp), fill)
        proj = torch.zeros(b, (h + g) * qp + g * vp)
        want = torch.zeros(b, h, vp, dtype=torch.float64)
        for i, m in enumerate(lens):
            k, v = (torch.randn(m, g, x, generator=gen).to(dtype).float() for x in (qp, vp))
            for p in range(m):
                kc[perm[i, p // bs], p % bs], vc[perm[i, p // bs], p % bs] = k[p], v[p]
            if m == 0:
                continue
            q = torch.stack([_peaked(m - 1, k[:, x // (h // g)], win, scale, i + x) for x in range(h)]).to(dtype).float()
            proj[i, :h * qp] = q.reshape(-1)
            lo = max(0, m - win)
            kk, vv = (y[lo:].double().repeat_interleave(h // g, 1) for y in (k, v))
            p = torch.softmax(torch.einsum("hd,jhd->hj", q.double(), kk) * scale, -1)
            want[i] = torch.einsum("hj,jhd->hd", p, vv)
        for nsplit in (None, 1, 3):
            got = ops.window_decode_attention(proj.to(device, dtype), lay, kc.to(device, dtype), vc.to(device, dtype),
                                              perm.to(device, torch.int32), torch.tensor(lens, dtype=torch.int32, device=device), n,
                                              scale, window, nsplit=nsplit)
            close(got.reshape(b * h, -1), want.reshape(b * h, -1), dtype, tol=1e-5 if dtype == torch.float32 else 1.5e-2)


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
        assert eng.bm.num_free_blocks == 64
        assert eng.state_slots.num_free == 8 if eng.cfg.is_recurrent else eng.state_slots is None


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [5, 2], [16], [17, 1, 1, 2], [33, 4, 1]], ids=str)
def test_portions(device, cuts):
    n = 50
    for name in ("mixed", "memory_first", "values_regrouped"):
        seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
        close(run_schedule(engine(name, device, block=4), seq, cuts), want)
    if device == "cuda":
        close_routed(run_schedule(engine("mixed", device, torch.bfloat16), M.tokens(n, M.ZOO["mixed"]["vocab"]), cuts),
                     _expected("mixed", n), torch.bfloat16, 0.7)


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[1], [2], [40, 7], [129, 1]], ids=str)
def test_bf16_does_not_depend_on_the_cut(cuts):
    """The same bf16 model whole and in portions: without close calls of a router the two differ by rounding only."""
    cfg = M.config([(M.attention(8, 2, 64, 64, 40, 0.3, rot_dims=32), M.moe(4, 4, 64, 64)), (M.mlstm(2, 48, 80), M.moe(3, 3, 64)),
                    (M.attention(4, 1, 96, 128, 50, 0.3, rot_dims=96), None)], width=128)
    w, seq = M.weights(cfg, 3), M.tokens(140, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    whole = run_schedule(make_engine(cfg, w, "cuda", torch.bfloat16), seq, [140])
    close(whole, want, torch.bfloat16)
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
    """Decoding right after a first portion of one token: windows and states that are not full yet."""
    for name in ("mixed", "values_regrouped", "memory_first"):
        close(run_schedule(engine(name, device), M.tokens(12, M.ZOO[name]["vocab"]), [1]), _expected(name, 12))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["attention", "mlstm"])
def test_one_kind_of_layer_only(device, case):
    """A model without recurrent layers takes no state slots, one without attention no cache memory."""
    cfg = M.config([(MIXER_CASES[case], M.moe()), (MIXER_CASES[case], None)])
    w, seq = M.weights(cfg, 8), M.tokens(40, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = make_engine(cfg, w, device, graphs=(1,) if device == "cuda" else ())
    assert (eng.state_slots is None) == (case == "attention") and (eng.kv_bytes_per_block() == 0) == (case != "attention")
    close(run_schedule(eng, seq, [11, 6, 1]), want)
    out = eng.generate([seq[:9]], SamplingParams(n=2, temperature=0.0, max_tokens=5))[0].outputs
    assert out[0].token_ids == out[1].token_ids and out[0].token_ids[0] == int(want[8].argmax())


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    n = 220
    eng = engine("mixed", device, graphs=(1, 2) if device == "cuda" else ())
    close(run_schedule(eng, M.tokens(n, M.ZOO["mixed"]["vocab"]), [10, 1]), _expected("mixed", n))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "memory_first"])
def test_a_far_token_reaches_through_the_memory_only(device, name):
    """Two sequences that differ in their first token: past every window the logits still differ where the matrix memory
    carries it, and are the oracle's in both."""
    vocab, n = M.ZOO[name]["vocab"], 60
    a = M.tokens(n, vocab, 4)
    b = [(a[0] + 7) % vocab] + a[1:]
    want = [O.forward(M.ZOO[name], _weights(name), s) for s in (a, b)]
    assert float((want[0][-1] - want[1][-1]).abs().max()) > 1e-4
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
@pytest.mark.parametrize("name", ["many_heads", "values_regrouped", "memory_first"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_graph_decode_is_the_eager_decode(dtype, name):
    """A captured step (its sublayers on two streams) advances every state exactly once, also the step whose capture it
    is."""
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
    assert c.architecture == "Sunatar" and len(w.layers) == 3 and c.is_moe and c.is_recurrent and c.windows == (9, 17)
    assert w.lm_head.data_ptr() != w.embed.data_ptr() and w.layers[0].norm2 is None
    assert HybridConfig.from_json(M.ZOO["many_heads"]).windows == (19, None)
    for change, message in (({"l0.mix.stray": torch.zeros(3)}, "stray"), ({"head": torch.zeros(3, 3)}, "head")):
        with pytest.raises(ValueError, match=message):
            build_hybrid_weights(c, {**_weights("mixed"), **change}, "cpu")
    with pytest.raises(KeyError, match="q.b"):
        build_hybrid_weights(c, {k: v for k, v in _weights("mixed").items() if k != "l0.mix.q.b"}, "cpu")
    for layers, message in (([(M.attention(5, 2), None)], "divide"), ([(M.attention(rot_dims=7), None)], "even"),
                            ([(M.attention(), M.moe(3, 4))], "top 4"), ([({"type": "latent_attention", "mixer": {}}, None)], "mixer type"),
                            ([(M.attention(), None), (M.attention(vdim=11), None)], "value sizes")):
        with pytest.raises(ValueError, match=message):
            HybridConfig.from_json(M.config(layers))
    with pytest.raises(ValueError, match="prefix caching"):
        LLMEngine(c, "cpu", enable_prefix_caching=True)


def test_prefix_caching_without_recurrent_layers():
    cfg = M.config([(M.attention(), M.moe()), (M.attention(window=5), None)])
    w, seq = M.weights(cfg, 2), M.tokens(30, cfg["vocab"])
    eng = LLMEngine(HybridConfig.from_json(cfg, torch.float32), "cpu", max_num_seqs=2, max_model_len=64, block_size=4,
                    enable_prefix_caching=True)
    eng.runner.bind_weights(build_hybrid_weights(eng.cfg, w, "cpu"))
    eng.init_cache(32)
    want = O.forward(cfg, w, seq)
    for _ in range(2):
        out = eng.generate([seq], SamplingParams(temperature=0.0, max_tokens=1))
        assert out[0].outputs[0].token_ids[0] == int(want[-1].argmax())
    assert eng.bm.stats()["prefix_hits"] > 0


def test_cache_follows_the_layers():
    eng = engine("memory_first", "cpu")
    cache = eng.runner.cache
    assert [sorted(r) for r in cache.rows] == [[], ["k", "v"], ["k", "v"], [], ["k", "v"]]
    assert [sorted(s) for s in cache.slots] == [["memory", "norm", "peak"], [], [], ["memory", "norm", "peak"], []]
    assert eng.kv_bytes_per_block() == 16 * 4 * (1 * (12 + 8) + 5 * (8 + 16) + 7 * (16 + 12))
    assert eng.state_bytes() == 8 * 4 * (2 * (32 * 16 + 32 + 1) + 4 * (16 * 48 + 16 + 1))


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
