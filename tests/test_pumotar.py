"""Pumotar decoders through the rollout engine against the plain restatement in ``pumotar_oracle`` (fp64).

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

import pumotar_models as M
import pumotar_oracle as O
from mindspeed_rl_b200 import ops
from mindspeed_rl_b200.models import registry
from mindspeed_rl_b200.models.hybrid_config import HybridConfig
from mindspeed_rl_b200.rollout.engine import LLMEngine
from mindspeed_rl_b200.rollout.hybrid_weights import build_hybrid_weights
from mindspeed_rl_b200.rollout.layer_cache import OutOfSlots, StateSlots
from mindspeed_rl_b200.rollout.scheduler import SamplingParams

CUDA = pytest.param("cuda", marks=pytest.mark.gpu)
DEVICES = ["cpu", CUDA]
# bf16: the positions of the worst rounding (nearly tied scores, small norms) reach several times the mean
TOL = {torch.float32: 3e-5, torch.bfloat16: 9e-2}


@functools.lru_cache(maxsize=None)
def _weights(name, seed=0):
    return M.weights(M.ZOO[name], seed)


@functools.lru_cache(maxsize=None)
def _expected(name, n, seed=0):
    """Oracle logits of the first ``n`` tokens of a fixed sequence."""
    return O.forward(M.ZOO[name], _weights(name), M.tokens(n, M.ZOO[name]["vocab"], seed))


def make_engine(name, device, dtype=torch.float32, *, w=None, cfg=None, seqs=8, budget=512, blocks=64, block=16, model_len=512,
                graphs=()):
    cfg = HybridConfig.from_json(cfg or M.ZOO[name], dtype)
    eng = LLMEngine(cfg, device, max_num_seqs=seqs, max_model_len=model_len, max_num_batched_tokens=budget, block_size=block,
                    enforce_eager=not graphs, graph_batch_sizes=graphs)
    eng.runner.bind_weights(build_hybrid_weights(cfg, w or _weights(name), device))
    eng.init_cache(blocks)
    return eng


def close(got, want, dtype=torch.float32, tol=None):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(err.max()) < (tol or TOL[dtype]), (float(err.max()), int(err.argmax()))
    if tol is None and dtype == torch.bfloat16:
        assert float(err.mean()) < 1.5e-2, float(err.mean())


def run_schedule(eng, seq, cuts, rid="r", end=True):
    """Logits of every token of ``seq`` fed in portions of the given sizes (the last size repeats)."""
    at, k, out = 0, 0, []
    while at < len(seq):
        n = min(cuts[min(k, len(cuts) - 1)], len(seq) - at)
        last = at + n == len(seq)
        out.append(eng.replay([(rid, seq[at:at + n], list(range(n)))], [rid] if last and end else []).float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


# ---- mechanisms alone -------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [40, 42, 1100])
def test_norms_and_residual(device, width):
    g = torch.Generator().manual_seed(3)
    x, w, d = (torch.randn(5, width, generator=g) for _ in range(3))
    table, ids = torch.randn(9, width, generator=g), torch.tensor([3, 0, 8, 8, 1])
    w = w[0] * 0.3
    dev = dict(device=device)
    resid, y = ops.embed_norm(ids.to(**dev), table.to(**dev), 0.75, w.to(**dev), 1e-3, 1.0)
    close(resid, table[ids].double() * 0.75, tol=1e-6)
    close(y, O.norm_offset(table[ids].double() * 0.75, w.double(), 1e-3), tol=1e-6)
    resid = x.clone().to(**dev)
    y = ops.add_norm_(resid, d.to(**dev), w.to(**dev), 1e-2, 0.0)
    close(resid, x.double() + d, tol=1e-6)
    close(y, O.rms(x.double() + d, 1e-2) * w, tol=1e-6)
    # a tiny row shows whether eps is inside the root
    tiny = torch.full((1, width), 1e-3)
    y = ops.add_norm_(tiny.clone().to(**dev), torch.zeros(1, width, **dev), torch.zeros(width, **dev), 1e-4, 1.0)
    close(y, tiny.double() / (1e-6 + 1e-4) ** 0.5, tol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("f", [24, 13])
def test_gated_activations(device, f):
    x = torch.randn(7, 2 * f, generator=torch.Generator().manual_seed(1)) * 3
    g, u = x.double().split(f, -1)
    want = {"gelu_tanh": O.gelu_tanh(g) * u, "silu": O.silu(g) * u}
    gc, uc = g.clamp(max=0.9), u.clamp(-0.9, 0.9)
    want["clamped_swish"] = gc * torch.sigmoid(1.702 * gc) * (uc + 1)
    for act, ref in want.items():
        close(ops.glu_fwd(x.to(device), act, 0.9, 1.702), ref, tol=2e-6)
        close(ops.glu_fwd(x.to(device, torch.bfloat16), act, 0.9, 1.702), ref, tol=2e-2)


def _one_layer(mixer, mlp=None, **kw):
    return M.config([(mixer, mlp)], **kw)


MIXER_CASES = {
    "latent": M.latent(), "latent_part_rotated": M.latent(2, 5, 12, 7, 17, rot_dims=6), "latent_one_head": M.latent(1, 4, 2, 3, 5),
    "delta": M.delta(), "delta_one_tap": M.delta(2, 2, 6, 9, 1), "delta_grouped": M.delta(6, 2, 33, 5, 6),
    "delta_single": M.delta(1, 1, 4, 4, 2),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", sorted(MIXER_CASES))
def test_mixer_alone(device, case):
    cfg = _one_layer(MIXER_CASES[case])
    w = M.weights(cfg, 5)
    seq = M.tokens(37, cfg["vocab"], 2)
    trace = []
    O.forward(cfg, w, seq, trace=trace)
    for dtype in (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16):
        eng = make_engine(None, device, dtype, cfg=cfg, w=w)
        seen = []
        eng.runner.layer_probe = lambda run, r: seen.append(r.float().cpu().clone())
        eng.replay([("a", seq, [])], ["a"])
        close(seen[0], trace[0], dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("mlp", ["dense", "moe", "all_experts", "no_shared", "one_expert"])
def test_feed_forward_alone(device, mlp):
    f = {"dense": M.dense(31), "moe": M.moe(), "all_experts": M.moe(3, 3, 8), "no_shared": M.moe(4, 2, 40, shared_ff=0),
         "one_expert": M.moe(1, 1, 64, limit=0.2, shared_ff=5, shared_limit=0.1)}[mlp]
    cfg = _one_layer(M.latent(1, 4, 2, 3, 5), f, width=64)
    w = M.weights(cfg, 6)
    if f["kind"] == "moe":          # the clamps must bind for a good part of the entries
        x = O.norm_offset(w["embed"].double() * cfg["embedding"]["scale"], w["l0.norm2"].double(), 1e-4)
        assert float((x @ w["l0.mlp.e0.gate"].double().t() > f["expert"]["limit"]).double().mean()) > 0.1
    seq = M.tokens(50, cfg["vocab"], 3)
    trace = []
    O.forward(cfg, w, seq, trace=trace)
    for dtype in (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16):
        eng = make_engine(None, device, dtype, cfg=cfg, w=w)
        seen = []
        eng.runner.layer_probe = lambda run, r: seen.append(r.float().cpu().clone())
        eng.replay([("a", seq, [])], ["a"])
        close(seen[0], trace[0], dtype)


def test_looped_layers_run_in_order_with_a_cache_each():
    cfg = HybridConfig.from_json(M.ZOO["mixed"])
    assert cfg.run_order == [0, 1, 2, 1, 2] == O.layer_order(M.ZOO["mixed"])
    assert HybridConfig.from_json(M.ZOO["odd_sizes"]).run_order == [0, 1] * 3
    assert HybridConfig.from_json(M.ZOO["grouped_heads"]).run_order == [0, 1]
    eng = make_engine("mixed", "cpu")
    cache = eng.runner.cache
    assert ["latent" in c for c in cache.rows] == [False, True, False, True, False]
    ptrs = [c["latent"].data_ptr() for c in cache.rows if c] + [c["state"].data_ptr() for c in cache.slots if c]
    assert len(set(ptrs)) == 5
    assert eng.kv_bytes_per_block() == 2 * 16 * (32 + 16) * 4 and eng.state_bytes() > 0


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("taps", [1, 3])
def test_delta_recurrence_far_write(device, taps):
    """A value written under a key of its own is read back unchanged many tokens later when the decay is one, and is
    lost when the key's channels decay."""
    lay = ops.DeltaLayout(1, 1, 8, 8, taps, 0, 8, 16, 24)
    n, far = 203, 6
    proj = torch.zeros(n, 32)
    proj[:, 8 + 1] = 5.0                                   # all other tokens write under channel 1
    proj[far, 8:16] = torch.eye(8)[4] * 5.0
    proj[far, 16:24] = torch.arange(1.0, 9.0)
    proj[-1, 0:8] = torch.eye(8)[4] * 5.0                  # the last token asks for channel 4
    proj[:, 24] = 20.0                                     # write strength one
    conv = torch.zeros(lay.channels, taps)
    conv[:, -1] = 1.0                                      # the current token only
    gate = torch.full((n, 8), 30.0)
    for decay, keeps in ((-40.0, True), (3.0, False)):
        w = ops.DeltaWeights(conv, torch.zeros(1), torch.full((8,), decay), torch.ones(8))
        ring, state = torch.zeros(2, taps, lay.channels), torch.zeros(2, 1, 8, 8)
        t = dict(device=device)
        cu = torch.tensor([0, n], dtype=torch.int32)
        out = ops.delta_prefill(proj.to(**t), torch.zeros(n, 8, **t), gate.to(**t), lay,
                                ops.DeltaWeights(*(x.to(**t) for x in (w.conv, w.a_log, w.dt_bias, w.norm))), ring.to(**t),
                                state.to(**t), torch.zeros(n, dtype=torch.int32, **t), cu.to(**t),
                                torch.zeros(1, dtype=torch.int32, **t), torch.tensor([1], **t), 1e-6)
        v = O.silu(torch.arange(1.0, 9.0).double())
        want = v / v.pow(2).mean().sqrt() if keeps else torch.zeros(8).double()
        assert torch.allclose(out[-1].double().cpu(), want, atol=2e-4), (decay, out[-1])


# ---- schedules --------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_whole_prompt_then_decode(device, name):
    n = 70
    seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
    for dtype in (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16):
        eng = make_engine(name, device, dtype)
        close(run_schedule(eng, seq, [n]), want, dtype)
        close(run_schedule(eng, seq, [30, 1]), want, dtype)
        assert eng.bm.num_free_blocks == 64 and eng.state_slots.num_free == 8


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [5, 2], [16], [17, 1, 1, 2], [33, 4, 1]], ids=str)
def test_portions(device, cuts):
    n = 50
    for name in ("mixed", "odd_sizes"):
        seq, want = M.tokens(n, M.ZOO[name]["vocab"]), _expected(name, n)
        close(run_schedule(make_engine(name, device, block=4), seq, cuts), want)
    if device == "cuda":
        close(run_schedule(make_engine("mixed", device, torch.bfloat16), M.tokens(n, M.ZOO["mixed"]["vocab"]), cuts),
              _expected("mixed", n), torch.bfloat16)


@pytest.mark.parametrize("device", DEVICES)
def test_token_budget_cuts_a_step_without_effect(device):
    seq, want = M.tokens(70, M.ZOO["mixed"]["vocab"]), _expected("mixed", 70)
    eng = make_engine("mixed", device, budget=9)
    got = eng.replay([("a", seq[:40], list(range(40))), ("b", seq[:11], [0, 10]), ("c", seq[:1], [0])])
    close(got, torch.cat([want[:40], want[[0, 10]], want[:1]]))


@pytest.mark.parametrize("device", DEVICES)
def test_unequal_batches_match_each_alone(device):
    vocab = M.ZOO["mixed"]["vocab"]
    lens, total = [1, 2, 17, 40, 5], 46
    seqs = [M.tokens(total, vocab, s) for s in range(len(lens))]
    want = [_expected("mixed", total, s) for s in range(len(lens))]
    eng = make_engine("mixed", device, graphs=(8,) if device == "cuda" else ())
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
    eng = make_engine("mixed", device, blocks=13, block=4, seqs=2)
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
    """Decoding right after a first portion of one token: convolution windows and states that are not full yet."""
    for name in ("mixed", "one_tap", "odd_sizes"):
        n = 12
        close(run_schedule(make_engine(name, device), M.tokens(n, M.ZOO[name]["vocab"]), [1]), _expected(name, n))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["latent", "delta_grouped"])
def test_one_kind_of_layer_only(device, case):
    """A model without recurrent layers takes no state slots, one without attention no cache memory."""
    cfg = M.config([(MIXER_CASES[case], M.moe()), (MIXER_CASES[case], None)], loop=(1, 2, 2))
    w = M.weights(cfg, 8)
    seq = M.tokens(40, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = make_engine(None, device, cfg=cfg, w=w, graphs=(1,) if device == "cuda" else ())
    assert (eng.state_slots is None) == (case == "latent") and (eng.kv_bytes_per_block() == 0) == (case != "latent")
    close(run_schedule(eng, seq, [11, 6, 1]), want)
    out = eng.generate([seq[:9]], SamplingParams(n=2, temperature=0.0, max_tokens=5))[0].outputs
    assert out[0].token_ids == out[1].token_ids and out[0].token_ids[0] == int(want[8].argmax())


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    n = 220
    eng = make_engine("mixed", device, graphs=(1, 2) if device == "cuda" else ())
    close(run_schedule(eng, M.tokens(n, M.ZOO["mixed"]["vocab"]), [10, 1]), _expected("mixed", n))


# ---- attention: single keys that stand out -----------------------------------------------------------
def _peaked(n, lay, target, seed=0):
    """Latent rows and one query whose score stands out at ``target`` through the unrotated part (first head) and
    the rotated part (second head)."""
    g = torch.Generator().manual_seed(seed)
    rows = torch.zeros(n, lay.CP)
    rows[:, :lay.rank] = torch.randn(n, lay.rank, generator=g)
    rows[:, lay.RP:lay.RP + lay.dr] = torch.randn(n, lay.dr, generator=g)
    q = torch.zeros(lay.heads, lay.CP)
    q[0, :lay.rank] = rows[target, :lay.rank] * 3
    q[1, lay.RP:lay.RP + lay.dr] = rows[target, lay.RP:lay.RP + lay.dr] * 8
    q[2:, :] = torch.randn(lay.heads - 2, lay.CP, generator=g)
    q[:, lay.rank:lay.RP] = 0
    q[:, lay.RP + lay.dr:] = 0
    return rows, q


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,rank,dr,bs", [(3, 24, 8, 16), (20, 72, 16, 8), (40, 130, 24, 32), (70, 40, 16, 64), (4, 300, 32, 4)])
def test_decode_attention_keys_at_borders(device, heads, rank, dr, bs):
    lay = ops.LatentLayout(heads, 8, dr, 8, rank, 8 + dr, 8, 0, dr)
    n = 333
    blocks = (n + bs - 1) // bs
    for dtype in (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16):
        targets = [0, 15, 16, 31, 63, 64, 127, 128, 200, n - 2, n - 1]
        lens = [n] * len(targets) + [1, 2, 16, 17, 64, 65]         # and sequences that end there
        targets += [0, 1, 15, 16, 63, 64]
        b = len(lens)
        perm = torch.randperm(b * blocks, generator=torch.Generator().manual_seed(1)).view(b, blocks)
        cache = torch.full((b * blocks, bs, lay.CP), float("nan") if device == "cuda" else 7.0)   # what freed pages hold must not matter
        q = torch.empty(b, heads, lay.CP)
        want = torch.empty(b, heads, lay.RP, dtype=torch.float64)
        for i, (m, target) in enumerate(zip(lens, targets)):
            rows, q[i] = _peaked(m, lay, target, i)
            rows, q[i] = rows.to(dtype).float(), q[i].to(dtype).float()
            for p in range(m):
                cache[perm[i, p // bs], p % bs] = rows[p]
            s = torch.softmax(q[i].double() @ rows.double().t() * 0.5, -1)
            want[i] = s @ rows[:, :lay.RP].double()
            if m > 1:
                assert float(s[0, target]) > 0.9                     # the key does stand out
        for nsplit, t5 in ((None, True), (1, True), (3, True), (5, False), (1, False)):
            got = ops.latent_decode_attention(q.to(device, dtype), cache.to(device, dtype), lay,
                                              perm.to(device, torch.int32), torch.tensor(lens, dtype=torch.int32, device=device),
                                              n, 0.5, nsplit=nsplit, use_tcgen05=t5)
            close(got.reshape(b * heads, -1), want.reshape(b * heads, -1), dtype, tol=1e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("qp,vp,dn,dr", [(20, 10, 12, 8), (64, 64, 40, 16), (128, 128, 64, 64), (192, 128, 128, 64)])
def test_prompt_attention_keys_at_borders(device, qp, vp, dn, dr):
    h, scale = 2, 0.4
    lay = ops.LatentLayout(h, dn, dr, vp, 16, qp, vp, h * qp, dr)
    dtypes = (torch.float32,) if device == "cpu" else (torch.float32, torch.bfloat16)
    for dtype in dtypes:
        for lens_q, lens_k in (([150, 1, 33], [150, 1, 33]), ([40, 2, 65], [170, 2, 130])):
            g = torch.Generator().manual_seed(7)
            tq, tk = sum(lens_q), sum(lens_k)
            k, v = torch.randn(tk, h, qp, generator=g), torch.randn(tk, h, vp, generator=g)
            k[..., dn + dr:] = 0
            q = torch.zeros(tq, h * qp + 16)
            want = torch.zeros(tq, h, vp, dtype=torch.float64)
            k, v = k.to(dtype).float(), v.to(dtype).float()
            q0 = k0 = 0
            for lq, lk in zip(lens_q, lens_k):
                for i in range(lq):
                    pos = lk - lq + i
                    target = [0, pos, max(pos - 1, 0), pos // 2, min(63, pos), min(64, pos), min(31, pos)][i % 7]
                    qi = (k[k0 + target] * (25.0 / dn ** 0.5 / dn ** 0.5)).to(dtype).float()
                    if pos + 1 < lk:               # the next key would win if the mask let it in
                        qi = (qi + k[k0 + pos + 1] * (50.0 / dn)).to(dtype).float()
                    q[q0 + i, :h * qp] = qi.reshape(-1)
                    s = torch.einsum("hd,jhd->hj", qi.double(), k[k0:k0 + pos + 1].double()) * scale
                    want[q0 + i] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[k0:k0 + pos + 1].double())
                q0, k0 = q0 + lq, k0 + lk
            cu = [torch.tensor([0] + list(torch.tensor(x).cumsum(0)), dtype=torch.int32, device=device) for x in (lens_q, lens_k)]
            kv = torch.cat([k.reshape(tk, -1), v.reshape(tk, -1)], 1).to(device, dtype).contiguous()
            got = ops.latent_prefill_attention(q.to(device, dtype), kv, lay, cu[0], cu[1], max(lens_q), scale)
            close(got.view(tq, -1), want.view(tq, -1), dtype, tol=1e-5 if dtype == torch.float32 else 2e-2)


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
    eng = make_engine("mixed", device, graphs=(2, 4) if device == "cuda" else (), **kw)
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
    eng = make_engine("mixed", device, block=4, budget=7, seqs=6, graphs=(8,) if device == "cuda" else ())
    for o, w in zip(eng.generate(prompts, SamplingParams(n=3, temperature=0.0, max_tokens=9)), want):
        for c in o.outputs:
            assert c.token_ids[:len(w)] == w
    a = eng.generate(prompts[:2], SamplingParams(n=4, temperature=1.0, max_tokens=12, seed=5))
    b = make_engine("mixed", device).generate(prompts[:2], SamplingParams(n=4, temperature=1.0, max_tokens=12, seed=5))
    for x, y in zip(a, b):               # sampled: the same draws whatever the batch, the pages and the slots
        assert [c.token_ids for c in x.outputs] == [c.token_ids for c in y.outputs]
        # what was sampled has the log-probability the oracle gives it
        for c in x.outputs:
            ids = x.prompt_token_ids + c.token_ids
            lp = torch.log_softmax(O.forward(M.ZOO["mixed"], _weights("mixed"), ids), -1)
            for j, (tok, got) in enumerate(zip(c.token_ids, c.logprobs)):
                assert abs(float(lp[len(x.prompt_token_ids) - 1 + j, tok]) - got) < 1e-3
    with pytest.raises(ValueError, match="state slots"):
        eng.add_request(None, [1, 2], SamplingParams(n=7))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_graph_decode_is_the_eager_decode(dtype):
    """A captured step advances every state exactly once, also the step whose capture it is."""
    seqs = [M.tokens(40, M.ZOO["many_heads"]["vocab"], s) for s in range(3)]
    got = []
    for graphs in ((), (4,)):
        eng = make_engine("many_heads", "cuda", dtype, graphs=graphs)
        eng.replay([(str(i), s[:20 + i], []) for i, s in enumerate(seqs)])
        steps = [eng.replay([(str(i), [s[20 + i + k]], [0]) for i, s in enumerate(seqs)]).float().cpu() for k in range(10)]
        got.append(torch.stack(steps))
    close(got[1].flatten(0, 1), got[0].flatten(0, 1), dtype, tol=1e-5 if dtype == torch.float32 else 1e-2)


# ---- framework ------------------------------------------------------------------------------------------
def test_state_slots():
    s = StateSlots(2)
    assert [s.allocate(), s.allocate()] == [0, 1] and s.num_free == 0
    with pytest.raises(OutOfSlots):
        s.allocate()
    s.free(0)
    with pytest.raises(KeyError):
        s.free(0)
    assert s.allocate() == 0


def test_registry_and_loading_errors(tmp_path):
    cfg = M.ZOO["mixed"]
    M.save(cfg, _weights("mixed"), str(tmp_path / "m"))
    c, w = registry.load_model(str(tmp_path / "m"), torch.float32, "cpu")
    assert c.architecture == "Pumotar" and len(w.layers) == 3 and c.is_moe and c.is_recurrent
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.architecture_of({"architecture": "Nobody"})
    bad = dict(_weights("mixed"))
    bad["l0.mix.stray"] = torch.zeros(3)
    with pytest.raises(ValueError, match="stray"):
        build_hybrid_weights(c, bad, "cpu")
    with pytest.raises(ValueError, match="mixer type"):
        HybridConfig.from_json({**cfg, "layers": [{"type": "x", "mixer": {}, "mlp": None}]})
    with pytest.raises(ValueError, match="prefix caching"):
        LLMEngine(c, "cpu", enable_prefix_caching=True)


def test_registry_serves_the_decoder_family_too(tmp_path):
    from mindspeed_rl_b200.models.gpt import GPTModel, PackedMeta
    from mindspeed_rl_b200.checkpoint.convert import mcore_to_hf, save_hf_state

    raw = dict(architectures=["Qwen2ForCausalLM"], num_hidden_layers=2, hidden_size=32, intermediate_size=48, num_attention_heads=4,
               num_key_value_heads=2, vocab_size=40, rms_norm_eps=1e-6, rope_theta=1e4, max_position_embeddings=64)
    cfg = registry._decoder_config(raw, torch.float32)
    torch.manual_seed(0)
    m = GPTModel(cfg, device="cpu")
    for p in m.parameters():
        p.data.mul_(4.0)
    save_hf_state(mcore_to_hf({(0, 0, 0): dict(m.named_parameters())}, cfg), str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    c, w = registry.load_model(str(tmp_path), torch.float32, "cpu")
    eng = LLMEngine(c, "cpu", max_num_seqs=2, max_model_len=64, block_size=4)
    eng.runner.bind_weights(w)
    eng.init_cache(32)
    seq = M.tokens(14, 40)
    with torch.no_grad():
        want = m.forward_logits(torch.tensor(seq), PackedMeta.from_lengths([14], "cpu"))
    close(run_schedule(eng, seq, [5, 3, 1]), want.double(), tol=1e-4)


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
    assert sorted(os.listdir(out)) == ["0.f32", "7.f32"]
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
