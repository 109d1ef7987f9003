"""Small random models for the Gapevik tests: configurations as ``config.json`` holds them, weights by name."""
from __future__ import annotations

import torch

from pumotar_models import save, tokens  # noqa: F401  (the same file formats)


def attention(heads=4, kv_heads=2, dim=12, vdim=10, conv=3, chunk=9, scale=0.5, softcap=5.0, base=100.0, rot_dims=8):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "softcap": softcap,
         "rot": {"base": base, "dims": rot_dims}}
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m}


def latent(heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=24, q_rank=20, window=11, scale=0.35, base=50.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=12, vdim=8, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts=5, identity=2, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}}


def config(layers, width=48, vocab=61, eps=1e-4, scale=1.7, mult=0.6, weights_of=()):
    """``weights_of``: (layer, owner) pairs; the layer repeats its owner's entry."""
    out = {"architecture": "Gapevik", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "residual_mult": mult, "layers": [{**mixer, "mlp": mlp} for mixer, mlp in layers]}
    for i, j in weights_of:
        out["layers"][i] = {**out["layers"][j], "weights_of": j}
    return out


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights with lively parts: peaked soft-max that reaches its cap, sinks that matter, corrections that change
    the choice of experts, gates that open and close, decays that span short and long memories."""
    g = torch.Generator().manual_seed(seed)
    w_, v = cfg["width"], cfg["vocab"]
    out = {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).to(dtype)

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    def conv(name, rows, taps):
        out[name] = (torch.randn(rows, taps, generator=g) * 0.7).to(dtype)

    out["embed"] = torch.randn(v, w_, generator=g).to(dtype)
    vec("final.norm", w_, 1.0)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", w_, 1.0)
        h, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            for n, rows in (("q", h * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * dv)):
                lin(p + "mix." + n, rows, w_)
                conv(p + f"mix.{n}.conv", rows, m["conv"])
            vec(p + "mix.q.norm", d, 1.3)
            vec(p + "mix.k.norm", d, 1.3)
            lin(p + "mix.g", h, w_, 1.5)
        elif layer["type"] == "latent_attention":
            lin(p + "mix.dq", m["q_rank"], w_)
            vec(p + "mix.dq.norm", m["q_rank"], 1.3)
            lin(p + "mix.uq", h * (d + m["rot_dim"]), m["q_rank"], 1.5)
            lin(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], w_)
            vec(p + "mix.dkv.norm", m["kv_rank"], 1.2)
            lin(p + "mix.uk", h * d, m["kv_rank"], 1.3)
            lin(p + "mix.uv", h * dv, m["kv_rank"])
            vec(p + "mix.sink", h, 1.5, 1.0)
            lin(p + "mix.g", h, w_, 1.5)
        else:
            kd, hv = m["kv_heads"] * d, h * dv
            for n, rows in (("q", kd), ("k", kd), ("v", hv)):
                lin(p + "mix." + n, rows, w_)
                conv(p + f"mix.{n}.conv", rows, m["conv"])
            lin(p + "mix.b", h, w_)
            lin(p + "mix.a", h, w_)
            vec(p + "mix.dt_bias", h, 0.0, 1.0)
            out[p + "mix.A_log"] = (torch.rand(h, generator=g) * 5 - 4).to(dtype)
            vec(p + "mix.norm", dv, 1.0)
            lin(p + "mix.g", hv, w_, 1.5)
        lin(p + "mix.o", w_, h * dv)
        f = layer.get("mlp")
        if f is None:
            continue
        vec(p + "norm2", w_, 1.0)
        n = f["router"]["experts"] + f["router"].get("identity", 0)
        for e in range(f["router"]["experts"]):
            lin(p + f"mlp.e{e}.gate", f["expert"]["ff"], w_, 1.5)
            lin(p + f"mlp.e{e}.up", f["expert"]["ff"], w_, 1.5)
            lin(p + f"mlp.e{e}.down", w_, f["expert"]["ff"], 2.0)
        lin(p + "mlp.router", n, w_, 1.5)
        vec(p + "mlp.correction", n, 0.0, 0.25)
    return out


# a set of shapes that differ from one another in every size; names say what is special about each
ZOO = {
    "mixed": config([(attention(), moe()), (latent(), moe(4, 3, 3, 20)), (delta(), moe(7, 1, 2, 9)), (attention(), moe())],
                    weights_of=[(3, 0)]),
    "odd_sizes": config([(delta(6, 3, 10, 7, 5), None), (latent(5, 9, 10, 11, 19, 13, 5), moe(3, 5, 4, 13)),
                         (attention(6, 3, 14, 9, 2, 16, rot_dims=6), moe(6, 2, 1, 31)), (delta(3, 1, 6, 5, 2), moe(2, 1, 3, 12)),
                         (latent(5, 9, 10, 11, 19, 13, 5), None)], width=42, vocab=53, eps=1e-3, mult=0.35, weights_of=[(4, 1)]),
    "one_tap": config([(attention(1, 1, 6, 6, 1, 4, rot_dims=6, softcap=50.0), moe(3, 0, 3, 16)), (delta(2, 2, 20, 20, 1), moe(2, 2, 1, 8)),
                       (latent(1, 6, 6, 6, 7, 9, 1), None)], width=36, vocab=33, scale=0.6, mult=1.0),
    "wide_heads": config([(attention(4, 1, 80, 72, 4, 33, 0.07, 9.0, rot_dims=64), moe(4, 2, 2, 64)), (delta(2, 1, 72, 100, 3), None),
                          (attention(2, 1, 160, 72, 3, 20, 0.05, rot_dims=40), None), (latent(2, 96, 32, 80, 72, 40, 33, 0.08), None),
                          (latent(2, 128, 64, 128, 112, 56, None, 0.06), moe(3, 1, 2, 40)),
                          (attention(2, 2, 200, 132, 2, None, 0.05, rot_dims=66), None)], width=80, vocab=71),
    "many_heads": config([(attention(40, 2, 16, 24, 4, 19, 0.4, rot_dims=16), None), (latent(40, 8, 16, 24, 136, 100, 27, 0.3), moe(60, 10, 6, 24)),
                          (delta(12, 3, 36, 40, 4), moe(9, 3, 4, 64))], width=128, vocab=90),
}
