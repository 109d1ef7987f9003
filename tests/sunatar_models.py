"""Small random models for the Sunatar tests: configurations as ``config.json`` holds them, weights by name."""
from __future__ import annotations

import torch

from pumotar_models import save, tokens  # noqa: F401  (the same file formats)

SCALING = {"factor": 3.0, "low": 1.0, "high": 3.0, "original": 40}


def attention(heads=4, kv_heads=2, dim=12, vdim=10, window=9, scale=0.4, base=100.0, rot_dims=8, scaling=SCALING, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
         "rot": {"base": base, "dims": rot_dims}}
    if scaling:
        m["rot"]["scaling"] = scaling
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def mlstm(heads=3, dim=12, vdim=20, gate_cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def moe(experts=5, top=2, ff=24, shared_ff=16):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff}
    return out


def config(layers, width=48, vocab=61, eps=1e-4, scale=1.7):
    return {"architecture": "Sunatar", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "layers": [{**mixer, "mlp": mlp} for mixer, mlp in layers]}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights with lively parts: peaked soft-max, gates that reach their cap, scores far from one half, means of
    rows far from zero (so that a norm without the mean shows)."""
    g = torch.Generator().manual_seed(seed)
    w_, v = cfg["width"], cfg["vocab"]
    out = {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).to(dtype)

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    def glu(p, ff, gain=1.5):
        lin(p + "gate", ff, w_, gain)
        lin(p + "up", ff, w_, gain)
        lin(p + "down", w_, ff)

    out["embed"] = (0.7 + torch.randn(v, w_, generator=g)).to(dtype)
    lin("head", v, w_)
    vec("final.norm", w_, 1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", w_, 1.0)
        h, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            for n, rows in (("q", h * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * dv)):
                lin(p + "mix." + n, rows, w_)
                vec(p + f"mix.{n}.b", rows, 0.1, 0.5)
            vec(p + "mix.q.norm", h * d, 1.3)
            vec(p + "mix.k.norm", m["kv_heads"] * d, 1.3)
            out[p + "mix.vmix"] = torch.tensor(0.2 + 0.15 * i).to(dtype)
        else:
            for n, rows in (("q", h * d), ("k", h * d), ("v", h * dv), ("g", h * dv)):
                lin(p + "mix." + n, rows, w_, 1.5)
            vec(p + "mix.norm", h * dv, 1.0)
            lin(p + "mix.i", h, w_, 3.0)
            vec(p + "mix.i.b", h, -0.5, 2.0)
            lin(p + "mix.f", h, w_, 2.0)
            vec(p + "mix.f.b", h, 3.5, 1.0)            # long memories among short ones
        lin(p + "mix.o", w_, h * dv)
        f = layer.get("mlp")
        if f is None:
            continue
        for e in range(f["router"]["experts"]):
            glu(p + f"mlp.e{e}.", f["expert"]["ff"])
        lin(p + "mlp.router", f["router"]["experts"], w_, 2.0)
        if f.get("shared"):
            glu(p + "mlp.shared.", f["shared"]["ff"])
    return out


# a set of shapes that differ from one another in every size; names say what is special about each
ZOO = {
    "mixed": config([(attention(), moe()), (mlstm(), moe(7, 3, 20)), (attention(6, 2, 14, 10, 17, rot_dims=14), moe(4, 1, 9, 0))]),
    "memory_first": config([(mlstm(2, 20, 8, 5.0), moe(6, 2, 12)), (attention(3, 1, 10, 6, 4, rot_dims=4, v_mix=False), None),
                            (attention(5, 5, 6, 14, 23, rot_dims=6, scaling=None), moe(4, 4, 31)), (mlstm(4, 9, 33, 20.0), None),
                            (attention(7, 7, 16, 10, 11), moe())], width=64, vocab=97, eps=1e-3),
    "values_regrouped": config([(attention(4, 2, 12, 12, 7), moe(3, 2, 16)), (attention(6, 3, 10, 8, 12, rot_dims=6), moe(8, 2, 32)),
                                (attention(4, 4, 20, 6, 30, rot_dims=20), None)], width=36, vocab=33, scale=0.6),
    "wide_heads": config([(attention(4, 1, 96, 72, 33, 0.15, rot_dims=64), moe(4, 2, 64, 64)), (mlstm(2, 80, 144, 12.0), moe(9, 4, 64)),
                          (attention(2, 1, 160, 72, 20, 0.1, rot_dims=40), None), (attention(2, 1, 64, 72, 70, 0.15, rot_dims=64), None)],
                         width=80, vocab=71),
    "many_heads": config([(attention(40, 2, 16, 24, 19, 0.4, rot_dims=16), None), (mlstm(12, 36, 40), moe(70, 6, 24, 40)),
                          (attention(24, 24, 16, 2, None), None)], width=128, vocab=90),
}
