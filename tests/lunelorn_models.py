"""Small random models for the Lunelorn tests: configurations as ``config.json`` holds them, weights by name."""
from __future__ import annotations

import torch

from pumotar_models import save, tokens  # noqa: F401  (the same file formats)


def retention(heads=3, dim=12, vdim=10, decay=(0.5, 0.9, 0.995)):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def parallel(heads=4, kv_heads=2, dim=12, vdim=10, scale=0.7, base=100.0, rot_dims=8, width=20, left=0.7, right=1.3):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                 "rot": {"base": base, "dims": rot_dims}},
        "right": {"width": width}, "left_scale": left, "right_scale": right}}


def wkv(heads=3, dim=12, rank=6):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "rank": rank}


def moe(experts=5, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width=48, vocab=61, eps=2e-2, side=6, cap=9.0, loop=None):
    """The bottleneck's rank is a matter of the tensors: it stays beside the configuration under ``ranks``."""
    out = {"architecture": "Lunelorn", "norm": {"eps": eps}, "vocab": vocab, "width": width, "token_side": {"dim": side},
           "logit_softcap": cap, "layers": [{"type": m["type"], "mixer": m["mixer"], "mlp": mlp} for m, mlp in layers],
           "ranks": [m.get("rank") for m, _ in layers]}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights with lively parts: peaked soft-max, gates that open and close, decays that span short and long
    memories, token inputs and pass vectors that matter, logits that reach the cap."""
    g = torch.Generator().manual_seed(seed)
    w_, v, n = cfg["width"], cfg["vocab"], len(cfg["layers"])
    dim = cfg["token_side"]["dim"]
    out = {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).to(dtype)

    def vec(name, *size, mean=0.0, std=0.3):
        out[name] = (mean + std * torch.randn(*size, generator=g)).to(dtype)

    vec("embed", v, w_, std=0.4)
    vec("embed.norm", w_, mean=0.9)
    vec("final.norm", w_, mean=1.0)
    lin("head", v, w_, 5.0)
    vec("side.embed", v, n * dim, std=1.0)
    if cfg.get("loop"):
        vec("loop.step", cfg["loop"]["times"], w_, std=0.5)
    for i, (layer, rank) in enumerate(zip(cfg["layers"], cfg["ranks"])):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", w_, mean=1.0)
        vec(p + "norm1b", w_, mean=0.8)
        if layer["type"] == "retention":
            h, d, dv = m["heads"], m["dim"], m["vdim"]
            for t, rows in (("q", h * d), ("k", h * d), ("v", h * dv), ("g", h * dv)):
                lin(p + "mix." + t, rows, w_, 1.5)
            lin(p + "mix.o", w_, h * dv)
        elif layer["type"] == "parallel":
            s, r = m["left"], m["right"]["width"]
            for t, rows in (("q", s["heads"] * s["dim"]), ("k", s["kv_heads"] * s["dim"]), ("v", s["kv_heads"] * s["vdim"])):
                lin(p + "mix.left." + t, rows, w_, 1.3)
            lin(p + "mix.left.o", w_, s["heads"] * s["vdim"])
            for t in "zxg":
                lin(p + "mix.right." + t, r, w_, 1.5)
            vec(p + "mix.right.z.b", r, mean=-2.0, std=2.0)
            vec(p + "mix.right.x.b", r, std=0.7)
            lin(p + "mix.right.o", w_, r)
        else:
            hd = m["heads"] * m["dim"]
            for t in "rkvgw":
                out[p + "mix.mu." + t] = torch.rand(w_, generator=g).to(dtype)
            for t in "rkvg":
                lin(p + "mix." + t, hd, w_, 1.2)
            lin(p + "mix.w1", rank, w_, 1.5)
            lin(p + "mix.w2", hd, rank, 1.5)
            vec(p + "mix.w0", hd, mean=-3.0, std=2.0)
            vec(p + "mix.u", m["heads"], m["dim"], std=1.0)
            vec(p + "mix.norm", hd, mean=1.0)
            lin(p + "mix.o", w_, hd)
        f = layer.get("mlp")
        if f is not None:
            vec(p + "norm2", w_, mean=1.0)
            vec(p + "norm2b", w_, mean=0.8)
            for e in range(f["router"]["experts"]):
                lin(p + f"mlp.e{e}.gate", f["expert"]["ff"], w_, 1.5)
                lin(p + f"mlp.e{e}.up", f["expert"]["ff"], w_, 1.5)
                lin(p + f"mlp.e{e}.down", w_, f["expert"]["ff"], 2.0)
            lin(p + "mlp.router", f["router"]["experts"], w_, 1.5)
        lin(p + "side.gate", dim, w_, 1.5)
        lin(p + "side.proj", w_, dim)
        vec(p + "side.norm", w_, mean=0.6)
    return out


# a set of shapes that differ from one another in every size; names say what is special about each
ZOO = {
    "mixed": config([(wkv(), moe()), (parallel(), moe(4, 1, 20)), (retention(), None)], loop=(0, 2, 2)),
    "late_loop": config([(parallel(6, 3, 10, 14, 0.4, 60.0, 10, 24, 1.1, 0.4), None), (retention(2, 9, 17, (0.3, 0.99)), moe(3, 3, 13)),
                         (wkv(2, 10, 3), moe(6, 1, 31))], width=42, vocab=53, eps=3e-2, side=5, cap=4.0, loop=(1, 3, 3)),
    "no_loop": config([(retention(1, 16, 8, (1.0,)), moe(1, 1, 16)), (wkv(1, 4, 1), None), (parallel(1, 1, 4, 2, 1.0, 30.0, 2, 7, 1.0, 1.0), moe(2, 2, 8))],
                      width=36, vocab=33, side=8, cap=30.0),
    "once": config([(wkv(5, 7, 9), None), (retention(5, 6, 6, (0.0, 0.2, 0.7, 0.97, 0.9995)), moe(7, 3, 9))], width=40, vocab=47, side=1,
                   loop=(1, 2, 1)),
    "wide_heads": config([(parallel(4, 1, 80, 72, 0.07, 5000.0, 64, 100), moe(4, 2, 64)), (retention(2, 72, 130, (0.9, 0.999)), None),
                          (parallel(2, 2, 160, 96, 0.05, rot_dims=40, width=66), None), (wkv(2, 72, 12), None),
                          (parallel(2, 1, 200, 132, 0.05, rot_dims=66, width=40), None), (wkv(1, 136, 8), moe(3, 1, 40))], width=80, vocab=71,
                         side=16, loop=(2, 4, 2)),
    "many_heads": config([(parallel(40, 2, 16, 24, 0.5, rot_dims=16, width=136), moe(60, 6, 24)), (retention(12, 36, 40, [0.8 + 0.016 * i for i in range(12)]), None),
                          (wkv(9, 32, 16), moe(9, 4, 64))], width=128, vocab=90, side=16),
}
