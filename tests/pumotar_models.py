"""Small random models for the Pumotar tests: configurations as ``config.json`` holds them, weights by name."""
from __future__ import annotations

import torch


def latent(heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=24, scale=0.3, base=500.0, rot_dims=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}}


def delta(heads=4, kv_heads=2, dim=12, vdim=8, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, limit=0.7, shared_ff=16, shared_limit=1.3):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def config(layers, width=48, vocab=61, loop=None, eps=1e-4, scale=1.7):
    out = {"architecture": "Pumotar", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "layers": [{**mixer, "mlp": mlp} for mixer, mlp in layers]}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def weights(cfg, seed=0, low_rank=10, dtype=torch.bfloat16):
    """Random weights with lively gates: clamps bind, soft-max is peaked, decays span short and long memories."""
    g = torch.Generator().manual_seed(seed)
    w_, v = cfg["width"], cfg["vocab"]
    out = {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).to(dtype)

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    lin("embed", v, w_, w_ ** 0.5)
    vec("final.norm", w_)

    def glu(p, ff, gain=1.0):
        lin(p + "gate", ff, w_, gain)
        lin(p + "up", ff, w_, gain)
        lin(p + "down", w_, ff)

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", w_)
        if layer["type"] == "latent_attention":
            h = m["heads"]
            lin(p + "mix.q", h * (m["dim"] + m["rot_dim"]), w_, 2.0)
            lin(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], w_, 2.0)
            vec(p + "mix.dkv.norm", m["kv_rank"], 1.0)
            lin(p + "mix.uk", h * m["dim"], m["kv_rank"])
            lin(p + "mix.uv", h * m["vdim"], m["kv_rank"])
            lin(p + "mix.o", w_, h * m["vdim"])
        else:
            kd, hv = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", kd), ("k", kd), ("v", hv)):
                lin(p + f"mix.{n}", rows, w_)
                out[p + f"mix.{n}.conv"] = (torch.randn(rows, m["conv"], generator=g) * 0.7).to(dtype)
            lin(p + "mix.b", m["heads"], w_)
            out[p + "mix.A_log"] = (torch.rand(m["heads"], generator=g) * 5 - 4).to(dtype)
            vec(p + "mix.norm", m["vdim"], 1.0)
            lin(p + "mix.a1", low_rank, w_)
            lin(p + "mix.a2", m["heads"] * m["dim"], low_rank, 2.0)
            vec(p + "mix.dt_bias", m["heads"] * m["dim"], 0.0, 1.0)
            lin(p + "mix.g1", low_rank, w_)
            lin(p + "mix.g2", hv, low_rank, 2.0)
            lin(p + "mix.o", w_, hv)
        f = layer.get("mlp")
        if f is None:
            continue
        vec(p + "norm2", w_)
        if f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
        else:
            e, top = f["router"]["experts"], f["router"]["top"]
            for x in range(e):
                glu(p + f"mlp.e{x}.", f["expert"]["ff"], 1.5)
            out[p + "mlp.table"] = torch.stack([torch.randperm(e, generator=g)[:top] for _ in range(v)]).to(torch.int32)
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"], 1.5)
                lin(p + "mlp.shared.sg", 1, w_)
    return out


def save(cfg, w, folder):
    import json
    import os

    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({k: t.contiguous() for k, t in w.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# a set of shapes that differ from one another in every size; names say what is special about each
ZOO = {
    "mixed": config([(delta(), dense()), (latent(), moe()), (delta(4, 4, 8, 12, 2), moe(4, 1, 20))], loop=(1, 3, 2)),
    "grouped_heads": config([(delta(6, 2, 16, 24, 3), moe(7, 3, 32)), (latent(2, 16, 4, 32, 40), dense(24))], width=64, vocab=97),
    "one_tap": config([(delta(2, 1, 20, 20, 1), None), (latent(1, 6, 6, 6, 7, rot_dims=4), moe(3, 3, 9, shared_ff=0))],
                      width=36, vocab=33),
    "odd_sizes": config([(delta(3, 3, 10, 7, 5), dense(27)), (latent(5, 9, 10, 11, 19), moe(6, 4, 13, shared_ff=11))], width=42,
                        vocab=53, loop=(0, 2, 3)),
    "wide_heads": config([(latent(2, 96, 32, 80, 72, scale=0.08), dense(64)), (delta(2, 2, 72, 100, 4), None),
                          (latent(2, 128, 64, 128, 112, scale=0.05), None)], width=80, vocab=71, loop=(0, 1, 2)),
    "many_heads": config([(latent(40, 8, 16, 24, 136, scale=0.2), None), (delta(12, 3, 36, 40, 4), moe(9, 4, 64, shared_ff=64))],
                         width=128, vocab=90),
}
