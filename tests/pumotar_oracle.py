"""Plain, slow restatement of the Pumotar equations for the tests: one function per mechanism, token by
token where the mechanism is defined token by token, in double precision by default.  It shares no code
with the product path and reads nothing but a config dictionary and a name -> tensor dictionary.

``forward(cfg, weights, tokens)`` is one sequence from its first token; ``PumotarState`` is not needed here
because every mechanism is written over whole sequences.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_offset(x, w, eps):
    """RMS norm whose stored weight is an offset from one."""
    return rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x [T, ..., d]``: neighbours (2i, 2i+1) of the first ``dims`` entries turn by ``pos * base^(-2i/dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(x.dtype) * float(base) ** (-2.0 * i / dims)
        a = a.view(-1, *([1] * (x.dim() - 2)))
        c, s = torch.cos(a), torch.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Latent attention over one whole sequence ``h [T, W]``; ``w`` maps the names after ``mix.``."""
    t = h.shape[0]
    hn, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(t)
    q = (h @ w["q"].t()).view(t, hn, dn + dr)
    ckr = h @ w["dkv"].t()
    c = rms(ckr[:, :r], eps) * w["dkv.norm"]
    kr = rotate_pairs(ckr[:, r:].unsqueeze(1), pos, m["rot"]["dims"], m["rot"]["base"])[:, 0]
    qr = rotate_pairs(q[..., dn:], pos, m["rot"]["dims"], m["rot"]["base"])
    kn = (c @ w["uk"].t()).view(t, hn, dn)
    v = (c @ w["uv"].t()).view(t, hn, dv)
    out = torch.empty(t, hn, dv, dtype=h.dtype)
    for i in range(t):
        s = torch.einsum("hd,jhd->hj", q[i, :, :dn], kn[:i + 1]) + torch.einsum("hd,jd->hj", qr[i], kr[:i + 1])
        p = torch.softmax(s * m["scale"], dim=-1)
        out[i] = torch.einsum("hj,jhd->hd", p, v[:i + 1])
    return out.reshape(t, hn * dv) @ w["o"].t()


def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal per-channel convolution ``x [T, C]``, ``w [C, taps]`` (last tap = current token), then silu."""
    t, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for i in range(t):
        for k in range(taps):
            j = i - (taps - 1 - k)
            if j >= 0:
                out[i] += x[j] * w[:, k]
    return silu(out)


def delta_recurrence(q, k, v, g, beta, s0: Optional[torch.Tensor] = None):
    """``q, k [T, H, d]``, ``v [T, H, dv]``, ``g [T, H, d]``, ``beta [T, H]`` -> ``o [T, H, dv]``, final state."""
    t, hn, d = k.shape
    s = torch.zeros(hn, d, v.shape[-1], dtype=k.dtype) if s0 is None else s0.clone()
    o = torch.empty(t, hn, v.shape[-1], dtype=k.dtype)
    for i in range(t):
        s = s * g[i].unsqueeze(-1)
        u = beta[i].unsqueeze(-1) * (v[i] - torch.einsum("hdv,hd->hv", s, k[i]))
        s = s + k[i].unsqueeze(-1) * u.unsqueeze(1)
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    return o, s


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t = h.shape[0]
    hn, kvh, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].t(), w["q.conv"]).view(t, kvh, d)
    k = short_conv(h @ w["k"].t(), w["k.conv"]).view(t, kvh, d)
    v = short_conv(h @ w["v"].t(), w["v.conv"]).view(t, hn, dv)
    head_of = torch.arange(hn) // (hn // kvh)
    q = (unit(q) * d ** -0.5)[:, head_of]
    k = unit(k)[:, head_of]
    beta = torch.sigmoid(h @ w["b"].t())
    a = (h @ w["a1"].t()) @ w["a2"].t() + w["dt_bias"]
    g = torch.exp(-torch.exp(w["A_log"]).view(1, hn, 1) * softplus(a).view(t, hn, d))
    o, _ = delta_recurrence(q, k, v, g, beta)
    gate = torch.sigmoid((h @ w["g1"].t()) @ w["g2"].t()).view(t, hn, dv)
    o = rms(o, eps) * w["norm"] * gate
    return o.reshape(t, hn * dv) @ w["o"].t()


def dense_mlp(h, w):
    return (gelu_tanh(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.t(), max=limit)
    u = torch.clamp(h @ up.t(), min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def table_moe(h, tokens, w, m):
    """Experts picked by a table over token ids, equal weights, plus a sigmoid-gated shared expert."""
    top, limit = m["router"]["top"], m["expert"]["limit"]
    out = torch.zeros_like(h)
    for i, tok in enumerate(tokens):
        for e in w["table"][tok].tolist():
            out[i] += clamped_expert(h[i], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], limit) / top
    if m.get("shared"):
        y = clamped_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"], m["shared"]["limit"])
        out = out + torch.sigmoid(h @ w["shared.sg"].t()) * y
    return out


def layer_order(cfg: dict) -> List[int]:
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    body = list(range(lp["start"], lp["stop"]))
    return list(range(lp["start"])) + body * lp["times"] + list(range(lp["stop"], n))


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: (v if not v.is_floating_point() else v.to(dtype))
            for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, trace: Optional[list] = None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` collects the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    embed = weights["embed"].to(dtype)
    x = embed[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i in layer_order(cfg):
        spec = cfg["layers"][i]
        lw = _sub(weights, f"l{i}.", dtype)
        mixer = {"latent_attention": latent_attention, "channel_delta": channel_delta}[spec["type"]]
        x = x + mixer(norm_offset(x, lw["norm1"], eps), _sub(lw, "mix.", dtype), spec["mixer"], eps)
        if spec.get("mlp"):
            h = norm_offset(x, lw["norm2"], eps)
            mw = _sub(lw, "mlp.", dtype)
            x = x + (dense_mlp(h, mw) if spec["mlp"]["kind"] == "dense" else table_moe(h, tokens, mw, spec["mlp"]))
        if trace is not None:
            trace.append(x.clone())
    return norm_offset(x, weights["final.norm"].to(dtype), eps) @ embed.t()
