"""Plain, slow restatement of the Gapevik equations for the tests: one function per mechanism, written over whole
sequences (the recurrence token by token), in double precision by default.  It shares no code with the product path
and reads nothing but a config dictionary and a name -> tensor dictionary.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def short_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal per-channel convolution ``u [T, C]``, ``w [C, taps]`` (last tap = current token)."""
    t, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < t:
            y[back:] += u[:t - back] * w[:, j]
    return y


def _angles(n: int, rot: dict) -> torch.Tensor:
    f = [float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    return torch.arange(n).to(F64)[:, None] * torch.tensor(f, dtype=F64)


def rotate_pairs(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """``x [T, heads, d]``, row = position: neighbours (2i, 2i + 1) of the first ``dims`` entries turn together."""
    a = _angles(x.shape[0], rot)
    out = x.clone()
    for i in range(rot["dims"] // 2):
        c, s = a[:, i].cos().to(x.dtype)[:, None], a[:, i].sin().to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def rotate_halves(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """The same with entry i turning with entry i + dims / 2."""
    a, half = _angles(x.shape[0], rot), rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        c, s = a[:, i].cos().to(x.dtype)[:, None], a[:, i].sin().to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def chunk_start(i: int, size: Optional[int]) -> int:
    return 0 if not size else i // size * size


def window_start(i: int, size: Optional[int]) -> int:
    return 0 if not size else max(0, i - size + 1)


def capped(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if not cap else cap * torch.tanh(s / cap)


def weights_of_scores(s: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Soft-max over the last axis of ``s [H, n]``; ``sink [H]`` adds exp(sink) to the denominator."""
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, sink[:, None]], -1), -1)[:, :-1]


def attend(q, k, v, scale: float, first, cap: Optional[float] = None, sink: Optional[torch.Tensor] = None):
    """``q [T, H, d]`` over ``k [T, G, d]``, ``v [T, G, dv]``: token i sees the tokens from ``first(i)`` to itself."""
    t, h = q.shape[:2]
    of = torch.arange(h) // (h // k.shape[1])
    out = torch.empty(t, h, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        lo = first(i)
        s = capped(torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1, of]) * scale, cap)
        out[i] = torch.einsum("hj,jhd->hd", weights_of_scores(s, sink), v[lo:i + 1, of])
    return out


def head_gate(o: torch.Tensor, h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return o * torch.sigmoid(h @ w.t())[..., None]


def attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, g, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].t(), w["q.conv"]).view(t, hn, d)
    k = short_conv(h @ w["k"].t(), w["k.conv"]).view(t, g, d)
    v = short_conv(h @ w["v"].t(), w["v.conv"]).view(t, g, dv)
    q = rotate_pairs(rms(q, eps) * w["q.norm"], m["rot"])
    k = rotate_pairs(rms(k, eps) * w["k.norm"], m["rot"])
    size = (m.get("mask") or {}).get("size")
    o = attend(q, k, v, m["scale"], lambda i: chunk_start(i, size), m.get("softcap"))
    return head_gate(o, h, w["g"]).reshape(t, hn * dv) @ w["o"].t()


def latent_attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = ((rms(h @ w["dq"].t(), eps) * w["dq.norm"]) @ w["uq"].t()).view(t, hn, d + r)
    ckr = h @ w["dkv"].t()
    c = rms(ckr[:, :rank], eps) * w["dkv.norm"]
    kr = rotate_halves(ckr[:, None, rank:], m["rot"]).expand(t, hn, r)
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], m["rot"])], -1)
    k = torch.cat([(c @ w["uk"].t()).view(t, hn, d), kr], -1)
    size = (m.get("mask") or {}).get("size")
    o = attend(q, k, (c @ w["uv"].t()).view(t, hn, dv), m["scale"], lambda i: window_start(i, size), None, w["sink"])
    return head_gate(o, h, w["g"]).reshape(t, hn * dv) @ w["o"].t()


def delta_recurrence(q, k, v, g, beta, s: Optional[torch.Tensor] = None):
    """``q, k [T, H, d]``, ``v [T, H, dv]``, ``g, beta [T, H]`` -> ``o [T, H, dv]``, final state."""
    t, hn, d = k.shape
    s = torch.zeros(hn, d, v.shape[-1], dtype=k.dtype) if s is None else s.clone()
    o = torch.empty(t, hn, v.shape[-1], dtype=k.dtype)
    for i in range(t):
        s = s * g[i][:, None, None]
        u = beta[i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", s, k[i]))
        s = s + k[i][:, :, None] * u[:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    return o, s


def delta(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, kvh, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    of = torch.arange(hn) // (hn // kvh)
    q = unit(silu(short_conv(h @ w["q"].t(), w["q.conv"])).view(t, kvh, d))[:, of] * d ** -0.5
    k = unit(silu(short_conv(h @ w["k"].t(), w["k.conv"])).view(t, kvh, d))[:, of]
    v = silu(short_conv(h @ w["v"].t(), w["v.conv"])).view(t, hn, dv)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].t() + w["dt_bias"]))
    o, _ = delta_recurrence(q, k, v, g, torch.sigmoid(h @ w["b"].t()))
    o = rms(o, eps) * w["norm"] * silu(h @ w["g"].t()).view(t, hn, dv)
    return o.reshape(t, hn * dv) @ w["o"].t()


def glu(x, gate, up, down):
    return (silu(x @ gate.t()) * (x @ up.t())) @ down.t()


def choose(s: torch.Tensor, correction: torch.Tensor, top: int) -> List[int]:
    """Experts of the largest corrected scores of one token, best first (the lower expert among equals)."""
    c = (s + correction).tolist()
    return sorted(range(len(c)), key=lambda e: (-c[e], e))[:top]


def mixture(h, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    r = m["router"]
    s = torch.softmax(h @ w["router"].t(), -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t], w["correction"], r["top"]):
            y = h[t] if e >= r["experts"] else glu(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
            out[t] += s[t, e] * y
    return out


def owner(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"attention": attention, "latent_attention": latent_attention, "delta": delta}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, trace: Optional[list] = None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` collects the residual stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    embed = weights["embed"].to(dtype)
    x = embed[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, spec in enumerate(cfg["layers"]):
        lw = _sub(weights, f"l{owner(cfg, i)}.", dtype)
        y = MIXERS[spec["type"]](x, _sub(lw, "mix.", dtype), spec["mixer"], eps)
        x = x + mult * rms(y, eps) * lw["norm1"]
        if spec.get("mlp"):
            y = mixture(x, _sub(lw, "mlp.", dtype), spec["mlp"])
            x = x + mult * rms(y, eps) * lw["norm2"]
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * weights["final.norm"].to(dtype)) @ embed.t()
