"""Plain, slow restatement of the Lunelorn equations for the tests: one function per mechanism, written over whole
sequences (the recurrences token by token), in double precision by default.  It shares no code with the product path
and reads nothing but a config dictionary and a name -> tensor dictionary.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def turn(x: torch.Tensor, dims: int, base: float, sign: float = 1.0) -> torch.Tensor:
    """``x [T, heads, d]``, row = position: entry i of the first ``dims`` turns with entry i + dims / 2."""
    half, out = dims // 2, x.clone()
    p = torch.arange(x.shape[0], dtype=F64)
    for i in range(half):
        a = sign * p * float(base) ** (-2.0 * i / dims)
        c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def attend(q, k, v, scale: float) -> torch.Tensor:
    """Causal soft-max of ``q [T, H, d]`` over ``k [T, G, d]``, ``v [T, G, dv]``."""
    t, h = q.shape[:2]
    of = torch.arange(h) // (h // k.shape[1])
    out = torch.empty(t, h, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        p = torch.softmax(torch.einsum("hd,jhd->hj", q[i], k[:i + 1, of]) * scale, -1)
        out[i] = torch.einsum("hj,jhd->hd", p, v[:i + 1, of])
    return out


def turned_attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Values are normed and turned by their own position; the output is turned back by the query's."""
    t, hn, g, d, dv, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q = turn((h @ w["q"].t()).view(t, hn, d), rot["dims"], rot["base"])
    k = turn((h @ w["k"].t()).view(t, g, d), rot["dims"], rot["base"])
    v = turn(rms((h @ w["v"].t()).view(t, g, dv), eps), dv, rot["base"])
    o = turn(attend(q, k, v, m["scale"]), dv, rot["base"], -1.0)
    return o.reshape(t, hn * dv) @ w["o"].t()


def min_gru_scan(z: torch.Tensor, cand: torch.Tensor, s: Optional[torch.Tensor] = None) -> torch.Tensor:
    """States ``[T, C]`` of ``S <- (1 - z) S + z cand``."""
    s = torch.zeros_like(z[0]) if s is None else s
    out = torch.empty_like(z)
    for i in range(z.shape[0]):
        s = (1.0 - z[i]) * s + z[i] * cand[i]
        out[i] = s
    return out


def min_gru(h, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    z = torch.sigmoid(h @ w["z"].t() + w["z.b"])
    u = h @ w["x"].t() + w["x.b"]
    s = min_gru_scan(z, torch.where(u >= 0, u + 0.5, torch.sigmoid(u)))
    return (s * silu(h @ w["g"].t())) @ w["o"].t()


def parallel(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    left = turned_attention(h, _sub(w, "left.", h.dtype), m["left"], eps)
    return m["left_scale"] * left + m["right_scale"] * min_gru(h, _sub(w, "right.", h.dtype))


def retention_recurrence(q, k, v, decay, s: Optional[torch.Tensor] = None):
    """``q, k [T, H, d]``, ``v [T, H, dv]``, ``decay [H]`` -> ``o [T, H, dv]``, final state."""
    s = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=k.dtype) if s is None else s.clone()
    o = torch.empty(*k.shape[:2], v.shape[2], dtype=k.dtype)
    for i in range(k.shape[0]):
        s = decay[:, None, None] * s + k[i][:, :, None] * v[i][:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    return o, s


def retention(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[n].t()).view(t, hn, d) for n in "qk")
    o, _ = retention_recurrence(q, k * d ** -0.5, (h @ w["v"].t()).view(t, hn, dv), torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o, eps).reshape(t, hn * dv) * silu(h @ w["g"].t())) @ w["o"].t()


def shifted(h: torch.Tensor) -> torch.Tensor:
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_recurrence(r, k, v, decay, u, s: Optional[torch.Tensor] = None):
    """``r, k, v, decay [T, H, d]``, ``u [H, d]`` -> ``o [T, H, d]``, final state."""
    s = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=k.dtype) if s is None else s.clone()
    o = torch.empty_like(v)
    for i in range(k.shape[0]):
        kv = k[i][:, :, None] * v[i][:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s + u[:, :, None] * kv, r[i])
        s = decay[i][:, :, None] * s + kv
    return o, s


def wkv(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, d = h.shape[0], m["heads"], m["dim"]
    mix = {n: h + (shifted(h) - h) * w["mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[n].t()).view(t, hn, d) for n in "rkv")
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].t()) @ w["w2"].t() + w["w0"])).view(t, hn, d)
    o, _ = wkv_recurrence(r, k, v, decay, w["u"])
    return (rms(o, eps).reshape(t, hn * d) * w["norm"] * silu(mix["g"] @ w["g"].t())) @ w["o"].t()


def choose(z: torch.Tensor, top: int) -> List[int]:
    """Experts of the largest logits of one token, best first (the lower expert among equals)."""
    c = z.tolist()
    return sorted(range(len(c)), key=lambda e: (-c[e], e))[:top]


def expert(x, gate, up, down):
    return (silu(x @ gate.t()) * (x @ up.t())) @ down.t()


def mixture(h, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    z = h @ w["router"].t()
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = choose(z[t], m["router"]["top"])
        for e, p in zip(chosen, torch.softmax(z[t, chosen], -1)):
            out[t] += p * expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def token_side(x, e: torch.Tensor, w: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    """What the layer's token rows ``e [T, dim]`` add to ``x``."""
    return rms((gelu_tanh(x @ w["gate"].t()) * e) @ w["proj"].t(), eps) * w["norm"]


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"retention": retention, "parallel": parallel, "wkv": wkv}


def run_order(cfg: dict):
    """(layer, pass number at which a pass starts here or None) of every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    passes = [(i, p if i == a else None) for p in range(lp["times"]) for i in range(a, b)]
    return [*((i, None) for i in range(a)), *passes, *((i, None) for i in range(b, n))]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, trace: Optional[list] = None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` collects the residual stream after every layer run."""
    eps, dim = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.tensor(tokens)
    top = {k: weights[k].to(dtype) for k in ("embed", "embed.norm", "side.embed", "final.norm", "head")}
    e0 = rms(top["embed"][ids], eps) * top["embed.norm"]
    x = e0.clone()
    for i, p in run_order(cfg):
        if p is not None:
            x = x + (e0 if p else 0.0) + weights["loop.step"][p].to(dtype)
        spec, lw = cfg["layers"][i], _sub(weights, f"l{i}.", dtype)
        y = MIXERS[spec["type"]](rms(x, eps) * lw["norm1"], _sub(lw, "mix.", dtype), spec["mixer"], eps)
        x = x + rms(y, eps) * lw["norm1b"]
        if spec.get("mlp"):
            y = mixture(rms(x, eps) * lw["norm2"], _sub(lw, "mlp.", dtype), spec["mlp"])
            x = x + rms(y, eps) * lw["norm2b"]
        x = x + token_side(x, top["side.embed"][ids, i * dim:(i + 1) * dim], _sub(lw, "side.", dtype), eps)
        if trace is not None:
            trace.append(x.clone())
    cap = cfg["logit_softcap"]
    return cap * torch.tanh((rms(x, eps) * top["final.norm"]) @ top["head"].t() / cap)
