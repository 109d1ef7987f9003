"""Plain, slow restatement of the Sunatar equations for the tests: one function per mechanism, written over whole
sequences (the matrix memory token by token), in double precision by default.  It shares no code with the product
path and reads nothing but a config dictionary and a name -> tensor dictionary.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def logsigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def frequencies(rot: dict) -> List[float]:
    """Angular frequency of every pair, rescaled by wavelength when ``rot['scaling']`` is given."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - mix) * f / s["factor"] + mix * f
        out.append(f)
    return out


def rotate_halves(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """``x [T, heads, d]``, row = position: entry i of the first ``dims`` turns with entry i + dims / 2."""
    out, half = x.clone(), rot["dims"] // 2
    pos = torch.arange(x.shape[0]).to(x.dtype)
    for i, f in enumerate(frequencies(rot)):
        c, s = torch.cos(pos * f)[:, None], torch.sin(pos * f)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def window_softmax(q, k, v, scale: float, window: Optional[int]) -> torch.Tensor:
    """``q [T, H, d]`` over ``k [T, G, d]``, ``v [T, G, dv]``: token i sees the last ``window`` tokens up to itself."""
    t, h = q.shape[:2]
    of = torch.arange(h) // (h // k.shape[1])
    out = torch.empty(t, h, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        lo = 0 if window is None else max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1, of]) * scale
        out[i] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[lo:i + 1, of])
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float, v_first: Optional[torch.Tensor] = None):
    """Output and the layer's own values (before mixing)."""
    t, hn, g, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ w["q"].t() + w["q.b"], eps) * w["q.norm"]
    k = rms(h @ w["k"].t() + w["k.b"], eps) * w["k.norm"]
    own = h @ w["v"].t() + w["v.b"]
    v = own if v_first is None else mix_values(own, v_first, w["vmix"])
    q, k = rotate_halves(q.view(t, hn, d), m["rot"]), rotate_halves(k.view(t, g, d), m["rot"])
    out = window_softmax(q, k, v.view(t, g, dv), m["scale"], (m.get("mask") or {}).get("size"))
    return out.reshape(t, hn * dv) @ w["o"].t(), own


def matrix_memory(q, k, v, i, f):
    """``q, k [T, H, d]`` (q scaled), ``v [T, H, dv]``, log gates ``i, f [T, H]`` -> ``o [T, H, dv]``."""
    t, hn, d = k.shape
    s = torch.zeros(hn, d, v.shape[-1], dtype=k.dtype)
    n, m = torch.zeros(hn, d, dtype=k.dtype), torch.zeros(hn, dtype=k.dtype)
    o = torch.empty(t, hn, v.shape[-1], dtype=k.dtype)
    for x in range(t):
        top = torch.maximum(f[x] + m, i[x])
        keep, take = torch.exp(f[x] + m - top), torch.exp(i[x] - top)
        s = keep[:, None, None] * s + take[:, None, None] * k[x][:, :, None] * v[x][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[x]
        m = top
        den = torch.maximum((n * q[x]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[x] = torch.einsum("hdv,hd->hv", s, q[x]) / den[:, None]
    return o


def gates(h, w, cap: float):
    i = cap * torch.tanh((h @ w["i"].t() + w["i.b"]) / cap)
    f = logsigmoid(cap * torch.tanh((h @ w["f"].t() + w["f.b"]) / cap))
    return i, f


def mlstm(h, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, hn, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].t()).view(t, hn, d) * d ** -0.5
    k, v = (h @ w["k"].t()).view(t, hn, d), (h @ w["v"].t()).view(t, hn, dv)
    o = matrix_memory(q, k, v, *gates(h, w, m["gate_cap"]))
    y = rms(o, eps).reshape(t, hn * dv) * w["norm"] * torch.sigmoid(h @ w["g"].t())
    return y @ w["o"].t()


def glu(x, gate, up, down):
    return (silu(x @ gate.t()) * (x @ up.t())) @ down.t()


def routed_experts(h, w, m: dict) -> torch.Tensor:
    """Experts of the largest sigmoid scores; a score scales its expert's input; plus the shared expert."""
    s = torch.sigmoid(h @ w["router"].t())
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(s[t], m["router"]["top"]).indices.tolist():
            out[t] += glu(s[t, e] * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if m.get("shared"):
        out = out + glu(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=F64, trace: Optional[list] = None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = weights["embed"].to(dtype)[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    v_first = None
    for i, spec in enumerate(cfg["layers"]):
        lw = _sub(weights, f"l{i}.", dtype)
        h = layer_norm(x, lw["norm1"], eps)
        m, mw = spec["mixer"], _sub(lw, "mix.", dtype)
        if spec["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, mw, m, eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        else:
            y = mlstm(h, mw, m, eps)
        if spec.get("mlp"):
            y = y + routed_experts(h, _sub(lw, "mlp.", dtype), spec["mlp"])
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return layer_norm(x, weights["final.norm"].to(dtype), eps) @ weights["head"].to(dtype).t()
