"""What soft-max attention may do to its scores and its heads beyond the plain form.

:class:`ScoreForm`: ``softcap`` c > 0 turns a scaled score s into ``c tanh(s / c)``; ``gate [T, heads]`` (logits in the
activation type, rows may be strided) multiplies a head's output by ``sigmoid(gate)``; ``sink [heads]`` (fp32) adds
``exp(sink)`` to a head's soft-max sum.  The attention kernels take all three in their loops and epilogues.
"""
from __future__ import annotations

from typing import NamedTuple, Optional

import torch

from ._lib import c_float, c_ll, ptr


class ScoreForm(NamedTuple):
    softcap: float = 0.0
    gate: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None

    def args(self):
        """``softcap, gate, gate row stride, sink`` of the kernels."""
        return (c_float(self.softcap), ptr(self.gate), c_ll(0 if self.gate is None else self.gate.stride(0)), ptr(self.sink))

    # ---- PyTorch formulation -----------------------------------------------------------------------
    def weights(self, scores: torch.Tensor, hide: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Soft-max weights of scaled scores ``[heads, ..., keys]``."""
        if self.softcap:
            scores = self.softcap * torch.tanh(scores / self.softcap)
        if hide is not None:
            scores = scores.masked_fill(hide, float("-inf"))
        if self.sink is None:
            return torch.softmax(scores, dim=-1)
        sink = self.sink.view(-1, *([1] * (scores.dim() - 1))).expand(*scores.shape[:-1], 1)
        return torch.softmax(torch.cat([scores, sink], dim=-1), dim=-1)[..., :-1]

    def gated(self, out: torch.Tensor) -> torch.Tensor:
        """``out [T, heads, n]`` (fp32) times the heads' gates."""
        return out if self.gate is None else out * torch.sigmoid(self.gate.float())[..., None]


PLAIN = ScoreForm()
