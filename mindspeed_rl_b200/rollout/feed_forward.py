"""Feed-forwards of layer-by-layer decoders in the rollout engine.

``forward`` does the feed-forward's work on ``h`` up to what is left to add; ``finish_`` adds it (and, in layers whose
sublayers run in parallel, the mixer's output ``delta``) to the fp32 residual and returns the next norm of the sum, so
that the add (and for expert layers the combine) and the norm are one kernel.  ``norm``: an ``ops.Norm``.  In designs
that norm a sublayer's output, ``finish_post_`` takes the place of ``finish_``; ``post``: an ``ops.PostNorm``.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import ops
from ..models.hybrid_config import ChosenMoESpec, GluSpec, ScoredMoESpec, SoftmaxMoESpec, TableMoESpec
from ..ops import moe as K
from ..ops.gemm import linear_f32, linear_fwd
from .mixers import _pad_cols, _pad_rows


class Glu:
    def __init__(self, spec: GluSpec, w: Dict[str, torch.Tensor], dtype, device):
        self.spec = spec
        self.gate_up = torch.cat([w["gate"], w["up"]]).to(device=device, dtype=dtype).contiguous()
        self.down = w["down"].to(device=device, dtype=dtype).contiguous()

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        s = self.spec
        return linear_fwd(ops.glu_fwd(linear_fwd(h, self.gate_up), s.act, s.limit, s.alpha), self.down)

    def forward(self, h: torch.Tensor, ids: torch.Tensor) -> torch.Tensor:
        return self(h)

    def finish_(self, resid, h, done, norm, delta: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.add_norm_(resid, done, *norm, delta2=delta)

    def finish_post_(self, resid, done, post, after, entry=None) -> torch.Tensor:
        return ops.post_add_(resid, done, post, after, entry)


class GroupedExperts:
    """Stacked expert weights and what every expert layer does once it knows its dispatch plan.  Expert widths are
    padded to the grouped GEMM's reduction tile (zero rows: the activations vanish there)."""

    def __init__(self, spec, w: Dict[str, torch.Tensor], dtype, device):
        self.spec = spec
        f = spec.expert.ff
        fp = (f + 63) // 64 * 64 if dtype == torch.bfloat16 else f
        up, down = [], []
        for e in range(spec.experts):
            up.append(torch.cat([_pad_rows(w[f"e{e}.gate"], fp), _pad_rows(w[f"e{e}.up"], fp)]))
            down.append(_pad_cols(w[f"e{e}.down"], fp))
        self.w1 = torch.stack(up).to(device=device, dtype=dtype).contiguous()        # [E, 2F, W]
        self.w2 = torch.stack(down).to(device=device, dtype=dtype).contiguous()      # [E, W, F]
        self.shared = self.shared_gate = None
        if spec.shared is not None:
            self.shared = Glu(spec.shared, {k: w["shared." + k] for k in ("gate", "up", "down")}, dtype, device)

    def run(self, h: torch.Tensor, plan: K.MoePlan, input_w: Optional[torch.Tensor] = None
            ) -> Tuple[torch.Tensor, K.MoePlan, Optional[torch.Tensor]]:
        s = self.spec
        gu = K.grouped_gemm_nt(K.moe_permute(h, plan, input_w), plan, self.w1)
        act = ops.glu_fwd(gu, s.expert.act, s.expert.limit, s.expert.alpha, plan=plan)
        y = K.grouped_gemm_nt(act, plan, self.w2)
        return y, plan, self.shared(h) if self.shared is not None else None

    def finish_(self, resid, h, done, norm, delta: Optional[torch.Tensor] = None) -> torch.Tensor:
        y, plan, shared = done
        return ops.moe_combine_norm_(resid, y, plan.pos, self.spec.top, self.output_w, h, shared, self.shared_gate, *norm,
                                     delta=delta)


class TableMoE(GroupedExperts):
    """The router is a table from token id to expert ids: the dispatch plan of a step depends on its ids only."""

    def __init__(self, spec: TableMoESpec, w: Dict[str, torch.Tensor], dtype, device):
        super().__init__(spec, w, dtype, device)
        table = w["table"].to(torch.int64)
        if table.shape[1] != spec.top or int(table.min()) < 0 or int(table.max()) >= spec.experts:
            raise ValueError(f"expert table {tuple(table.shape)} does not fit {spec.experts} experts, top {spec.top}")
        self.table = table.to(device)
        self.output_w = 1.0 / spec.top
        if spec.shared is not None:
            self.shared_gate = w["shared.sg"].reshape(-1).to(device=device, dtype=dtype).contiguous()

    def forward(self, h: torch.Tensor, ids: torch.Tensor):
        return self.run(h, K.moe_plan(self.table[ids], self.spec.experts))


class ScoredMoE(GroupedExperts):
    """Router logits are 32-bit; a chosen expert's score scales the rows that go into it."""
    output_w = 1.0

    def __init__(self, spec: ScoredMoESpec, w: Dict[str, torch.Tensor], dtype, device):
        super().__init__(spec, w, dtype, device)
        self.router = w["router"].to(device=device, dtype=dtype).contiguous()

    def forward(self, h: torch.Tensor, ids: torch.Tensor):
        idx, score = K.route_top(linear_f32(h, self.router), self.spec.top)
        return self.run(h, K.moe_plan(idx, self.spec.experts), score)


class WeightedExperts(GroupedExperts):
    """Experts whose outputs are added with a weight each, in designs that norm a sublayer's output."""

    def finish_post_(self, resid, done, post, after, entry=None) -> torch.Tensor:
        y, plan, shared, score = done
        return ops.moe_post_add_(resid, y, plan.pos, score, post, after, shared, entry)


class SoftmaxMoE(WeightedExperts):
    """Router scores are a 32-bit soft-max; what is chosen also depends on a correction per output.  Identity experts have
    no rows in the dispatch plan: the combine takes their input, the residual, where it adds the others."""

    def __init__(self, spec: SoftmaxMoESpec, w: Dict[str, torch.Tensor], dtype, device):
        super().__init__(spec, w, dtype, device)
        self.router = w["router"].to(device=device, dtype=dtype).contiguous()
        self.correction = w["correction"].reshape(-1).to(device=device, dtype=torch.float32).contiguous()
        if self.router.shape[0] != spec.outputs or self.correction.numel() != spec.outputs:
            raise ValueError(f"router {tuple(self.router.shape)} and correction {self.correction.numel()} do not fit {spec.outputs} "
                             "outputs")

    def forward(self, h: torch.Tensor, ids: torch.Tensor):
        idx, score = K.route_softmax_top(linear_f32(h, self.router), self.correction, self.spec.top)
        return *self.run(h, K.moe_plan(idx, self.spec.experts)), score


class ChosenMoE(WeightedExperts):
    """The experts of the largest 32-bit logits, weighted by a soft-max over the logits chosen."""

    def __init__(self, spec: ChosenMoESpec, w: Dict[str, torch.Tensor], dtype, device):
        super().__init__(spec, w, dtype, device)
        self.router = w["router"].to(device=device, dtype=dtype).contiguous()
        if self.router.shape[0] != spec.experts:
            raise ValueError(f"router {tuple(self.router.shape)} does not fit {spec.experts} experts")

    def forward(self, h: torch.Tensor, ids: torch.Tensor):
        idx, score = K.route_top(linear_f32(h, self.router), self.spec.top, chosen_softmax=True)
        return *self.run(h, K.moe_plan(idx, self.spec.experts)), score


FEED_FORWARDS = {GluSpec: Glu, TableMoESpec: TableMoE, ScoredMoESpec: ScoredMoE, SoftmaxMoESpec: SoftmaxMoE,
                 ChosenMoESpec: ChosenMoE}


def build_feed_forward(spec, w: Dict[str, torch.Tensor], dtype, device):
    return None if spec is None else FEED_FORWARDS[type(spec)](spec, w, dtype, device)
