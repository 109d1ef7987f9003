"""Feed-forwards of layer-by-layer decoders in the rollout engine.

``forward_norm_`` adds the feed-forward of ``h`` to the fp32 residual and returns the next norm of the sum, so
that the add (and for expert layers the combine) and the norm are one kernel.
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..models.hybrid_config import GluSpec, TableMoESpec
from ..ops import moe as K
from ..ops.gemm import linear_fwd
from .mixers import _pad_cols, _pad_rows


class Glu:
    def __init__(self, spec: GluSpec, w: Dict[str, torch.Tensor], dtype, device):
        self.spec = spec
        self.gate_up = torch.cat([w["gate"], w["up"]]).to(device=device, dtype=dtype).contiguous()
        self.down = w["down"].to(device=device, dtype=dtype).contiguous()

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        s = self.spec
        return linear_fwd(ops.glu_fwd(linear_fwd(h, self.gate_up), s.act, s.limit, s.alpha), self.down)

    def forward_norm_(self, resid, h, ids, norm_w, eps, offset) -> torch.Tensor:
        return ops.add_norm_(resid, self.forward(h), norm_w, eps, offset)


class TableMoE:
    """The router is a table from token id to expert ids: the dispatch plan of a step depends on its ids only.
    Expert widths are padded to the grouped GEMM's reduction tile (zero rows: both activations vanish there)."""

    def __init__(self, spec: TableMoESpec, w: Dict[str, torch.Tensor], dtype, device):
        self.spec = spec
        f = spec.expert.ff
        fp = (f + 63) // 64 * 64 if dtype == torch.bfloat16 else f
        up, down = [], []
        for e in range(spec.experts):
            up.append(torch.cat([_pad_rows(w[f"e{e}.gate"], fp), _pad_rows(w[f"e{e}.up"], fp)]))
            down.append(_pad_cols(w[f"e{e}.down"], fp))
        self.w1 = torch.stack(up).to(device=device, dtype=dtype).contiguous()        # [E, 2F, W]
        self.w2 = torch.stack(down).to(device=device, dtype=dtype).contiguous()      # [E, W, F]
        table = w["table"].to(torch.int64)
        if table.shape[1] != spec.top or int(table.min()) < 0 or int(table.max()) >= spec.experts:
            raise ValueError(f"expert table {tuple(table.shape)} does not fit {spec.experts} experts, top {spec.top}")
        self.table = table.to(device)
        self.shared = self.shared_gate = None
        if spec.shared is not None:
            self.shared = Glu(spec.shared, {k: w["shared." + k] for k in ("gate", "up", "down")}, dtype, device)
            self.shared_gate = w["shared.sg"].reshape(-1).to(device=device, dtype=dtype).contiguous()

    def forward_norm_(self, resid, h, ids, norm_w, eps, offset) -> torch.Tensor:
        s = self.spec
        plan = K.moe_plan(self.table[ids], s.experts)
        gu = K.grouped_gemm_nt(K.moe_permute(h, plan), plan, self.w1)
        act = ops.glu_fwd(gu, s.expert.act, s.expert.limit, s.expert.alpha, plan=plan)
        y = K.grouped_gemm_nt(act, plan, self.w2)
        shared = self.shared.forward(h) if self.shared is not None else None
        return ops.moe_combine_norm_(resid, y, plan.pos, s.top, 1.0 / s.top, h, shared, self.shared_gate, norm_w, eps,
                                     offset)


def build_feed_forward(spec, w: Dict[str, torch.Tensor], dtype, device):
    if spec is None:
        return None
    return (TableMoE if isinstance(spec, TableMoESpec) else Glu)(spec, w, dtype, device)
