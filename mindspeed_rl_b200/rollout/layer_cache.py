"""Carried state of decoders whose layers differ: paged latent rows and recurrent state slots.

``HybridCache`` holds one entry per layer *run* (a layer that is run several times in a row has an entry per
pass): latent-attention runs own paged rows ``[num_blocks, block_size, CP]`` addressed through the block manager's
tables, recurrent runs own ``ring [slots, taps, channels]`` and ``state [slots, heads, dim, vdim]`` (fp32)
addressed by a state slot per sequence.  ``StateSlots`` hands the slots out; the scheduler takes one when it
admits or forks a sequence and returns it when the sequence ends or is preempted.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..models.hybrid_config import HybridConfig
from ..ops.latent import pad16


class OutOfSlots(RuntimeError):
    pass


class StateSlots:
    """Free list of recurrent-state slots (lowest free slot first, so that a small batch stays compact)."""

    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self._free = list(range(num_slots - 1, -1, -1))
        self._used: set = set()

    @property
    def num_free(self) -> int:
        return len(self._free)

    def allocate(self) -> int:
        if not self._free:
            raise OutOfSlots()
        slot = self._free.pop()
        self._used.add(slot)
        return slot

    def free(self, slot: int) -> None:
        if slot not in self._used:
            raise KeyError(slot)
        self._used.discard(slot)
        self._free.append(slot)


def latent_row_width(spec) -> int:
    return pad16(spec.kv_rank) + pad16(spec.rot_dim)


def delta_channels(spec) -> int:
    return 2 * spec.kv_heads * spec.dim + spec.heads * spec.vdim


class HybridCache:
    def __init__(self, cfg: HybridConfig, num_blocks: int, block_size: int, num_slots: int, device):
        self.num_blocks, self.block_size, self.num_slots = num_blocks, block_size, num_slots
        dev = torch.device(device)
        # every row and slot is written before it is read (a sequence's first token ignores what its slot holds),
        # so nothing is cleared on the GPU; the CPU path multiplies by masks and wants finite values
        alloc = torch.empty if dev.type == "cuda" else torch.zeros
        self.latent: List[Optional[torch.Tensor]] = []
        self.ring: List[Optional[torch.Tensor]] = []
        self.state: List[Optional[torch.Tensor]] = []
        for li in cfg.run_order:
            m = cfg.layers[li].mixer
            if m.recurrent:
                self.latent.append(None)
                self.ring.append(alloc(num_slots, m.conv, delta_channels(m), dtype=cfg.params_dtype, device=dev))
                self.state.append(alloc(num_slots, m.heads, m.dim, m.vdim, dtype=torch.float32, device=dev))
            else:
                self.latent.append(alloc(num_blocks, block_size, latent_row_width(m), dtype=cfg.params_dtype, device=dev))
                self.ring.append(None)
                self.state.append(None)

    @staticmethod
    def bytes_per_block(cfg: HybridConfig, block_size: int) -> int:
        size = torch.empty(0, dtype=cfg.params_dtype).element_size()
        return sum(block_size * latent_row_width(cfg.layers[li].mixer) * size for li in cfg.run_order
                   if not cfg.layers[li].mixer.recurrent)

    @staticmethod
    def bytes_per_slot(cfg: HybridConfig) -> int:
        size = torch.empty(0, dtype=cfg.params_dtype).element_size()
        total = 0
        for li in cfg.run_order:
            m = cfg.layers[li].mixer
            if m.recurrent:
                total += m.conv * delta_channels(m) * size + m.heads * m.dim * m.vdim * 4
        return total

    def copy_block(self, src: int, dst: int) -> None:
        for c in self.latent:
            if c is not None:
                c[dst].copy_(c[src])

    def copy_slot(self, src: int, dst: int) -> None:
        for pair in (self.ring, self.state):
            for c in pair:
                if c is not None:
                    c[dst].copy_(c[src])
