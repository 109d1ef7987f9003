"""Carried state of decoders whose layers differ: paged rows (latents, keys and values) and recurrent state slots.

``HybridCache`` holds one entry per layer *run* (a layer that is run several times in a row has an entry per
pass): attention runs own paged rows ``[num_blocks, block_size, ...]`` addressed through the block manager's
tables, recurrent runs own state tensors ``[slots, ...]`` addressed by a state slot per sequence.  ``StateSlots`` hands the slots out; the scheduler takes one when it
admits or forks a sequence and returns it when the sequence ends or is preempted.
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch

from ..models.hybrid_config import HybridConfig


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


class HybridCache:
    """``rows[run]``: paged memory by name, ``[num_blocks, block_size, *row]``; ``slots[run]``: state by name,
    ``[num_slots, *shape]``.  What a layer has is what its mixer spec asks for."""

    def __init__(self, cfg: HybridConfig, num_blocks: int, block_size: int, num_slots: int, device):
        self.num_blocks, self.block_size, self.num_slots = num_blocks, block_size, num_slots
        dev = torch.device(device)
        # every row and slot is written before it is read (a sequence's first token ignores what its slot holds),
        # so nothing is cleared on the GPU; the CPU path multiplies by masks and wants finite values
        alloc = torch.empty if dev.type == "cuda" else torch.zeros
        self.rows: List[Dict[str, torch.Tensor]] = []
        self.slots: List[Dict[str, torch.Tensor]] = []
        dt = cfg.params_dtype
        for li in cfg.run_order:
            m = cfg.layers[li].mixer
            self.rows.append({n: alloc(num_blocks, block_size, *shape, dtype=dt, device=dev)
                              for n, shape in m.paged_rows(dt).items()})
            self.slots.append({n: alloc(num_slots, *shape, dtype=t, device=dev) for n, (shape, t) in m.slot_state(dt).items()})

    @staticmethod
    def bytes_per_block(cfg: HybridConfig, block_size: int) -> int:
        dt = cfg.params_dtype
        return sum(block_size * math.prod(shape) * dt.itemsize for li in cfg.run_order
                   for shape in cfg.layers[li].mixer.paged_rows(dt).values())

    @staticmethod
    def bytes_per_slot(cfg: HybridConfig) -> int:
        return sum(math.prod(shape) * t.itemsize for li in cfg.run_order
                   for shape, t in cfg.layers[li].mixer.slot_state(cfg.params_dtype).values())

    def copy_block(self, src: int, dst: int) -> None:
        for rows in self.rows:
            for c in rows.values():
                c[dst].copy_(c[src])

    def copy_slot(self, src: int, dst: int) -> None:
        for slots in self.slots:
            for c in slots.values():
                c[dst].copy_(c[src])
