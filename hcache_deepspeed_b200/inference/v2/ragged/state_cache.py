"""Per-sequence recurrent state beside the paged KV cache.

A recurrent layer keeps, for every live sequence, one fp32 matrix per head and the latest inputs of its short convolution.
Their size does not grow with the sequence, so they need no pages: a sequence owns ONE slot index, valid in every layer,
from its admission until it is flushed. Slots are handed out without being cleared. What a slot holds belongs to the
sequence only once its first token has run: the kernels take the state of a sequence at position 0 as zero, and read
convolution inputs of non-negative positions only.

Layouts per layer: ``ssm [slots, heads, vdim, state]`` fp32 (the state index innermost: one warp reads one row of it) and
``conv [slots, taps, conv_dim]`` fp32, the input of position p in ring entry ``p % taps``. The ring has one entry more than
a convolution looks back, so a single-token step can store the new input while other thread blocks still read the old ones.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ....utils.logging import inference_logger
from .blocked_allocator import BlockedAllocator
from .manager_configs import RecurrentLayerConfig


class RecurrentStateCache:

    def __init__(self, layers: Sequence[Optional[RecurrentLayerConfig]], max_slots: int, device: torch.device,
                 requested: Optional[int] = None) -> None:
        per_slot = sum(4 * (l.heads * l.vdim * l.state + l.taps * l.conv_dim) for l in layers if l is not None)
        n = requested
        if n is None:
            n = max_slots
            if device.type == "cuda":
                free, _ = torch.cuda.mem_get_info(device)
                n = max(1, min(n, free // 8 // max(1, per_slot)))
        self._allocator = BlockedAllocator(int(n))
        inference_logger().info(f"Allocating recurrent state: {n} slots x {per_slot} B = {n * per_slot / 2**30:.2f} GiB")
        self._ssm: List[Optional[torch.Tensor]] = []
        self._conv: List[Optional[torch.Tensor]] = []
        for l in layers:
            self._ssm.append(None if l is None else torch.zeros((n, l.heads, l.vdim, l.state), dtype=torch.float32, device=device))
            self._conv.append(None if l is None else torch.zeros((n, l.taps, l.conv_dim), dtype=torch.float32, device=device))

    @property
    def num_slots(self) -> int:
        return self._allocator.total_blocks

    @property
    def free_slots(self) -> int:
        return self._allocator.free_blocks

    def allocate(self) -> int:
        return int(self._allocator.allocate(1)[0])

    def free(self, slot: int) -> None:
        self._allocator.free(slot)

    def ssm(self, layer: int) -> torch.Tensor:
        return self._ssm[layer]

    def conv(self, layer: int) -> torch.Tensor:
        return self._conv[layer]
