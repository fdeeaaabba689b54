"""Configuration of the ragged state manager and the paged KV cache.

Field names, defaults and validation follow the reference so existing configs load unchanged
(``deepspeed/inference/v2/ragged/manager_configs.py:15-181``). ``offload`` is honoured here (the
reference accepts it but its KV offload raises NotImplementedError, ``ragged/kv_cache.py:166-184``).
"""
from __future__ import annotations

from enum import Enum
from typing import List, Optional, Tuple

from pydantic import NonNegativeInt, PositiveInt, model_validator

from ....config import DeepSpeedConfigModel, DtypeEnum


class KVCacheType(Enum):
    DENSE = "dense"
    """Every token's K/V is kept (the only type implemented, as in the reference)."""
    LOCAL = "local"
    """Sliding-window cache (declared for config compatibility)."""


class KVCacheConfig(DeepSpeedConfigModel):
    type: KVCacheType = KVCacheType.DENSE
    block_size: int = 128
    """Tokens per KV block."""
    num_allocation_groups: PositiveInt = 1
    cache_shape: Tuple[PositiveInt, PositiveInt, PositiveInt]
    """(num_layers, num_kv_heads on this rank, head_dim)."""
    cache_dtype: DtypeEnum = DtypeEnum.fp16
    max_blocks_per_allocation_group: PositiveInt = 64
    """Upper bound of blocks one sequence may own (= ceil(max_context / block_size))."""
    layer_shapes: Optional[List[Optional[Tuple[PositiveInt, PositiveInt, PositiveInt]]]] = None
    """(planes, kv_heads, head_dim) of every layer when they differ; ``cache_shape`` with two planes, K and V, otherwise. One plane:
    keys and values are read from the same rows. None: a layer with nothing of its own in the pages."""


class RecurrentLayerConfig(DeepSpeedConfigModel):
    """Per-sequence state of one recurrent layer: a ``heads`` x ``vdim`` x ``state`` matrix stack and the latest ``taps``
    inputs of ``conv_dim`` convolution channels (0: no convolution)."""
    heads: PositiveInt
    vdim: PositiveInt
    state: PositiveInt
    conv_dim: NonNegativeInt
    taps: NonNegativeInt


class AllocationMode(Enum):
    RESERVE = "reserve"
    """Use all free device memory except ``size`` bytes."""
    ALLOCATE = "allocate"
    """Use exactly ``size`` bytes."""
    TOKENS = "tokens"
    """Hold ``size`` tokens (rounded up to whole blocks)."""


class MemoryConfig(DeepSpeedConfigModel):
    mode: AllocationMode = AllocationMode.RESERVE
    size: PositiveInt = 1_000_000_000


class DSStateManagerConfig(DeepSpeedConfigModel):
    max_tracked_sequences: PositiveInt = 2048
    """Sequences whose KV state may be resident at once."""
    max_ragged_batch_size: PositiveInt = 768
    """Tokens per forward."""
    max_ragged_sequence_count: PositiveInt = 512
    """Sequences per forward."""
    max_context: PositiveInt = 8192
    """Longest sequence (prompt + generation) the engine will hold."""
    max_state_slots: Optional[PositiveInt] = None
    """Models with recurrent layers: sequences whose recurrent state may be resident (default: every tracked sequence, as
    far as an eighth of the free device memory holds them)."""
    memory_config: MemoryConfig = MemoryConfig()
    offload: bool = False
    """Allow whole-sequence KV offload to pinned host memory (``DSStateManager.offload_sequence``)."""

    @model_validator(mode="after")
    def _max_ragged_sequence_count_validator(self):
        if self.max_ragged_sequence_count > self.max_tracked_sequences:
            raise ValueError("max_ragged_sequence_count must be less than max_tracked_sequences")
        if self.max_ragged_sequence_count > self.max_ragged_batch_size:
            raise ValueError("max_ragged_sequence_count must be less than max_ragged_batch_size")
        return self
