"""Ring KV cache of sliding-window layers, addressed by position.

Like ``SlidingWindowKVCache`` a token at absolute position ``p`` lives in slot ``p % slots``, but the
positions of the slots follow from the number of stored tokens alone, so no position tensor is kept and
the kernels (``ops/window_ops.py``) append in place while they read: the slot being overwritten holds the
key that has just left the window.  Keys and values may have different head sizes.
"""

from __future__ import annotations

from typing import NamedTuple

import torch

from axlearn_b200.common.config import REQUIRED, Required, config_class
from axlearn_b200.common.kv_cache.base_kv_cache import BaseKVCache
from axlearn_b200.common.module import nowrap


class RingKVCache(BaseKVCache):
    @config_class
    class Config(BaseKVCache.Config):
        # Positions a query sees, itself included.
        window: Required[int] = REQUIRED

    class Shape(NamedTuple):
        batch_size: int
        kv_len: int
        num_kv_heads: int
        per_head_dim: int
        value_dim: int

    @nowrap
    def init_states(self, shape, *, dtype: torch.dtype, device=None) -> dict:
        dt = self._cache_dtype(dtype)
        slots = max(1, min(self._config.window, shape.kv_len))
        lead = (shape.batch_size, slots, shape.num_kv_heads)
        return {
            "key": torch.zeros(lead + (shape.per_head_dim,), dtype=dt, device=device),
            "value": torch.zeros(lead + (shape.value_dim,), dtype=dt, device=device),
        }
