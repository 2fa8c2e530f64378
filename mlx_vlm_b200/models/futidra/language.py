"""Futidra language model: the call surface of the layer-assembled decoders (`step`, `__call__`, `make_cache`,
`make_cache_row`, `make_pool`, `fused_greedy_decode_n`, `prefill_rows`: models/buzopel/language.py) over a
`StatePool`: a request's slot holds the rows of every caching layer — [keys | values] of an 'attention' layer, the latent
of a 'latent_attention' layer that has its own; the layers that borrow one hold shared views of it — and one span of fp32
state (convolution history + matrix states) per 'channel_delta' layer."""
from __future__ import annotations

from typing import List

import torch

from ..buzopel.language import LanguageModel as _LayeredLanguageModel
from ..cache import RunCache, StatePool


class LanguageModel(_LayeredLanguageModel):
    def __init__(self, args, core, engine_getter):
        super().__init__(args, core, engine_getter)
        self.model_type = "futidra"

    def make_pool(self, rows: int = 1, capacity: int = 0) -> StatePool:
        eng = self._engine()
        with torch.cuda.stream(eng.stream):
            return StatePool(self.core.n_cache_layers, self.core.row_dim, self.core.state_floats, eng.device, batch=rows,
                             capacity=capacity, dtype=eng.ops.cache_dtype)

    def make_cache_row(self, pool: StatePool, row: int) -> List[RunCache]:
        return [RunCache(pool, row, kv_layer=L.mixer.cache_index if L.kv_dim else None, kv_dim=L.kv_dim,
                         state_off=L.mixer.state_off, state_len=L.state_floats, shared=not getattr(L.mixer, "own_kv", True))
                for L in self.core.layers]

    def make_cache(self) -> List[RunCache]:
        return self.make_cache_row(self.make_pool(1), 0)
