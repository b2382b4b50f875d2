"""Attention as the difference of two maps over the same values (differential attention).

Every head has two queries and every key/value head two keys, laid out head by head as [map 1 | map 2] of ``head_dim`` columns
each; map m's scores are q_m . k_m * scale under a causal softmax of its own, and both maps weigh the same values
(``value_dim`` columns).  With the maps' outputs a1 and a2 and one number lambda for the layer,
lambda = exp(sum(lq1 * lk1)) - exp(sum(lq2 * lk2)) + diff (four vectors [head_dim], a constant ``diff``), a head's output is
a1 - lambda a2, divided by its root mean square over the head's columns (eps inside the root, no weight), times 1 - diff;
then the output projection over the heads side by side.  No position encoding, no biases.

How it runs: a cached key row is both keys side by side (2 head_dim columns), as the projection leaves them, and the two
queries of a head are rows that are zero outside their own map's columns, so that q_m . [k_1, k_2] = q_m . k_m.  The layer is
then ordinary grouped-query attention of 2 * heads query heads over ``kv_heads`` key/value heads on the framework's
kernels: keys and values are cached and read once for both maps, at the price of multiplying the zero half of each query (a
row is max(2 head_dim, value_dim) columns; where value_dim = 2 head_dim nothing is padding and the products are 4/3 of what
the two maps need).  One kernel takes the difference, the norm and the factor.

A layer with ``reads_only`` has no k and v projections: it attends with its own queries over the keys and values that an
earlier layer's call left in its cache.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import KVCacheNeed, Mixer, Runtime, WeightSpec
from .linear import Linear


class TwoMapAttention(Mixer):
    capture_safe = True
    kernels_only = True

    def __init__(self, prefix: str, hidden_size: int, heads: int, kv_heads: int, head_dim: int, value_dim: int, scale: float, diff: float,
                 eps: float, *, reads_only: bool = False, names: Optional[Dict[str, str]] = None, out_dtype: Optional[torch.dtype] = None):
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads are not a multiple of {kv_heads} kv heads")
        n = {"q": "q", "k": "k", "v": "v", "o": "o", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2", "lk2": "lk2"}
        n.update(names or {})
        self.names = {key: prefix + value for key, value in n.items()}
        self.hidden_size, self.heads, self.kv_heads, self.head_dim, self.value_dim = hidden_size, heads, kv_heads, head_dim, value_dim
        self.scale, self.diff, self.eps, self.reads_only, self.out_dtype = float(scale), float(diff), float(eps), reads_only, out_dtype
        self.pad_dim = -(-max(2 * head_dim, value_dim) // 8) * 8
        sources = [(self.names["q"], heads * 2 * head_dim)]
        if not reads_only:
            sources += [(self.names["k"], kv_heads * 2 * head_dim), (self.names["v"], kv_heads * value_dim)]
        self.qkv = Linear(sources, hidden_size)
        self.out = Linear([(self.names["o"], hidden_size)], heads * value_dim)
        self.factor = None  # lambda

    def cache_need(self) -> KVCacheNeed:
        return KVCacheNeed(self.kv_heads, self.pad_dim, None, key_dim=2 * self.head_dim, value_dim=self.value_dim)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {**self.qkv.weight_specs(), **self.out.weight_specs(),
                **{self.names[key]: WeightSpec((self.head_dim,), "bias") for key in ("lq1", "lk1", "lq2", "lk2")}}

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        self.qkv.load(weights, rt)
        self.out.load(weights, rt)
        lq1, lk1, lq2, lk2 = (weights.stored(self.names[key]).to(device="cpu", dtype=torch.float64) for key in ("lq1", "lk1", "lq2", "lk2"))
        self.factor = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + self.diff

    def forward(self, x, batch, cache, write_cache: bool = True) -> torch.Tensor:
        ops = self.rt.ops
        if write_cache == self.reads_only:
            raise ValueError("a two-map layer with k and v projections fills its cache, one without reads another layer's")
        nkv = 0 if self.reads_only else self.kv_heads
        table = batch.block_tables[cache.group]
        q = ops.qkv_rope_write(self.qkv.forward(x, torch.float32), self.heads, nkv, 2 * self.head_dim, self.value_dim, self.pad_dim, None,
                               None, None, None, None, 0, 0, cache.kv, table, batch.request_of_token, batch.positions, self.rt.dtype,
                               q_maps=2)
        mixed = ops.paged_attention(q, cache.kv, table, batch, None, self.scale)
        heads = ops.map_difference(mixed, self.heads, self.value_dim, self.pad_dim, self.factor, self.eps, 1.0 - self.diff)
        return self.out.forward(heads, self.out_dtype)
