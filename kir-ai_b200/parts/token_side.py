"""An input that every layer takes from a table row of the token's own: after the layer's sub-layers the stream x gets
rms(W_proj (gelu_tanh(W_gate x) * e)) * w added, e the layer's part of the token's row (columns ``first`` to ``first`` +
``dim``), rms with eps inside the root.  The table is shared by all layers.  The norm, the add and the stream's copy for the
next reader are one kernel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Part, Runtime, WeightSpec
from .linear import Linear


class TokenSideInput(Part):
    capture_safe = True
    kernels_only = True

    def __init__(self, prefix: str, table_name: str, hidden_size: int, dim: int, first: int, vocab_size: int, row: int, eps: float,
                 names: Optional[Dict[str, str]] = None):
        n = {"gate": "gate", "proj": "proj", "norm": "norm"}
        n.update(names or {})
        if first < 0 or first + dim > row:
            raise ValueError(f"columns {first} to {first + dim} do not lie inside a row of {row}")
        self.table_name, self.norm_name = table_name, prefix + n["norm"]
        self.hidden_size, self.dim, self.first, self.vocab_size, self.row, self.eps = hidden_size, dim, first, vocab_size, row, float(eps)
        self.gate = Linear([(prefix + n["gate"], dim)], hidden_size)
        self.proj = Linear([(prefix + n["proj"], hidden_size)], dim)
        self.table = self.weight = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {self.table_name: WeightSpec((self.vocab_size, self.row), "embedding"), **self.gate.weight_specs(), **self.proj.weight_specs(),
                self.norm_name: WeightSpec((self.hidden_size,), "norm")}

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        self.table = weights.on_device(self.table_name, rt.dtype)  # one copy for all layers
        self.gate.load(weights, rt)
        self.proj.load(weights, rt)
        self.weight = weights.on_device(self.norm_name, torch.float32)

    def add(self, x: torch.Tensor, resid: torch.Tensor, batch) -> Optional[torch.Tensor]:
        """The stream ``resid`` (32-bit, in place) takes the input; ``x`` is the stream in the runtime dtype.  Returns the new
        stream in that dtype, or None when that is the stream's own."""
        ops = self.rt.ops
        g = ops.token_gate(self.gate.forward(x, torch.float32), self.table, batch.token_ids, self.first)
        return ops.norm_add(resid, self.proj.forward(g, torch.float32), self.weight, self.eps,
                            None if self.rt.dtype == torch.float32 else self.rt.dtype)
