"""Gated linear attention: a matrix state per head whose rows decay each at a rate of their own.

Per head, with q = W_q h * d^(-1/2), k = W_k h (d columns) and v = W_v h (dv columns): a decay per key column
a = sigmoid(W_a2 (W_a1 h) + b)^(1 / ``tau``), the state S_t = diag(a_t) S_(t-1) + k_t v_t^T from S = 0, the read-out
o_t = S_t^T q_t.  Each head's o is divided by its root mean square (eps inside the root) and multiplied by one weight [dv]
that the heads share; the heads side by side are multiplied by silu(W_g h) and projected out.

One stacked product gives q, k, v, the gate and the short row W_a1 h in 32-bit; W_a2 runs on that row in 32-bit inside the
recurrence's kernels.  The size between W_a1 and W_a2 is the stored tensors' own.  What a request keeps between steps is one
slot row in 32-bit: S [H, d, dv], zero at a sequence's start.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Mixer, OpenSize, Runtime, StateNeed, WeightSpec
from .linear import Linear

DEFAULT_RANK = 16  # of the decays' projection where random weights are made


class DecayedLinearAttention(Mixer):
    capture_safe = True  # slots and row boundaries are read on the device; a step of single tokens walks one token
    kernels_only = True

    def __init__(self, prefix: str, hidden_size: int, heads: int, key_dim: int, value_dim: int, tau: float, eps: float,
                 names: Optional[Dict[str, str]] = None, out_dtype: Optional[torch.dtype] = None):
        if not tau > 0.0:
            raise ValueError(f"the decays' root must be positive, got {tau}")
        n = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1", "a2": "a2", "a2_bias": "a2.b"}
        n.update(names or {})
        self.names = {key: prefix + value for key, value in n.items()}
        self.hidden_size, self.heads, self.key_dim, self.value_dim = hidden_size, heads, key_dim, value_dim
        self.tau, self.eps, self.out_dtype = float(tau), float(eps), out_dtype
        self.inputs: Optional[Linear] = None  # made at load, when the stored tensors have told the decays' rank
        self.out = Linear([(self.names["o"], hidden_size)], heads * value_dim)
        self.up = self.up_bias = self.norm = None

    def cache_need(self) -> StateNeed:
        return StateNeed((self.heads * self.key_dim * self.value_dim,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, keys, values = self.names, self.heads * self.key_dim, self.heads * self.value_dim
        rank = OpenSize(n["a1"] + " rows", DEFAULT_RANK)
        return {n["q"]: WeightSpec((keys, self.hidden_size)), n["k"]: WeightSpec((keys, self.hidden_size)),
                n["v"]: WeightSpec((values, self.hidden_size)), n["g"]: WeightSpec((values, self.hidden_size)),
                n["a1"]: WeightSpec((rank, self.hidden_size)), n["a2"]: WeightSpec((keys, rank)), n["a2_bias"]: WeightSpec((keys,), "bias"),
                n["norm"]: WeightSpec((self.value_dim,), "norm"), **self.out.weight_specs()}

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        n, keys, values = self.names, self.heads * self.key_dim, self.heads * self.value_dim
        rank = weights.stored(n["a1"]).shape[0]
        self.inputs = Linear([(n["q"], keys), (n["k"], keys), (n["v"], values), (n["g"], values), (n["a1"], rank)], self.hidden_size)
        self.inputs.load(weights, rt)
        self.out.load(weights, rt)
        self.up = weights.on_device(n["a2"], torch.float32).t().contiguous()
        self.up_bias = weights.on_device(n["a2_bias"], torch.float32)
        self.norm = weights.on_device(n["norm"], torch.float32).repeat(self.heads).contiguous()

    def forward(self, x, batch, cache, write_cache: bool = True) -> torch.Tensor:
        rows = self.inputs.forward(x, torch.float32)
        mixed = self.rt.ops.channel_scan(rows, self.up, self.up_bias, self.tau, self.key_dim ** -0.5, cache.state, batch, self.heads,
                                         self.key_dim, self.value_dim, self.norm, self.eps, self.rt.dtype)
        return self.out.forward(mixed, self.out_dtype)
