"""A real-gated linear recurrence behind a short convolution, beside a gelu branch (the recurrent block of Griffin, with its
real-gated linear recurrent unit).

Two projections of the mixer's input h, each with a bias: the branch y = W_y h + b_y, and W_x h + b_x, which passes a causal
convolution per channel over ``conv_taps`` tokens (a bias, no activation; the stored taps' last column weighs the token
itself; zeros lie before a sequence's start) and gives u.  In each of ``blocks`` equal parts of the channels two square
matrices make the gates r = sigmoid(W_r u + b_r) and i = sigmoid(W_i u + b_i).  Per channel
a_t = exp(-c r_t softplus(lambda)), S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t, from S = 0 (``decay`` is the constant c).
The output is W_o (S * gelu_tanh(y)).

What a request keeps between steps is one slot row in 32-bit: the convolution's last ``conv_taps - 1`` input rows (with
their bias), then S; both start at zero.  The stacked input product leaves 32-bit rows; convolution, gates, decays and the
recurrence are 32-bit.  The gates' products run in 32-bit multiply-adds, or, for steps of many tokens in bfloat16, on the
tensor cores with u as two bfloat16 numbers, high + low (``ops.block_product_pairs``), so that u is not rounded to 16 bits
ahead of a gate either way.  A step of single tokens runs everything between the outer products as one kernel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Mixer, Runtime, StateNeed, WeightSpec
from .linear import Linear


class GatedLinearRecurrence(Mixer):
    capture_safe = True  # slots and row boundaries are read on the device; a step of single tokens walks one token
    kernels_only = True

    PAIRS_MIN_ROWS = 256  # tokens from which the gates' products run on the tensor cores

    def __init__(self, prefix: str, hidden_size: int, width: int, blocks: int, conv_taps: int, decay: float = 8.0,
                 names: Optional[Dict[str, str]] = None, out_dtype: Optional[torch.dtype] = None):
        if width % blocks:
            raise ValueError(f"{width} channels do not split into {blocks} equal blocks")
        if conv_taps < 1:
            raise ValueError("the convolution has at least one tap")
        n = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra", "r_bias": "ra.b",
             "i": "ri", "i_bias": "ri.b", "rate": "lam", "o": "o"}
        n.update(names or {})
        self.names = {key: prefix + value for key, value in n.items()}
        self.hidden_size, self.width, self.blocks, self.block, self.conv_taps = hidden_size, width, blocks, width // blocks, conv_taps
        self.decay, self.out_dtype = float(decay), out_dtype
        self.inputs = Linear(self.input_sources(), hidden_size)
        self.out = Linear([(self.names["o"], hidden_size)], width)
        self.conv_len = (conv_taps - 1) * width
        self.shares_products = False  # set by a mixer that makes this part's outer products itself
        self.gates = self.gate_pairs = None

    # what a mixer that shares its products with another's needs (``parts.side_by_side.ScaledPairMixer``)
    def input_sources(self):
        """The stored matrices that read the mixer's input, in the order in which their columns are expected."""
        return [(self.names["y"], self.width), (self.names["x"], self.width)]

    def output_source(self):
        """(matrix, columns it reads, column groups) of the output projection."""
        return self.names["o"], self.width, None

    def cache_need(self) -> StateNeed:
        return StateNeed((self.conv_len + self.width,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, W, d = self.names, self.width, self.block
        specs = {n["y_bias"]: WeightSpec((W,), "bias"), n["x_bias"]: WeightSpec((W,), "bias"),
                 n["conv"]: WeightSpec((W, self.conv_taps), "linear"), n["conv_bias"]: WeightSpec((W,), "bias"),
                 n["r"]: WeightSpec((self.blocks, d, d), "linear"), n["r_bias"]: WeightSpec((self.blocks, d), "bias"),
                 n["i"]: WeightSpec((self.blocks, d, d), "linear"), n["i_bias"]: WeightSpec((self.blocks, d), "bias"),
                 n["rate"]: WeightSpec((W,), "bias")}
        if not self.shares_products:
            specs = {**self.inputs.weight_specs(), **self.out.weight_specs(), **specs}
        return specs

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        n, d = self.names, self.block
        if not self.shares_products:
            self.inputs.load(weights, rt)
            self.out.load(weights, rt)
        for key in ("y_bias", "x_bias", "conv", "conv_bias"):
            setattr(self, key, weights.on_device(n[key], torch.float32))
        self.r_bias = weights.on_device(n["r_bias"], torch.float32).reshape(-1)
        self.i_bias = weights.on_device(n["i_bias"], torch.float32).reshape(-1)
        # the decay per unit of r: worked out in 64-bit, kept in 32-bit
        lam = weights.stored(n["rate"]).to(device=rt.device, dtype=torch.float64)
        self.rate = (-self.decay * torch.nn.functional.softplus(lam, threshold=40.0)).to(torch.float32).contiguous()
        stacked = torch.cat([weights.stored(n[key]).to(device=rt.device) for key in ("r", "i")], dim=1)  # [blocks, 2 d, d]
        self.gates = stacked.to(torch.float32).contiguous()
        # (what a step of single tokens reads: stored bfloat16 matrices as they are, which changes no product)
        self.step_gates = stacked.contiguous() if stacked.dtype == torch.bfloat16 else self.gates
        self.gate_pairs = None
        if rt.dtype == torch.bfloat16 and d % 4 == 0 and stacked.dtype == torch.bfloat16:
            pairs = torch.cat([stacked, stacked], dim=2).reshape(self.blocks * 2 * d, 2 * d).contiguous()
            self.gate_pairs = rt.ops.tile_weight(pairs) if (2 * d) % 128 == 0 else pairs

    def mix_into(self, rows: torch.Tensor, batch, cache, out: torch.Tensor, factor: float = 1.0) -> torch.Tensor:
        """Everything between the products: ``rows`` [T, 2 width] (float32, what the input matrices made: y, then x) to
        ``out`` [T, width], what the output projection reads, times ``factor``."""
        ops, tokens = self.rt.ops, rows.shape[0]
        if ops.real_gated_step_takes(batch, self.block):
            return ops.real_gated_step(rows, self.width, self.block, self.conv, self.x_bias, self.conv_bias, self.step_gates, self.r_bias,
                                       self.i_bias, self.y_bias, self.rate, cache.state, 0, self.conv_len, batch, out, factor)
        branch, x = rows[:, : self.width], rows[:, self.width : 2 * self.width]
        if self.gate_pairs is not None and tokens >= self.PAIRS_MIN_ROWS:
            u, pair = ops.conv_rows(x, self.conv, self.conv_bias, cache.state, 0, batch, in_bias=self.x_bias, pair_block=self.block,
                                    pair_tokens=-(-tokens // 128) * 128)
            gates = ops.block_product_pairs(pair, self.gate_pairs)
        else:
            u = ops.conv_rows(x, self.conv, self.conv_bias, cache.state, 0, batch, in_bias=self.x_bias)
            gates = ops.block_product(u, self.gates, self.blocks)
        return ops.real_gated_scan(u, gates, self.block, branch, self.r_bias, self.i_bias, self.y_bias, self.rate, cache.state,
                                   self.conv_len, batch, out, factor)

    def forward(self, x, batch, cache, write_cache: bool = True) -> torch.Tensor:
        rows = self.inputs.forward(x, torch.float32)
        out = torch.empty((rows.shape[0], self.width), dtype=self.rt.dtype, device=rows.device)
        return self.out.forward(self.mix_into(rows, batch, cache, out), self.out_dtype)
