"""Two mixers side by side on the same rows: out = (rms(left(h)) * w_left + rms(right(h)) * w_right) / 2, each output
divided by its root mean square over the model width (eps inside the root) and multiplied by a plain weight of its own.

Each side keeps what it needs (pages for attention, a state slot for a recurrence): ``cache_need()`` is the tuple of
both needs, the layer call names a cache layer for each, and ``forward`` gets the tuple of views.  Both sides are built
to leave 32-bit rows; the mean is 32-bit.

``ScaledPairMixer`` adds them up with constants instead: out = c_left left(h) + c_right right(h).  Where both sides can
leave their outer products to it (``input_sources``, ``mix_into``, ``output_source``; a side may say no with
``can_share_products``), one stacked product reads h for both sides, each side writes what its output projection reads,
times its constant, into its columns of one buffer, and one product over the output projections side by side makes the
sum; the constants multiply 32-bit values ahead of the rounding to the runtime dtype, so the matrices stay as stored.
Otherwise the sides run whole and a kernel adds their 32-bit rows.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Mixer, Runtime, WeightSpec
from .linear import Linear


class SideBySideMixer(Mixer):
    def __init__(self, left: Mixer, right: Mixer, hidden_size: int, left_weight: str, right_weight: str, eps: float):
        self.left, self.right, self.hidden_size, self.eps = left, right, hidden_size, float(eps)
        self.left_weight_name, self.right_weight_name = left_weight, right_weight
        self.left_weight = self.right_weight = None
        if left.cache_need() is None or right.cache_need() is None:
            raise ValueError("both sides keep something between steps in this arrangement")

    @property
    def capture_safe(self) -> bool:
        return bool(self.left.capture_safe) and bool(self.right.capture_safe)

    @property
    def kernels_only(self) -> bool:
        return bool(self.left.kernels_only) and bool(self.right.kernels_only)

    def cache_need(self):
        return (self.left.cache_need(), self.right.cache_need())

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {**self.left.weight_specs(), **self.right.weight_specs(),
                self.left_weight_name: WeightSpec((self.hidden_size,), "norm"),
                self.right_weight_name: WeightSpec((self.hidden_size,), "norm")}

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        self.left.load(weights, rt)
        self.right.load(weights, rt)
        self.left_weight = weights.on_device(self.left_weight_name, torch.float32)
        self.right_weight = weights.on_device(self.right_weight_name, torch.float32)

    def forward(self, x, batch, cache, write_cache: bool = True) -> torch.Tensor:
        left_view, right_view = cache
        a = self.left.forward(x, batch, left_view, write_cache)
        b = self.right.forward(x, batch, right_view, write_cache)
        a = a if a.dtype == torch.float32 else a.float()
        b = b if b.dtype == torch.float32 else b.float()
        return self.rt.ops.rms_pair_mean(a, b, self.left_weight, self.right_weight, self.eps)


class ScaledPairMixer(Mixer):
    def __init__(self, left: Mixer, right: Mixer, hidden_size: int, left_scale: float, right_scale: float,
                 out_dtype: Optional[torch.dtype] = None):
        self.left, self.right, self.hidden_size, self.out_dtype = left, right, hidden_size, out_dtype
        self.scales = (float(left_scale), float(right_scale))
        if left.cache_need() is None or right.cache_need() is None:
            raise ValueError("both sides keep something between steps in this arrangement")
        # the right side's columns come first in the stacked input product, the left side's in the buffer of the output product
        self.fused = all(hasattr(side, "mix_into") and getattr(side, "can_share_products", lambda: True)() for side in (left, right))
        if self.fused:
            left.shares_products = right.shares_products = True
            self.right_rows = sum(n for _, n in right.input_sources())
            self.inputs = Linear(right.input_sources() + left.input_sources(), hidden_size)
            self.out_parts = [left.output_source(), right.output_source()]
            self.out_columns = [used if groups is None else groups[0] * groups[2] for _, used, groups in self.out_parts]
            self.out = Linear([("", hidden_size)], sum(self.out_columns))  # filled from both sides' matrices at load

    @property
    def capture_safe(self) -> bool:
        return bool(self.left.capture_safe) and bool(self.right.capture_safe)

    @property
    def kernels_only(self) -> bool:
        return bool(self.left.kernels_only) and bool(self.right.kernels_only)

    def cache_need(self):
        return (self.left.cache_need(), self.right.cache_need())

    def weight_specs(self) -> Dict[str, WeightSpec]:
        specs = {**self.left.weight_specs(), **self.right.weight_specs()}
        if self.fused:
            specs.update(self.inputs.weight_specs())
            specs.update({name: WeightSpec((self.hidden_size, used), "linear") for name, used, _ in self.out_parts})
        return specs

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        self.left.load(weights, rt)
        self.right.load(weights, rt)
        if not self.fused:
            return
        self.inputs.load(weights, rt)
        pieces = []
        for (name, used, groups), columns in zip(self.out_parts, self.out_columns):
            matrix = weights.stored(name).to(device=rt.device, dtype=rt.dtype)
            if columns != used:  # heads narrower than their columns of the buffer: zero columns
                count, own, padded = groups
                wide = torch.zeros((self.hidden_size, count, padded), dtype=matrix.dtype, device=matrix.device)
                wide[:, :, :own] = matrix.view(self.hidden_size, count, own)
                matrix = wide.view(self.hidden_size, columns)
            pieces.append(matrix)
        self.out.load_matrix(torch.cat(pieces, dim=1), rt)

    def forward(self, x, batch, cache, write_cache: bool = True) -> torch.Tensor:
        left_view, right_view = cache
        left_scale, right_scale = self.scales
        if not self.fused:
            ops = self.rt.ops
            a = self.left.forward(x, batch, left_view, write_cache)
            b = self.right.forward(x, batch, right_view, write_cache)
            total = torch.zeros((x.shape[0], self.hidden_size), dtype=torch.float32, device=x.device)
            for rows, scale in ((a, left_scale), (b, right_scale)):
                ops.add_scaled_into_residual(total, [rows if rows.dtype == torch.float32 else rows.float()], scale)
            return total if (self.out_dtype or self.rt.dtype) == torch.float32 else total.to(self.rt.dtype)
        rows = self.inputs.forward(x, torch.float32)
        both = torch.empty((rows.shape[0], sum(self.out_columns)), dtype=self.rt.dtype, device=rows.device)
        split = self.out_columns[0]
        self.left.mix_into(rows[:, self.right_rows :], batch, left_view, both[:, :split], left_scale)
        self.right.mix_into(rows[:, : self.right_rows], batch, right_view, both[:, split:], right_scale)
        return self.out.forward(both, self.out_dtype)
