"""A residual stream kept as several copies (hyper-connections), read and rewritten around a sub-layer.

A sub-layer reads u = sum_f in[f] x_f of the copies x_1 .. x_s through its norm; from its output y every copy is made
afresh from all the old ones, x_t <- sum_f mix[f, t] x_f + out[t] y.  ``StreamConnection`` holds one sub-layer's in, mix and
out.  All copies equal the embedding's rows at the start, and the model's last norm reads their sum.

How it runs: the copies live as one 32-bit tensor [T, s, width] (as the embedding's [T, width] while they are still equal);
what a sub-layer produced travels to the next reader of the stream as a ``StreamUpdate``, and a norm that ``takes_streams``
makes the new copies, the next sub-layer's reading of them and the norm in one pass over the token's rows
(``ops.streams_norm``).  For any other norm the same kernel leaves u in 32-bit rows, which the norm then reads.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Norm, Part, Runtime, StreamUpdate, WeightSpec


class StreamConnection(Part):
    capture_safe = True
    kernels_only = True

    def __init__(self, prefix: str, copies: int, names: Optional[Dict[str, str]] = None):
        if copies < 1:
            raise ValueError(f"a stream has at least one copy, got {copies}")
        n = {"in": "in", "out": "out", "mix": "mix"}
        n.update(names or {})
        self.copies = copies
        self.names = {key: prefix + value for key, value in n.items()}
        self.read = self.add = self.mix = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        s, n = self.copies, self.names
        return {n["in"]: WeightSpec((s,), "norm"), n["out"]: WeightSpec((s,), "norm"), n["mix"]: WeightSpec((s, s), "identity")}

    def load(self, weights, rt: Runtime) -> None:
        self.rt = rt
        self.read, self.add, self.mix = (weights.on_device(self.names[key], torch.float32) for key in ("in", "out", "mix"))

    def enter(self, streams: torch.Tensor, left, norm: Norm):
        """(rows that the sub-layer reads, the streams it leaves its update for): the update ``left`` (a ``StreamUpdate``
        or None) is made, and the copies are read through ``norm``."""
        if getattr(norm, "takes_streams", False):
            return norm.forward_streams(streams, self.copies, left, self.read)
        u, streams = self.rt.ops.streams_norm(streams, self.copies, left.terms() if left is not None else None, self.read, None, 0.0,
                                              torch.float32)
        return norm.forward(u), streams

    def leave(self, y: torch.Tensor) -> StreamUpdate:
        """What is left to be done to the streams after the sub-layer produced ``y`` (32-bit rows)."""
        return StreamUpdate(y if y.dtype == torch.float32 else y.float(), self.mix, self.add)
