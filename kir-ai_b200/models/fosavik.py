"""The Fosavik decoder put together from parts.

Embedding rows plus a learned vector per position; the residual stream kept as several copies, of which every sub-layer
reads a weighted sum through an RMS norm and which are all made afresh from the old ones and the sub-layer's output; three
kinds of mixer, in whatever order the configuration lists them: attention as the difference of two maps over the same
values (a layer may read an earlier one's keys and values), a state-space mixer, and two mixers side by side on the same
rows, added with constants: grouped-query attention with a norm on queries and keys, values that are the keys as projected,
a window under which a sequence's first keys stay visible, one added to the softmax's denominator and one sigmoid gate per
head, next to a real-gated linear recurrence behind a short convolution; a clamped gated feed-forward, or none; the norm of
the copies' sum, then an output head of its own.

Tensor names: ``embed``, ``pos``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.{in,out,mix}``,
``l<i>.mix.*`` (two maps: ``q``, ``k``, ``v``, ``o``, ``lq1``, ``lk1``, ``lq2``, ``lk2``; state space: ``in``, ``conv``,
``conv.b``, ``dt_bias``, ``A_log``, ``D``, ``norm``, ``o``; side by side: ``left.{q,k,q.norm,k.norm,g,o}``,
``right.{y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,lam,o}``), ``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import torch

from ..config.fosavik import FosavikConfig
from ..parts import (Block, Embedding, GatedLinearRecurrence, GatedMLP, GQAttention, OutputHead, RMSNorm, ScaledPairMixer, StateSpaceMixer,
                     StreamConnection, TwoMapAttention)
from .plan import LayerCall, ModelPlan

_ATTENTION_NAMES = {"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}
_MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}
MLP_SLOPE = 1.702      # the design's constant inside the feed-forward's sigmoid
SINK_SCORE = 0.0       # one is added to the softmax's denominator
RECURRENCE_DECAY = 8.0  # the design's factor on the recurrence's log decay


def mixer_for_layer(cfg: FosavikConfig, layer, prefix: str):
    """The mixer of one configured layer, its tensors under ``prefix``; it leaves 32-bit rows."""
    m = layer.mixer
    if layer.kind == "attention":
        return TwoMapAttention(prefix, cfg.width, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.diff, cfg.norm_eps,
                               reads_only=m.kv_from is not None, out_dtype=torch.float32)
    if layer.kind == "mamba2":
        return StateSpaceMixer(prefix, cfg.width, m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups, cfg.norm_eps,
                               out_dtype=torch.float32)
    a, b = m.left, m.right
    left = GQAttention(prefix + "left.", cfg.width, a.heads, a.kv_heads, a.dim, None, window=a.window, scale=a.scale,
                       qk_norm_eps=cfg.norm_eps, names=_ATTENTION_NAMES, head_gate="g", keep_first=a.keep_first if a.window else 0,
                       keys_as_values=True, sink=SINK_SCORE, out_dtype=torch.float32)
    right = GatedLinearRecurrence(prefix + "right.", cfg.width, b.width, b.blocks, b.conv, RECURRENCE_DECAY, out_dtype=torch.float32)
    return ScaledPairMixer(left, right, cfg.width, m.left_scale, m.right_scale, out_dtype=torch.float32)


def feed_forward_for_layer(cfg: FosavikConfig, layer, prefix: str):
    if layer.mlp is None:
        return None
    return GatedMLP(prefix, cfg.width, layer.mlp.ff, "clamped", names=_MLP_NAMES, out_dtype=torch.float32, limit=layer.mlp.limit,
                    slope=MLP_SLOPE)


def build_fosavik_plan(cfg: FosavikConfig) -> ModelPlan:
    blocks, order, next_cache, cache_of = [], [], 0, {}
    for index, layer in enumerate(cfg.layers):
        base = f"l{index}."
        ffn = feed_forward_for_layer(cfg, layer, base + "mlp.")
        second = ffn is not None
        blocks.append(Block(RMSNorm(base + "norm1", cfg.width, cfg.norm_eps), mixer_for_layer(cfg, layer, base + "mix."),
                            RMSNorm(base + "norm2", cfg.width, cfg.norm_eps) if second else None, ffn, arrangement="streams",
                            connection1=StreamConnection(base + "hc1.", cfg.streams),
                            connection2=StreamConnection(base + "hc2.", cfg.streams) if second else None))
        if layer.kind == "parallel":
            # pages for the attention side, a state slot for the recurrence
            order.append(LayerCall(block=index, cache=(next_cache, next_cache + 1), write=True))
            next_cache += 2
        elif layer.kind == "attention" and layer.mixer.kv_from is not None:
            order.append(LayerCall(block=index, cache=cache_of[layer.mixer.kv_from], write=False))
        else:
            order.append(LayerCall(block=index, cache=next_cache, write=True))
            cache_of[index] = next_cache
            next_cache += 1
    return ModelPlan(
        embedding=Embedding("embed", cfg.vocab, cfg.width, position_table=("pos", cfg.max_positions)),
        blocks=blocks,
        order=order,
        final_norm=RMSNorm("final.norm", cfg.width, cfg.norm_eps),
        head=OutputHead("head", cfg.vocab, cfg.width),
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
    ).validate()
