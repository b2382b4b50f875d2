"""The Damilix decoder put together from parts.

Embedding rows through a norm; layers whose sub-layers read the stream itself and whose outputs are normed before they are
added, x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)), and after them an input from the token's own row of a second table;
three kinds of mixer, in whatever order the configuration lists them: latent attention whose queries come straight from the
stream (one small cached row per token for all heads, a learned sink and a sigmoid gate per head) with a rotation that pairs
neighbouring columns and may have its frequencies stretched by their index, the same with a rotation that pairs halves, and
gated linear attention with a decay per key column; a dense gated feed-forward, routed experts (softmax scores with a
correction on the choice, some experts the identity, beside them a gated branch that every token runs), or none; the model's
norm, then an output head of its own.

Tensor names: ``embed``, ``embed.norm``, ``side.embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (latent attention:
``q``, ``dkv``, ``dkv.norm``, ``uk``, ``uv``, ``sink``, ``g``, ``o``; linear attention: ``q``, ``k``, ``v``, ``g``, ``o``,
``norm``, ``a1``, ``a2``, ``a2.b``), ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router,correction,e<j>.{gate,up,down},
shared.{gate,up,down,sg}}``, ``l<i>.side.{gate,proj,norm}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import torch

from ..config.damilix import DamilixConfig, DenseMLP
from ..parts import (Block, DecayedLinearAttention, Embedding, GatedMLP, LatentAttention, OutputHead, RMSNorm, RotaryEmbedding, RoutedExperts,
                     TokenSideInput)
from .plan import LayerCall, ModelPlan

_MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}
_EXPERT_NAMES = {"router": "router", "correction": "correction", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down"}
_PAIRING = {"latent_attention": "neighbours", "latent_attention_2": "halves"}


def _rotary(rot, pairing: str) -> RotaryEmbedding:
    scaling = None
    if rot.scaling is not None:
        scaling = {"factor": rot.scaling.factor, "original": rot.scaling.original, "fast": rot.scaling.fast, "slow": rot.scaling.slow}
    return RotaryEmbedding(rot.dims, rot.base, rot.dims, scaling=scaling, precise=True, pairing=pairing)


def mixer_for_layer(cfg: DamilixConfig, layer, prefix: str):
    """The mixer of one configured layer, its tensors under ``prefix``; it leaves 32-bit rows."""
    m = layer.mixer
    if layer.kind == "gla":
        return DecayedLinearAttention(prefix, cfg.width, m.heads, m.dim, m.vdim, m.tau, cfg.norm_eps, out_dtype=torch.float32)
    return LatentAttention(prefix, cfg.width, m.heads, m.dim, m.rot_dim, m.vdim, None, m.kv_rank, m.scale, cfg.norm_eps,
                           _rotary(m.rot, _PAIRING[layer.kind]), out_dtype=torch.float32, head_gate="g", sink="sink")


def feed_forward_for_layer(cfg: DamilixConfig, layer, prefix: str):
    mlp = layer.mlp
    if mlp is None:
        return None
    if isinstance(mlp, DenseMLP):
        return GatedMLP(prefix, cfg.width, mlp.ff, "silu", names=_MLP_NAMES, out_dtype=torch.float32)
    shared = None
    if mlp.shared_ff is not None:
        shared = GatedMLP(prefix + "shared.", cfg.width, mlp.shared_ff, "silu", names=_MLP_NAMES, out_dtype=torch.float32)
    return RoutedExperts(prefix, cfg.width, mlp.ff, mlp.experts, mlp.top, activation="silu_gated", names=_EXPERT_NAMES,
                         out_dtype=torch.float32, scoring="softmax_corrected", shared=shared, correction=True, weight_scale=mlp.scale,
                         identity=mlp.identity, shared_gate="shared.sg" if shared is not None else None)


def build_damilix_plan(cfg: DamilixConfig) -> ModelPlan:
    blocks, order = [], []
    for index, layer in enumerate(cfg.layers):
        base = f"l{index}."
        ffn = feed_forward_for_layer(cfg, layer, base + "mlp.")
        blocks.append(Block(RMSNorm(base + "norm1", cfg.width, cfg.norm_eps), mixer_for_layer(cfg, layer, base + "mix."),
                            RMSNorm(base + "norm2", cfg.width, cfg.norm_eps) if ffn is not None else None, ffn, arrangement="out_norm",
                            side=TokenSideInput(base + "side.", "side.embed", cfg.width, cfg.side_dim, index * cfg.side_dim, cfg.vocab,
                                                len(cfg.layers) * cfg.side_dim, cfg.norm_eps)))
        order.append(LayerCall(block=index, cache=index, write=True))
    return ModelPlan(
        embedding=Embedding("embed", cfg.vocab, cfg.width, norm=("embed.norm", cfg.norm_eps)),
        blocks=blocks,
        order=order,
        final_norm=RMSNorm("final.norm", cfg.width, cfg.norm_eps),
        head=OutputHead("head", cfg.vocab, cfg.width),
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=None,
    ).validate()
