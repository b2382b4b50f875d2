"""Typed configuration of the Fosavik decoder.

config.json of this design is nested: ``architecture`` (a string), ``width``, ``vocab``, ``max_positions`` (rows of the learned
position table), ``streams`` (copies of the residual stream), ``norm.eps`` and ``layers``.  Every entry of ``layers`` has
``type`` (the kind of mixer), ``mixer`` (its sizes and constants) and ``mlp`` (null for a layer without feed-forward).  The
kinds of mixer:

* ``attention``: two maps over the same values: ``heads``, ``kv_heads``, ``dim`` (query/key size of one map of a head),
  ``vdim`` (value size of a head), ``scale`` (the factor on the scores), ``diff`` (the constant in the second map's weight),
  optionally ``kv_from`` (an earlier attention layer whose keys and values this one reads);
* ``parallel``: two mixers on the same rows.  ``left`` is attention whose values are its keys: ``heads``, ``kv_heads``,
  ``dim``, ``vdim`` (equal to ``dim``), ``scale`` and ``mask`` (``size`` of the window, ``keep_first`` = how many first tokens
  of a sequence every later position still sees).  ``right`` is a gated linear recurrence: ``width`` (channels), ``blocks``
  (equal parts with gate matrices of their own), ``conv`` (taps).  ``left_scale`` and ``right_scale`` multiply the sides;
* ``mamba2``: a state-space mixer: ``heads``, ``vdim`` (columns of a head), ``state`` (rows of a head's state), ``groups`` (of
  heads that share B and C), ``conv`` (taps), ``norm_groups`` (equal parts of the row that the output norm takes one by
  one).

The feed-forward: ``kind`` ``dense`` with ``ff`` and ``limit`` (of the clamp on gate and up).  Every size and constant that a
model of the design may set is read from there.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .base import ConfigError, optional_int, required_float, required_int

_FAMILY = "fosavik"
MIXER_KINDS = ("attention", "parallel", "mamba2")
MLP_KINDS = ("dense",)


def _mapping(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError.unsupported(f"{_FAMILY} config {where} missing {key}")
    return value


def _heads(m: Mapping[str, Any], where: str) -> Tuple[int, int]:
    heads, kv_heads = required_int(m, "heads", _FAMILY), required_int(m, "kv_heads", _FAMILY)
    if heads % kv_heads:
        raise ConfigError.invalid(f"{_FAMILY} config {where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    return heads, kv_heads


@dataclass(frozen=True)
class TwoMaps:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    kv_from: Optional[int] = None

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "TwoMaps":
        heads, kv_heads = _heads(m, where)
        source = m.get("kv_from")
        if source is not None and (not isinstance(source, int) or isinstance(source, bool) or source < 0):
            raise ConfigError.invalid(f"{_FAMILY} config {where}: kv_from must name a layer, got {source!r}")
        return cls(heads=heads, kv_heads=kv_heads, dim=required_int(m, "dim", _FAMILY), vdim=required_int(m, "vdim", _FAMILY),
                   scale=required_float(m, "scale", _FAMILY), diff=required_float(m, "diff", _FAMILY), kv_from=source)

    def to_dict(self) -> dict:
        out = {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class SinkAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: Optional[int]
    keep_first: int

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "SinkAttention":
        heads, kv_heads = _heads(m, where)
        dim = required_int(m, "dim", _FAMILY)
        vdim = dim if m.get("vdim") is None else required_int(m, "vdim", _FAMILY)
        if vdim != dim:
            raise ConfigError.invalid(f"{_FAMILY} config {where}: the values are the keys, yet vdim {vdim} differs from dim {dim}")
        window, keep_first = None, 0
        if m.get("mask") is not None:
            mask = _mapping(m, "mask", where)
            window = required_int(mask, "size", _FAMILY)
            keep_first = optional_int(mask, "keep_first", _FAMILY, 0)
            if keep_first < 0:
                raise ConfigError.invalid(f"{_FAMILY} config {where}: mask.keep_first must not be negative, got {keep_first}")
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, scale=required_float(m, "scale", _FAMILY), window=window, keep_first=keep_first)

    def to_dict(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.dim}
        if self.window is not None:
            out["mask"] = {"keep_first": self.keep_first, "size": self.window}
        return out


@dataclass(frozen=True)
class LinearRecurrence:
    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "LinearRecurrence":
        out = cls(width=required_int(m, "width", _FAMILY), blocks=required_int(m, "blocks", _FAMILY), conv=required_int(m, "conv", _FAMILY))
        if out.width % out.blocks:
            raise ConfigError.invalid(f"{_FAMILY} config {where}: {out.width} channels do not split into {out.blocks} equal blocks")
        return out

    def to_dict(self) -> dict:
        return {"blocks": self.blocks, "conv": self.conv, "width": self.width}


@dataclass(frozen=True)
class ParallelMixer:
    left: SinkAttention
    right: LinearRecurrence
    left_scale: float
    right_scale: float

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}


@dataclass(frozen=True)
class StateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "StateSpace":
        out = cls(heads=required_int(m, "heads", _FAMILY), vdim=required_int(m, "vdim", _FAMILY),
                  state=required_int(m, "state", _FAMILY), groups=required_int(m, "groups", _FAMILY),
                  conv=required_int(m, "conv", _FAMILY), norm_groups=required_int(m, "norm_groups", _FAMILY))
        if out.heads % out.groups:
            raise ConfigError.invalid(f"{_FAMILY} config {where}: {out.heads} heads are not a multiple of {out.groups} groups")
        if (out.heads * out.vdim) % out.norm_groups:
            raise ConfigError.invalid(f"{_FAMILY} config {where}: {out.heads * out.vdim} columns do not split into "
                                      f"{out.norm_groups} equal parts")
        return out

    def to_dict(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups,
                "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class DenseMLP:
    ff: int
    limit: float

    def to_dict(self) -> dict:
        return {"ff": self.ff, "kind": "dense", "limit": self.limit}


@dataclass(frozen=True)
class FosavikLayer:
    kind: str
    mixer: object
    mlp: Optional[DenseMLP]


def _mlp(mlp, where: str) -> Optional[DenseMLP]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind not in MLP_KINDS:
        raise ConfigError.unsupported(f"{_FAMILY} config {where}: feed-forward kind {kind!r} is unsupported; known: {', '.join(MLP_KINDS)}")
    limit = required_float(mlp, "limit", _FAMILY)
    if limit <= 0.0:
        raise ConfigError.invalid(f"{_FAMILY} config {where}: limit must be positive, got {limit}")
    return DenseMLP(ff=required_int(mlp, "ff", _FAMILY), limit=limit)


def _mixer(kind: str, m: Mapping[str, Any], where: str):
    if kind == "attention":
        return TwoMaps.from_dict(m, where)
    if kind == "mamba2":
        return StateSpace.from_dict(m, where)
    return ParallelMixer(SinkAttention.from_dict(_mapping(m, "left", where), where + ".left"),
                         LinearRecurrence.from_dict(_mapping(m, "right", where), where + ".right"),
                         required_float(m, "left_scale", _FAMILY), required_float(m, "right_scale", _FAMILY))


@dataclass(frozen=True)
class FosavikConfig:
    width: int
    vocab: int
    max_positions: int
    streams: int
    norm_eps: float
    layers: Tuple[FosavikLayer, ...]

    architecture = "Fosavik"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FosavikConfig":
        if raw.get("architecture") != cls.architecture:
            raise ConfigError.unsupported(f"config is not a {cls.architecture} model: architecture={raw.get('architecture')!r}")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError.unsupported(f"{_FAMILY} config missing layers")
        layers = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]"
            if not isinstance(entry, Mapping):
                raise ConfigError.invalid(f"{_FAMILY} config {where} must be an object")
            kind = entry.get("type")
            if kind not in MIXER_KINDS:
                raise ConfigError.unsupported(f"{_FAMILY} config {where}: layer type {kind!r} is unsupported; known: {', '.join(MIXER_KINDS)}")
            mixer = _mixer(kind, _mapping(entry, "mixer", where), where + ".mixer")
            source = getattr(mixer, "kv_from", None)
            if source is not None:
                own = layers[source].mixer if source < index else None
                if not isinstance(own, TwoMaps) or own.kv_from is not None:
                    raise ConfigError.invalid(f"{_FAMILY} config {where}: kv_from {source} is no earlier attention layer with keys of its own")
                if (own.heads, own.kv_heads, own.dim, own.vdim) != (mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ConfigError.invalid(f"{_FAMILY} config {where}: head sizes differ from those of layer {source}, whose keys it reads")
            layers.append(FosavikLayer(kind, mixer, _mlp(entry.get("mlp"), where + ".mlp")))
        eps = required_float(_mapping(raw, "norm", "root"), "eps", _FAMILY)
        if eps < 0.0:
            raise ConfigError.invalid(f"{_FAMILY} config norm.eps must be non-negative")
        return cls(width=required_int(raw, "width", _FAMILY), vocab=required_int(raw, "vocab", _FAMILY),
                   max_positions=required_int(raw, "max_positions", _FAMILY), streams=required_int(raw, "streams", _FAMILY), norm_eps=eps,
                   layers=tuple(layers))

    def to_dict(self) -> dict:
        """The config.json content that parses back to this configuration."""
        layers = [{"type": layer.kind, "mixer": layer.mixer.to_dict(), "mlp": None if layer.mlp is None else layer.mlp.to_dict()}
                  for layer in self.layers]
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "max_positions": self.max_positions,
                "streams": self.streams, "norm": {"eps": self.norm_eps}, "layers": layers}
