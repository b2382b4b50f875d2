"""Typed configuration of the Damilix decoder.

config.json of this design is nested: ``architecture`` (a string), ``width``, ``vocab``, ``norm.eps``,
``token_side.dim`` (columns of a token's own input per layer) and ``layers``.  Every entry of ``layers`` has ``type`` (the
kind of mixer), ``mixer`` (its sizes and constants) and ``mlp`` (null for a layer without feed-forward).  The kinds of
mixer:

* ``latent_attention`` (the rotation pairs neighbouring columns) and ``latent_attention_2`` (it pairs halves): ``heads``,
  ``dim`` (unrotated) and ``rot_dim`` (rotated query/key columns of a head), ``vdim``, ``kv_rank`` (size of the cached
  latent), ``scale`` (the factor on the scores), ``rot`` (``base``; ``dims`` equals ``rot_dim``; optionally ``scaling``
  with ``factor``, ``original``, ``fast``, ``slow``);
* ``gla``: ``heads``, ``dim`` (key columns of a head), ``vdim`` (value columns) and ``tau`` (the decays are a sigmoid to
  the power 1 / tau).  The size between the two matrices that make the decays is the stored tensors' own.

The kinds of feed-forward: ``dense`` with ``ff``; ``moe`` with ``expert`` (``ff``), ``router`` (``experts``, ``top``,
``scale``, optionally ``identity``: experts that hand the input on) and optionally ``shared`` (``ff``).  Every size and
constant that a model of the design may set is read from there.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .base import ConfigError, optional_int, required_float, required_int
from .bikilix import IndexScaling

_FAMILY = "damilix"
LATENT_KINDS = ("latent_attention", "latent_attention_2")
MIXER_KINDS = LATENT_KINDS + ("gla",)
MLP_KINDS = ("dense", "moe")


def _mapping(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError.unsupported(f"{_FAMILY} config {where} missing {key}")
    return value


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    scaling: Optional[IndexScaling] = None

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "Rotation":
        scaling = None
        if raw.get("scaling") is not None:
            sc = _mapping(raw, "scaling", where)
            scaling = IndexScaling(*(required_float(sc, key, _FAMILY) for key in ("factor", "original", "fast", "slow")))
            if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0.0:
                raise ConfigError.invalid(f"{_FAMILY} config {where}.scaling needs positive constants")
        dims = required_int(raw, "dims", _FAMILY)
        if dims % 2:
            raise ConfigError.invalid(f"{_FAMILY} config {where}.dims must be even, got {dims}")
        base = required_float(raw, "base", _FAMILY)
        if base <= 1.0:
            raise ConfigError.invalid(f"{_FAMILY} config {where}.base must exceed one, got {base}")
        return cls(base=base, dims=dims, scaling=scaling)

    def to_dict(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = self.scaling.to_dict()
        return out


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation

    def to_dict(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot": self.rot.to_dict(), "rot_dim": self.rot_dim,
                "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class DecayMixer:
    heads: int
    dim: int
    vdim: int
    tau: float

    def to_dict(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}


@dataclass(frozen=True)
class DenseMLP:
    ff: int

    def to_dict(self) -> dict:
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class ExpertsMLP:
    ff: int
    experts: int
    identity: int
    top: int
    scale: float
    shared_ff: Optional[int] = None

    def to_dict(self) -> dict:
        out = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top, "scale": self.scale}}
        if self.identity:
            out["router"]["identity"] = self.identity
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class DamilixLayer:
    kind: str
    mixer: object
    mlp: object  # DenseMLP, ExpertsMLP or None


def _mixer(kind: str, m: Mapping[str, Any], where: str):
    heads, dim, vdim = (required_int(m, key, _FAMILY) for key in ("heads", "dim", "vdim"))
    if kind == "gla":
        tau = required_float(m, "tau", _FAMILY)
        if tau <= 0.0:
            raise ConfigError.invalid(f"{_FAMILY} config {where}: tau must be positive, got {tau}")
        return DecayMixer(heads=heads, dim=dim, vdim=vdim, tau=tau)
    rot = Rotation.from_dict(_mapping(m, "rot", where), where + ".rot")
    rot_dim = required_int(m, "rot_dim", _FAMILY)
    if rot.dims != rot_dim:
        raise ConfigError.invalid(f"{_FAMILY} config {where}: rot.dims {rot.dims} must equal rot_dim {rot_dim}")
    return LatentMixer(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=required_int(m, "kv_rank", _FAMILY),
                       scale=required_float(m, "scale", _FAMILY), rot=rot)


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind not in MLP_KINDS:
        raise ConfigError.unsupported(f"{_FAMILY} config {where}: feed-forward kind {kind!r} is unsupported; known: {', '.join(MLP_KINDS)}")
    if kind == "dense":
        return DenseMLP(ff=required_int(mlp, "ff", _FAMILY))
    expert, router = _mapping(mlp, "expert", where), _mapping(mlp, "router", where)
    experts, top = required_int(router, "experts", _FAMILY), required_int(router, "top", _FAMILY)
    identity = optional_int(router, "identity", _FAMILY, 0)
    if not 0 < top <= experts + identity:
        raise ConfigError.invalid(f"{_FAMILY} config {where}: a token uses {top} of {experts + identity} experts")
    shared_ff = None
    if mlp.get("shared") is not None:
        shared_ff = required_int(_mapping(mlp, "shared", where), "ff", _FAMILY)
    return ExpertsMLP(ff=required_int(expert, "ff", _FAMILY), experts=experts, identity=identity, top=top,
                      scale=required_float(router, "scale", _FAMILY), shared_ff=shared_ff)


@dataclass(frozen=True)
class DamilixConfig:
    width: int
    vocab: int
    norm_eps: float
    side_dim: int
    layers: Tuple[DamilixLayer, ...]

    architecture = "Damilix"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DamilixConfig":
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
            layers.append(DamilixLayer(kind, _mixer(kind, _mapping(entry, "mixer", where), where + ".mixer"),
                                       _mlp(entry.get("mlp"), where + ".mlp")))
        eps = required_float(_mapping(raw, "norm", "root"), "eps", _FAMILY)
        if eps < 0.0:
            raise ConfigError.invalid(f"{_FAMILY} config norm.eps must be non-negative")
        return cls(width=required_int(raw, "width", _FAMILY), vocab=required_int(raw, "vocab", _FAMILY), norm_eps=eps,
                   side_dim=required_int(_mapping(raw, "token_side", "root"), "dim", _FAMILY), layers=tuple(layers))

    def to_dict(self) -> dict:
        """The config.json content that parses back to this configuration."""
        layers = [{"type": layer.kind, "mixer": layer.mixer.to_dict(), "mlp": None if layer.mlp is None else layer.mlp.to_dict()}
                  for layer in self.layers]
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "token_side": {"dim": self.side_dim}, "layers": layers}
