"""Typed configuration of the Bozevik decoder, read from config.json keys.

A Bozevik model is a list of layers, each with latent attention and an optional feed-forward whose RESULTS are layer-
normalised before they join the stream; every mixer reads its input moved towards the token before it, and what goes on
from a layer is a stored average over everything earlier layers left.  config.json carries:

* ``architecture`` "Bozevik", ``vocab``, ``width``, ``norm.eps``, ``logit_scale``;
* ``layers``: per layer ``type`` ("latent_attention"), ``mixer`` and ``mlp`` (null; ``kind`` "dense" with ``ff`` and
  ``limit``; or ``kind`` "moe" with ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top`` and, optionally,
  ``shared.ff`` and ``shared.limit``).

Mixer: ``heads``, ``dim`` (unrotated query/key size of a head), ``rot_dim`` (rotated size), ``vdim``, ``kv_rank``,
``q_rank``, ``scale``, ``rot`` (``base``; ``dims`` equals ``rot_dim``) and, optionally, ``kv_from``: the layer whose
cached latent this layer reads instead of making its own.

Every size and constant comes from here; this module is the only place that knows the key names.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .lazilorn_config import _number
from .model_config import ConfigError
from .zisesun_config import _count, _get


def _positive(raw: dict[str, Any], key: str, where: str) -> float:
    value = _number(raw, key, where)
    if not value > 0:
        raise ConfigError(f"config.json: {where}: {key!r} must be positive, got {value}")
    return value


@dataclass(frozen=True)
class SharedLatentConfig:
    heads: int
    dim: int            # unrotated query / key size of a head
    rot_dim: int        # rotated query / key size of a head; one key part serves all heads
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    base: float         # of the rotation
    kv_from: int | None = None      # layer whose cached latent and rotated key part this layer reads

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SharedLatentConfig":
        rot_dim = _count(raw, "rot_dim", where)
        if rot_dim % 2:
            raise ConfigError(f"config.json: {where}: 'rot_dim' must be even, got {rot_dim}")
        rot = _get(raw, "rot", dict, where)
        if rot.get("dims", rot_dim) != rot_dim:
            raise ConfigError(f"config.json: {where}.rot: 'dims' ({rot['dims']}) must equal 'rot_dim' ({rot_dim})")
        base = _number(rot, "base", where + ".rot")
        if not base > 1:
            raise ConfigError(f"config.json: {where}.rot: 'base' must be above 1, got {base}")
        kv_from = raw.get("kv_from")
        if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int) or kv_from < 0):
            raise ConfigError(f"config.json: {where}: 'kv_from' must be a layer index, got {kv_from!r}")
        return cls(_count(raw, "heads", where), _count(raw, "dim", where), rot_dim, _count(raw, "vdim", where),
                   _count(raw, "kv_rank", where), _count(raw, "q_rank", where), _number(raw, "scale", where), base, kv_from)

    def to_dict(self) -> dict[str, Any]:
        raw: dict[str, Any] = dict(heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim,
                                   kv_rank=self.kv_rank, q_rank=self.q_rank, scale=self.scale,
                                   rot=dict(base=self.base, dims=self.rot_dim))
        if self.kv_from is not None:
            raw["kv_from"] = self.kv_from
        return raw


@dataclass(frozen=True)
class UnitConfig:
    """A clamped gated feed-forward: the dense one, an expert, or the shared expert."""

    ff: int
    limit: float

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "UnitConfig":
        return cls(_count(raw, "ff", where), _positive(raw, "limit", where))

    def to_dict(self) -> dict[str, Any]:
        return dict(ff=self.ff, limit=self.limit)


@dataclass(frozen=True)
class UnitFeedForwardConfig:
    unit: UnitConfig                    # the dense one, or every expert
    experts: int = 0                    # 0: dense
    top: int = 0
    shared: UnitConfig | None = None

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "UnitFeedForwardConfig":
        kind = _get(raw, "kind", str, where)
        if kind == "dense":
            return cls(UnitConfig.from_dict(raw, where))
        if kind != "moe":
            raise ConfigError(f"config.json: {where}: feed-forward kind {kind!r} is not built (known: dense, moe)")
        router = _get(raw, "router", dict, where)
        experts, top = _count(router, "experts", where + ".router"), _count(router, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"config.json: {where}.router: 'top' ({top}) is more than 'experts' ({experts})")
        shared = raw.get("shared")
        return cls(UnitConfig.from_dict(_get(raw, "expert", dict, where), where + ".expert"), experts, top,
                   UnitConfig.from_dict(shared, where + ".shared") if shared is not None else None)

    def to_dict(self) -> dict[str, Any]:
        if not self.experts:
            return dict(kind="dense", **self.unit.to_dict())
        raw: dict[str, Any] = dict(kind="moe", expert=self.unit.to_dict(), router=dict(experts=self.experts, top=self.top))
        if self.shared is not None:
            raw["shared"] = self.shared.to_dict()
        return raw


@dataclass(frozen=True)
class BozevikLayerConfig:
    type: str
    mixer: SharedLatentConfig
    mlp: UnitFeedForwardConfig | None

    def to_dict(self) -> dict[str, Any]:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp is not None else None)


@dataclass(frozen=True)
class BozevikConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: tuple[BozevikLayerConfig, ...]
    architecture: str = "Bozevik"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "BozevikConfig":
        where = "Bozevik"
        eps = _number(_get(raw, "norm", dict, where), "eps", where + ".norm")
        if eps < 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {eps}")
        entries = _get(raw, "layers", list, where)
        if not entries:
            raise ConfigError("config.json: 'layers' is empty")
        layers: list[BozevikLayerConfig] = []
        for index, entry in enumerate(entries):
            here = f"layers[{index}]"
            kind = _get(entry, "type", str, here)
            if kind != "latent_attention":
                raise ConfigError(f"config.json: {here}: mixer type {kind!r} is not built (known: latent_attention)")
            mixer = SharedLatentConfig.from_dict(_get(entry, "mixer", dict, here), here + ".mixer")
            if mixer.kv_from is not None:
                owner = layers[mixer.kv_from].mixer if mixer.kv_from < index else None
                if (owner is None or owner.kv_from is not None
                        or (owner.kv_rank, owner.rot_dim, owner.base) != (mixer.kv_rank, mixer.rot_dim, mixer.base)):
                    raise ConfigError(
                        f"config.json: {here}: 'kv_from' must name an earlier layer that makes its own latent, with the "
                        f"same kv_rank, rot_dim and rotation; got {mixer.kv_from}")
            mlp = entry.get("mlp")
            layers.append(BozevikLayerConfig(
                kind, mixer, UnitFeedForwardConfig.from_dict(mlp, here + ".mlp") if mlp is not None else None))
        return cls(vocab=_count(raw, "vocab", where), width=_count(raw, "width", where), norm_eps=eps,
                   logit_scale=_number(raw, "logit_scale", where), layers=tuple(layers),
                   architecture=str(raw.get("architecture", "Bozevik")))

    def to_dict(self) -> dict[str, Any]:
        return dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                    logit_scale=self.logit_scale, layers=[layer.to_dict() for layer in self.layers])
