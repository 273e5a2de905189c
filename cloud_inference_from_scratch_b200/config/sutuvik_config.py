"""Typed configuration of the Sutuvik decoder, read from config.json keys.

A Sutuvik model is a list of pre-norm layers (RMS norms in groups) with a short convolution in front of every mixer, an
optional feed-forward of routed experts and a side input of the tokens after it.  config.json carries:

* ``architecture`` "Sutuvik", ``vocab``, ``width``, ``logit_scale``, ``norm`` (``eps``, ``groups``), ``canon.taps`` (the
  convolution in front of the mixers), ``token_side.dim``;
* ``layers``: per layer ``type`` ("mamba2", "attention" or "attention_2"), ``mixer`` (its sizes and constants) and
  ``mlp`` (null, or ``kind`` "moe" with ``expert.ff``, ``router.experts``, ``router.top`` and ``router.groups`` with
  ``count`` and ``keep``).

Mixer "attention": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``q_temp`` (``coef``, ``every``), ``v_mix``.
Mixer "attention_2": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap``, ``rot`` (``base``, ``dims``,
``scaling`` with ``factor``, ``low``, ``high``, ``original``), ``v_mix``.  Mixer "mamba2": ``heads``, ``vdim``, ``state``,
``groups``, ``conv`` (taps), ``norm_groups``.

Every size and constant comes from here; this module is the only place that knows the key names.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .lazilorn_config import _number
from .model_config import ConfigError
from .zisesun_config import _count, _get


def _heads(raw: dict[str, Any], where: str) -> dict[str, Any]:
    heads, kv_heads = _count(raw, "heads", where), _count(raw, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    return dict(heads=heads, kv_heads=kv_heads, dim=_count(raw, "dim", where), vdim=_count(raw, "vdim", where),
                scale=_number(raw, "scale", where), v_mix=bool(raw.get("v_mix", False)))


@dataclass(frozen=True)
class BandedRotationConfig:
    base: float
    dims: int                                                  # rotated elements of a head
    scaling: tuple[float, float, float, float] | None          # factor, low, high, original

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str, head: int) -> "BandedRotationConfig":
        base, dims = _number(raw, "base", where), _count(raw, "dims", where)
        if not base > 1:
            raise ConfigError(f"config.json: {where}: 'base' must be above 1, got {base}")
        if dims % 2 or dims > head:
            raise ConfigError(f"config.json: {where}: 'dims' must be even and within a head of {head}, got {dims}")
        scaling = raw.get("scaling")
        if scaling is not None:
            here = where + ".scaling"
            scaling = tuple(_number(scaling, key, here) for key in ("factor", "low", "high", "original"))
            if min(scaling) <= 0 or scaling[1] > scaling[2]:
                raise ConfigError(f"config.json: {here}: all positive and 'low' not above 'high', got {scaling}")
        return cls(base, dims, scaling)

    def to_dict(self) -> dict[str, Any]:
        raw: dict[str, Any] = dict(base=self.base, dims=self.dims)
        if self.scaling is not None:
            raw["scaling"] = dict(zip(("factor", "low", "high", "original"), self.scaling))
        return raw


@dataclass(frozen=True)
class BiasedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int            # size of a query / key head
    vdim: int           # size of a value head
    scale: float
    v_mix: bool
    heat: tuple[float, int] | None      # coef, every

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "BiasedAttentionConfig":
        heat = raw.get("q_temp")
        if heat is not None:
            heat = (_number(heat, "coef", where + ".q_temp"), _count(heat, "every", where + ".q_temp"))
        return cls(heat=heat, **_heads(raw, where))

    def to_dict(self) -> dict[str, Any]:
        raw: dict[str, Any] = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                                   scale=self.scale, v_mix=self.v_mix)
        if self.heat is not None:
            raw["q_temp"] = dict(coef=self.heat[0], every=self.heat[1])
        return raw


@dataclass(frozen=True)
class RotatedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool
    softcap: float
    rot: BandedRotationConfig

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "RotatedAttentionConfig":
        sizes = _heads(raw, where)
        softcap = _number(raw, "softcap", where)
        if not softcap > 0:
            raise ConfigError(f"config.json: {where}: 'softcap' must be positive, got {softcap}")
        return cls(softcap=softcap, rot=BandedRotationConfig.from_dict(_get(raw, "rot", dict, where), where + ".rot", sizes["dim"]),
                   **sizes)

    def to_dict(self) -> dict[str, Any]:
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale,
                    v_mix=self.v_mix, softcap=self.softcap, rot=self.rot.to_dict())


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int           # taps
    norm_groups: int

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "Mamba2Config":
        sizes = {key: _count(raw, key, where) for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}
        if sizes["heads"] % sizes["groups"]:
            raise ConfigError(f"config.json: {where}: 'heads' ({sizes['heads']}) must be a multiple of 'groups' ({sizes['groups']})")
        if sizes["heads"] * sizes["vdim"] % sizes["norm_groups"]:
            raise ConfigError(f"config.json: {where}: 'norm_groups' ({sizes['norm_groups']}) must divide heads * vdim")
        return cls(**sizes)

    def to_dict(self) -> dict[str, Any]:
        return dict(heads=self.heads, vdim=self.vdim, state=self.state, groups=self.groups, conv=self.conv,
                    norm_groups=self.norm_groups)


@dataclass(frozen=True)
class RoutedConfig:
    ff: int
    experts: int
    top: int
    groups: int         # equal groups of neighbouring experts
    keep: int           # groups that experts are chosen from

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "RoutedConfig":
        kind = _get(raw, "kind", str, where)
        if kind != "moe":
            raise ConfigError(f"config.json: {where}: feed-forward kind {kind!r} is not built (known: moe)")
        here = where + ".router"
        router = _get(raw, "router", dict, where)
        experts, top = _count(router, "experts", here), _count(router, "top", here)
        groups, keep = 1, 1
        if router.get("groups") is not None:
            groups, keep = (_count(router["groups"], key, here + ".groups") for key in ("count", "keep"))
        if experts % groups or keep > groups:
            raise ConfigError(f"config.json: {here}.groups: {keep} of {groups} equal groups of {experts} experts")
        if top > experts // groups * keep:
            raise ConfigError(f"config.json: {here}: 'top' ({top}) is more than the {experts // groups * keep} experts to choose from")
        return cls(_count(_get(raw, "expert", dict, where), "ff", where + ".expert"), experts, top, groups, keep)

    def to_dict(self) -> dict[str, Any]:
        return dict(kind="moe", expert=dict(ff=self.ff),
                    router=dict(experts=self.experts, top=self.top, groups=dict(count=self.groups, keep=self.keep)))


MIXERS = {"mamba2": Mamba2Config, "attention": BiasedAttentionConfig, "attention_2": RotatedAttentionConfig}


@dataclass(frozen=True)
class SutuvikLayerConfig:
    type: str
    mixer: Mamba2Config | BiasedAttentionConfig | RotatedAttentionConfig
    mlp: RoutedConfig | None

    def to_dict(self) -> dict[str, Any]:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp is not None else None)


@dataclass(frozen=True)
class SutuvikConfig:
    vocab: int
    width: int
    logit_scale: float
    norm_eps: float
    norm_groups: int
    canon_taps: int
    side_dim: int
    layers: tuple[SutuvikLayerConfig, ...]
    architecture: str = "Sutuvik"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "SutuvikConfig":
        where = "Sutuvik"
        norm = _get(raw, "norm", dict, where)
        eps, groups = _number(norm, "eps", where + ".norm"), _count(norm, "groups", where + ".norm")
        width = _count(raw, "width", where)
        if eps < 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {eps}")
        if width % groups:
            raise ConfigError(f"config.json: norm.groups ({groups}) must divide 'width' ({width})")
        entries = _get(raw, "layers", list, where)
        if not entries:
            raise ConfigError("config.json: 'layers' is empty")
        layers: list[SutuvikLayerConfig] = []
        mixed: set[int] = set()
        for index, entry in enumerate(entries):
            here = f"layers[{index}]"
            kind = _get(entry, "type", str, here)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {here}: mixer type {kind!r} is not built (known: {sorted(MIXERS)})")
            mixer = MIXERS[kind].from_dict(_get(entry, "mixer", dict, here), here + ".mixer")
            if getattr(mixer, "v_mix", False):
                mixed.add(mixer.kv_heads * mixer.vdim)
            mlp = entry.get("mlp")
            layers.append(SutuvikLayerConfig(
                kind, mixer, RoutedConfig.from_dict(mlp, here + ".mlp") if mlp is not None else None))
        if len(mixed) > 1:
            raise ConfigError(f"config.json: layers with 'v_mix' must agree about kv_heads * vdim, got {sorted(mixed)}")
        return cls(vocab=_count(raw, "vocab", where), width=width,
                   logit_scale=_number(raw, "logit_scale", where) if "logit_scale" in raw else 1.0, norm_eps=eps,
                   norm_groups=groups, canon_taps=_count(_get(raw, "canon", dict, where), "taps", where + ".canon"),
                   side_dim=_count(_get(raw, "token_side", dict, where), "dim", where + ".token_side"),
                   layers=tuple(layers), architecture=str(raw.get("architecture", "Sutuvik")))

    def to_dict(self) -> dict[str, Any]:
        return dict(architecture=self.architecture, vocab=self.vocab, width=self.width, logit_scale=self.logit_scale,
                    norm=dict(eps=self.norm_eps, groups=self.norm_groups), canon=dict(taps=self.canon_taps),
                    token_side=dict(dim=self.side_dim), layers=[layer.to_dict() for layer in self.layers])
