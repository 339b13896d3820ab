"""The typed configuration of the Zivazen design, read from config.json's own keys.

A Zivazen config.json names the design under `architecture` and gives `vocab`, `width`, `norm.eps` and `layers`. A layer
entry has `type` ("attention" or "parallel"), the mixer's sizes and constants under `mixer` and the feed-forward under
`mlp` (null for a layer without one). An attention mixer has `heads`, `kv_heads`, `dim`, `vdim`, `scale`, optionally `rot`
(`base`, `dims`, optionally `scaling` with `factor`, `low`, `high`, `original`), optionally `mask` (`size`: chunks of that
many positions) and optionally `v_mix` (true: the layer's values are mixed with those of the first such layer). A parallel
mixer has `left` (an attention's keys without `v_mix`; `mask.size` is a window), `right` (`heads`, `vdim`, `state`,
`groups`, `conv`, `norm_groups`), `left_scale` and `right_scale`. A feed-forward of kind "dense" has `ff`; of kind "moe"
`expert.ff`, `router` (`experts`, `top`, `scale`, optionally `groups` with `count` and `keep`) and optionally `shared.ff`.
Nothing here is a size of a particular model."""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from .registry import ConfigError

MIXER_TYPES = ("attention", "parallel")
MLP_KINDS = ("dense", "moe")
DEFAULT_MAX_POSITION = 32768
"""The design has no longest sequence; this bounds the cache unless `max_position` is given."""


def _need(where: str, mapping: Any, keys) -> None:
    if not isinstance(mapping, Mapping):
        raise ConfigError(f"{where} must be an object")
    missing = [k for k in keys if k not in mapping]
    if missing:
        raise ConfigError(f"{where} has no {', '.join(missing)}")


def _positive(where: str, mapping: Mapping, keys) -> None:
    for key in keys:
        if not isinstance(mapping[key], int) or isinstance(mapping[key], bool) or mapping[key] <= 0:
            raise ConfigError(f"{where}.{key} must be a positive integer, not {mapping[key]!r}")


def _check_rotation(where: str, rot: Any, dim: int) -> None:
    _need(where, rot, ("base", "dims"))
    dims = rot["dims"]
    if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{where}.dims must be even and at most dim, not {dims!r}")
    if dims and not float(rot["base"]) > 0:
        raise ConfigError(f"{where}.base must be positive")
    scaling = rot.get("scaling")
    if scaling is not None:
        keys = ("factor", "low", "high", "original")
        _need(f"{where}.scaling", scaling, keys)
        if not all(float(scaling[key]) > 0 for key in keys) or not float(scaling["high"]) > float(scaling["low"]):
            raise ConfigError(f"{where}.scaling: factor, low, high and original must be positive and high above low")


def _check_attention(where: str, mixer: Any) -> None:
    _need(where, mixer, ("heads", "kv_heads", "dim", "vdim", "scale"))
    _positive(where, mixer, ("heads", "kv_heads", "dim", "vdim"))
    if mixer["heads"] % mixer["kv_heads"]:
        raise ConfigError(f"{where}: {mixer['heads']} heads are not a multiple of {mixer['kv_heads']} kv_heads")
    if not float(mixer["scale"]) > 0:
        raise ConfigError(f"{where}.scale must be positive")
    if mixer.get("rot") is not None:
        _check_rotation(f"{where}.rot", mixer["rot"], mixer["dim"])
    if mixer.get("mask") is not None:
        _need(f"{where}.mask", mixer["mask"], ("size",))
        _positive(f"{where}.mask", mixer["mask"], ("size",))


def _check_parallel(where: str, mixer: Any) -> None:
    _need(where, mixer, ("left", "right", "left_scale", "right_scale"))
    _check_attention(f"{where}.left", mixer["left"])
    right, keys = mixer["right"], ("heads", "vdim", "state", "groups", "conv", "norm_groups")
    _need(f"{where}.right", right, keys)
    _positive(f"{where}.right", right, keys)
    if right["heads"] % right["groups"]:
        raise ConfigError(f"{where}.right: {right['heads']} heads are not a multiple of {right['groups']} groups")
    if right["heads"] * right["vdim"] % right["norm_groups"]:
        raise ConfigError(f"{where}.right: heads x vdim is not a multiple of {right['norm_groups']} norm_groups")


def _check_mlp(where: str, mlp: Any) -> None:
    _need(where, mlp, ("kind",))
    if mlp["kind"] not in MLP_KINDS:
        raise ConfigError(f"{where}.kind {mlp['kind']!r} is not supported (supported: {', '.join(MLP_KINDS)})")
    if mlp["kind"] == "dense":
        _need(where, mlp, ("ff",))
        _positive(where, mlp, ("ff",))
        return
    _need(where, mlp, ("expert", "router"))
    _need(f"{where}.expert", mlp["expert"], ("ff",))
    _positive(f"{where}.expert", mlp["expert"], ("ff",))
    router = mlp["router"]
    _need(f"{where}.router", router, ("experts", "top", "scale"))
    _positive(f"{where}.router", router, ("experts", "top"))
    open_experts = router["experts"]
    if router.get("groups") is not None:
        groups = router["groups"]
        _need(f"{where}.router.groups", groups, ("count", "keep"))
        _positive(f"{where}.router.groups", groups, ("count", "keep"))
        if router["experts"] % groups["count"] or groups["keep"] > groups["count"]:
            raise ConfigError(f"{where}.router.groups: the best {groups['keep']} of {groups['count']} groups of "
                              f"{router['experts']} experts")
        open_experts = groups["keep"] * (router["experts"] // groups["count"])
    if router["top"] > open_experts:
        raise ConfigError(f"{where}.router: top {router['top']} of {open_experts} experts")
    if mlp.get("shared") is not None:
        _need(f"{where}.shared", mlp["shared"], ("ff",))
        _positive(f"{where}.shared", mlp["shared"], ("ff",))


def mixes_values(layer: Mapping) -> bool:
    return layer["type"] == "attention" and bool(layer["mixer"].get("v_mix"))


def _check_layers(layers) -> None:
    mixing = None
    for index, layer in enumerate(layers):
        where = f"layers[{index}]"
        _need(where, layer, ("type", "mixer"))
        if layer["type"] not in MIXER_TYPES:
            raise ConfigError(f"{where}.type {layer['type']!r} is not supported (supported: {', '.join(MIXER_TYPES)})")
        (_check_attention if layer["type"] == "attention" else _check_parallel)(f"{where}.mixer", layer["mixer"])
        if layer.get("mlp") is not None:
            _check_mlp(f"{where}.mlp", layer["mlp"])
        if mixes_values(layer):
            size = layer["mixer"]["kv_heads"] * layer["mixer"]["vdim"]
            if mixing is not None and mixing != (layer["mixer"]["kv_heads"], layer["mixer"]["vdim"]):
                raise ConfigError(f"{where}.mixer: {size} values a token cannot be mixed with the first layer's "
                                  f"{mixing[0] * mixing[1]} (kv_heads and vdim must be equal)")
            mixing = (layer["mixer"]["kv_heads"], layer["mixer"]["vdim"])


@dataclass(frozen=True)
class ZivazenConfig:
    model_type = "Zivazen"

    vocab: int
    width: int
    norm_eps: float
    layers: tuple = field(default_factory=tuple)
    """The layer entries as config.json gives them (checked)."""
    max_position: int = DEFAULT_MAX_POSITION
    eos_token_ids: tuple[int, ...] = field(default_factory=tuple)

    def __post_init__(self) -> None:
        for name in ("vocab", "width", "max_position"):
            if int(getattr(self, name)) <= 0:
                raise ConfigError(f"{name} must be positive, not {getattr(self, name)}")
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, not {self.norm_eps}")
        if not self.layers:
            raise ConfigError("layers is empty")
        _check_layers(self.layers)

    @classmethod
    def from_hf(cls, config: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "ZivazenConfig":
        if config.get("architecture") != "Zivazen":
            raise ConfigError(f"architecture {config.get('architecture')!r} is not 'Zivazen'")
        _need("config.json", config, ("vocab", "width", "norm", "layers"))
        _need("norm", config["norm"], ("eps",))
        if not isinstance(config["layers"], (list, tuple)):
            raise ConfigError("layers must be a list")
        eos = config.get("eos_token_id")
        eos = [] if eos is None else ([int(t) for t in eos] if isinstance(eos, (list, tuple)) else [int(eos)])
        return cls(
            vocab=int(config["vocab"]), width=int(config["width"]), norm_eps=float(config["norm"]["eps"]),
            layers=tuple(copy.deepcopy(layer) for layer in config["layers"]),
            max_position=int(config.get("max_position", DEFAULT_MAX_POSITION)),
            eos_token_ids=tuple(eos),
        )

    def to_hf(self) -> dict:
        """The config.json that reads back as this configuration."""
        out: dict[str, Any] = {"architecture": "Zivazen", "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "layers": [copy.deepcopy(layer) for layer in self.layers]}
        if self.max_position != DEFAULT_MAX_POSITION:
            out["max_position"] = self.max_position
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
