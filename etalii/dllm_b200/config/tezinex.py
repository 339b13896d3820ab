"""The typed configuration of the Tezinex design, read from config.json's own keys.

A Tezinex config.json names the design under `architecture` and gives `vocab`, `width`, `norm.eps`, `residual_mult`,
optionally `logit_softcap`, and `layers`. A layer entry has `type` ("channel_delta" or "attention"), the mixer's sizes
and constants under `mixer` and the feed-forward under `mlp` (kind "dense" with `ff`, or null for a layer without one).
A channel_delta mixer has `heads`, `kv_heads`, `dim`, `vdim` and `conv`; an attention mixer `heads`, `kv_heads`, `dim`,
`vdim`, `scale`, optionally `softcap`, optionally `mask` (`size` and optionally `keep_first`) and optionally `kv_from`:
the layer whose keys and values this one reads instead of projecting its own. The inner sizes of a channel_delta
mixer's low-rank projections are those of its tensors. Nothing here is a size of a particular model."""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from .registry import ConfigError

MIXER_TYPES = ("channel_delta", "attention")
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


def _check_mixer(where: str, kind: str, mixer: Any) -> None:
    _need(where, mixer, ("heads", "kv_heads", "dim", "vdim", *(("conv",) if kind == "channel_delta" else ("scale",))))
    _positive(where, mixer, ("heads", "kv_heads", "dim", "vdim"))
    if mixer["heads"] % mixer["kv_heads"]:
        raise ConfigError(f"{where}: {mixer['heads']} heads are not a multiple of {mixer['kv_heads']} kv_heads")
    if kind == "channel_delta":
        _positive(where, mixer, ("conv",))
        return
    if not float(mixer["scale"]) > 0:
        raise ConfigError(f"{where}.scale must be positive")
    if mixer.get("softcap") is not None and not float(mixer["softcap"]) > 0:
        raise ConfigError(f"{where}.softcap must be positive")
    if mixer.get("mask") is not None:
        _need(f"{where}.mask", mixer["mask"], ("size",))
        _positive(f"{where}.mask", mixer["mask"], ("size",))
        keep = mixer["mask"].get("keep_first", 0)
        if not isinstance(keep, int) or isinstance(keep, bool) or keep < 0:
            raise ConfigError(f"{where}.mask.keep_first must be an integer and not negative, not {keep!r}")


def _check_layers(layers) -> None:
    for index, layer in enumerate(layers):
        where = f"layers[{index}]"
        _need(where, layer, ("type", "mixer"))
        if layer["type"] not in MIXER_TYPES:
            raise ConfigError(f"{where}.type {layer['type']!r} is not supported (supported: {', '.join(MIXER_TYPES)})")
        _check_mixer(f"{where}.mixer", layer["type"], layer["mixer"])
        mlp = layer.get("mlp")
        if mlp is not None:
            _need(f"{where}.mlp", mlp, ("kind", "ff"))
            if mlp["kind"] != "dense":
                raise ConfigError(f"{where}.mlp.kind {mlp['kind']!r} is not supported (supported: dense)")
            _positive(f"{where}.mlp", mlp, ("ff",))
    for index, layer in enumerate(layers):
        source = layer["mixer"].get("kv_from")
        if source is None:
            continue
        where = f"layers[{index}].mixer.kv_from"
        if not isinstance(source, int) or isinstance(source, bool) or not 0 <= source < index:
            raise ConfigError(f"{where} must name an earlier layer, not {source!r}")
        if layer["type"] != "attention" or layers[source]["type"] != "attention":
            raise ConfigError(f"{where}: keys and values are shared between attention layers only")
        other, own = layers[source]["mixer"], layer["mixer"]
        if other.get("kv_from") is not None:
            raise ConfigError(f"{where}: layer {source} has no keys and values of its own")
        for key in ("kv_heads", "dim", "vdim"):
            if other[key] != own[key]:
                raise ConfigError(f"{where}: layer {source}'s {key} ({other[key]!r}) differs from this layer's "
                                  f"({own[key]!r})")


@dataclass(frozen=True)
class TezinexConfig:
    model_type = "Tezinex"

    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: float | None = None
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
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError(f"logit_softcap must be positive, not {self.logit_softcap}")
        if not self.layers:
            raise ConfigError("layers is empty")
        _check_layers(self.layers)

    @classmethod
    def from_hf(cls, config: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "TezinexConfig":
        if config.get("architecture") != "Tezinex":
            raise ConfigError(f"architecture {config.get('architecture')!r} is not 'Tezinex'")
        _need("config.json", config, ("vocab", "width", "norm", "residual_mult", "layers"))
        _need("norm", config["norm"], ("eps",))
        if not isinstance(config["layers"], (list, tuple)):
            raise ConfigError("layers must be a list")
        eos = config.get("eos_token_id")
        eos = [] if eos is None else ([int(t) for t in eos] if isinstance(eos, (list, tuple)) else [int(eos)])
        softcap = config.get("logit_softcap")
        return cls(
            vocab=int(config["vocab"]), width=int(config["width"]), norm_eps=float(config["norm"]["eps"]),
            residual_mult=float(config["residual_mult"]), logit_softcap=None if softcap is None else float(softcap),
            layers=tuple(copy.deepcopy(layer) for layer in config["layers"]),
            max_position=int(config.get("max_position", DEFAULT_MAX_POSITION)),
            eos_token_ids=tuple(eos),
        )

    def to_hf(self) -> dict:
        """The config.json that reads back as this configuration."""
        out: dict[str, Any] = {
            "architecture": "Tezinex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult, "layers": [copy.deepcopy(layer) for layer in self.layers],
        }
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.max_position != DEFAULT_MAX_POSITION:
            out["max_position"] = self.max_position
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
