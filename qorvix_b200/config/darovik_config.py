"""Configuration of the Darovik decoder, read from its own config.json keys.

A Darovik model keeps its residual as several streams (`streams`) that every sublayer reads as a weighted sum and writes back to
(hyper-connections).  A layer is latent attention without positions and with a sink per head ('latent_attention') or
differential attention over a sliding window without positions ('attention'), then a feed-forward that is ungated with biases
('dense'), small gated experts behind a sigmoid router with groups ('moe'), or absent.  A stretch of layers may run several
times in a row with the same weights (`loop`).  config.json gives every size and constant layer by layer, so nothing about a
layer is assumed from another.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .deganex_config import _need, _positive_int
from .model_config import ConfigError, ModelConfig

MIXER_SIZES = {
    "latent_attention": ("heads", "dim", "vdim", "kv_rank"),
    "attention": ("heads", "kv_heads", "dim", "vdim"),
}
MIXER_CONSTANTS = {"latent_attention": ("scale",), "attention": ("scale", "diff")}
MLP_KINDS = ("dense", "moe")
MAX_STREAMS = 16                  # what the streams' kernel takes


@dataclass(frozen=True)
class DarovikConfig(ModelConfig):
    """Field names follow config.json; `layers` keeps each layer's entry as it is written there."""
    vocab_size: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    residual_mult: float = 1.0
    streams: int = 1
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times): layers start..stop-1 run `times` times
    layers: Tuple[dict, ...] = field(default_factory=tuple)

    @staticmethod
    def from_dict(d: dict) -> "DarovikConfig":
        layers = _need(d, "layers", "config")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        loop = None
        if d.get("loop") is not None:
            lp = d["loop"]
            loop = (int(_need(lp, "start", "loop")), int(_need(lp, "stop", "loop")), _positive_int(lp, "times", "loop"))
        cfg = DarovikConfig(
            architecture=str(d.get("architecture") or (d.get("architectures") or ["Darovik"])[0]),
            vocab_size=_positive_int(d, "vocab", "config"), width=_positive_int(d, "width", "config"),
            norm_eps=float(_need(_need(d, "norm", "config"), "eps", "norm")),
            residual_mult=float(d.get("residual_mult", 1.0)), streams=_positive_int(d, "streams", "config"), loop=loop,
            layers=tuple(copy.deepcopy(l) for l in layers), eos_token_id=d.get("eos_token_id"))
        cfg.validate()
        return cfg

    def run_order(self) -> List[int]:
        """The layers in execution order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def validate(self) -> None:
        if self.norm_eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if self.streams > MAX_STREAMS:
            raise ConfigError(f"config.json: streams {self.streams} is more than the {MAX_STREAMS} the kernel takes")
        if self.loop is not None:
            a, b, _ = self.loop
            if not 0 <= a < b <= len(self.layers):
                raise ConfigError(f"config.json: loop.start {a} and loop.stop {b} name no stretch of the {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXER_SIZES:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not a known mixer (known: {', '.join(MIXER_SIZES)})")
            m = _need(layer, "mixer", where)
            for key in MIXER_SIZES[kind]:
                _positive_int(m, key, where + ".mixer")
            for key in MIXER_CONSTANTS[kind]:
                _need(m, key, where + ".mixer")
            if kind == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"config.json: {where}.mixer.heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
                if m.get("mask") is not None:
                    _positive_int(m["mask"], "size", where + ".mixer.mask")
            self._validate_mlp(layer.get("mlp"), where + ".mlp")

    @staticmethod
    def _validate_mlp(f, where: str) -> None:
        if f is None:
            return
        kind = _need(f, "kind", where)
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}.kind '{kind}' is not known (known: {', '.join(MLP_KINDS)})")
        if kind == "dense":
            _positive_int(f, "ff", where)
            return
        _positive_int(_need(f, "expert", where), "ff", where + ".expert")
        r = _need(f, "router", where)
        experts, top = _positive_int(r, "experts", where + ".router"), _positive_int(r, "top", where + ".router")
        _need(r, "scale", where + ".router")
        count = keep = 1
        if r.get("groups") is not None:
            count, keep = (_positive_int(r["groups"], key, where + ".router.groups") for key in ("count", "keep"))
        if experts % count:
            raise ConfigError(f"config.json: {where}.router.groups.count {count} does not divide the {experts} experts")
        if keep > count:
            raise ConfigError(f"config.json: {where}.router.groups.keep {keep} is more than the {count} groups")
        if top > keep * (experts // count):
            raise ConfigError(f"config.json: {where}.router.top {top} is more than the {keep * (experts // count)} experts of the kept groups")

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "streams": self.streams,
                             "layers": [copy.deepcopy(l) for l in self.layers]}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
