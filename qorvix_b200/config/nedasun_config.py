"""Configuration of the Nedasun decoder, read from its own config.json keys.

A Nedasun model is a list of layers with a norm on both sides of every sublayer: x += norm1b(mixer(norm1(x))), x +=
norm2b(ff(norm2(x))).  The mixer is rotary grouped-query attention with soft-capped scores, a sink per head and mixed heads
('attention', optionally blending its values with those of the first such layer) or a delta rule with one decay per head
('delta'); the feed-forward is a clamped gated one ('dense'), routed experts with identity experts and a shared one
('moe'), or absent.  config.json gives every size and constant layer by layer, so nothing about a layer is assumed from
another.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, Tuple

from .deganex_config import _need, _positive_int
from .model_config import ConfigError, ModelConfig

MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "rot"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}
MIXER_SIZES = {
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}
MLP_KINDS = ("dense", "moe")


def _positive_number(d: dict, key: str, where: str) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not v > 0:
        raise ConfigError(f"config.json: {where}.{key} must be a positive number, not {v!r}")
    return float(v)


@dataclass(frozen=True)
class NedasunConfig(ModelConfig):
    """Field names follow config.json; `layers` keeps each layer's entry as it is written there."""
    vocab_size: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    layers: Tuple[dict, ...] = field(default_factory=tuple)

    @staticmethod
    def from_dict(d: dict) -> "NedasunConfig":
        layers = _need(d, "layers", "config")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        cfg = NedasunConfig(
            architecture=str(d.get("architecture") or (d.get("architectures") or ["Nedasun"])[0]),
            vocab_size=_positive_int(d, "vocab", "config"), width=_positive_int(d, "width", "config"),
            norm_eps=float(_need(_need(d, "norm", "config"), "eps", "norm")),
            layers=tuple(copy.deepcopy(l) for l in layers), eos_token_id=d.get("eos_token_id"))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.norm_eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXER_KEYS:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not a known mixer (known: {', '.join(MIXER_KEYS)})")
            m = _need(layer, "mixer", where)
            for key in MIXER_KEYS[kind]:
                _need(m, key, where + ".mixer")
            for key in MIXER_SIZES[kind]:
                _positive_int(m, key, where + ".mixer")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"config.json: {where}.mixer.heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
            if kind == "attention":
                dims = _need(m["rot"], "dims", where + ".mixer.rot")
                _need(m["rot"], "base", where + ".mixer.rot")
                if not isinstance(dims, int) or dims < 0 or dims % 2 or dims > m["dim"]:
                    raise ConfigError(f"config.json: {where}.mixer.rot.dims {dims!r} must be even and at most {m['dim']}")
                if m.get("softcap") is not None:
                    _positive_number(m, "softcap", where + ".mixer")
            elif m["conv"] > 16:
                raise ConfigError(f"config.json: {where}.mixer.conv {m['conv']} is more than the 16 taps the convolution kernel takes")
            elif m["dim"] > 256:
                raise ConfigError(f"config.json: {where}.mixer.dim {m['dim']} is more than the 256 key entries the recurrence's kernel takes")
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
            _positive_number(f, "limit", where)
            return
        for part in ("expert",) + (("shared",) if f.get("shared") is not None else ()):
            e = _need(f, part, where)
            _positive_int(e, "ff", f"{where}.{part}")
            _positive_number(e, "limit", f"{where}.{part}")
        r = _need(f, "router", where)
        experts, top = _positive_int(r, "experts", where + ".router"), _positive_int(r, "top", where + ".router")
        _need(r, "scale", where + ".router")
        identity = r.get("identity", 0) or 0
        if not isinstance(identity, int) or identity < 0:
            raise ConfigError(f"config.json: {where}.router.identity must be a number of experts, not {identity!r}")
        if top > experts + identity:
            raise ConfigError(f"config.json: {where}.router.top {top} is more than its {experts + identity} experts")

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                             "norm": {"eps": self.norm_eps}, "layers": [copy.deepcopy(l) for l in self.layers]}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
