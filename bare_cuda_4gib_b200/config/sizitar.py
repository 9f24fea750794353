"""Typed configuration of the Sizitar decoder, read from its own `config.json` layout:

    architecture, vocab, width, norm.eps, logit_scale, loop: {start, stop, times} | null,
    layers: [{type: "delta" | "channel_delta" | "attention", mixer: {...}, mlp: {...} | null}, ...]

    delta, channel_delta mixer:  heads, kv_heads, dim, vdim, conv (, rank: of channel_delta's low-rank projections,
                                 needed for random weights only; a weight file's own shapes say it)
    attention mixer:             heads, kv_heads, dim, vdim, conv, scale, rot.{dims, base}
    mlp:                         kind "dense", ff; or kind "moe", expert.ff, router.{experts, top}, shared.ff

Layers loop.start .. loop.stop - 1 run loop.times times in a row with the same tensors, each run with a
cache or state of its own.  Every size and every constant that may differ between models of the design is
read here and nowhere else; a key that is wrong or missing is named in the error.  The design states no
largest position: a request is as long as the cache pool lets it be.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..errors import ConfigError
from .dopudra import _get

MIXER_TYPES = ("delta", "channel_delta", "attention")


def _mixer(m, where: str, kind: str) -> None:
    heads, kv = _get(m, "heads", where), _get(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: '{where}heads' {heads} is not a multiple of '{where}kv_heads' {kv}")
    dim = _get(m, "dim", where)
    _get(m, "vdim", where)
    _get(m, "conv", where)
    if m.get("rank") is not None:
        _get(m, "rank", where)
    if kind != "attention":
        return
    _get(m, "scale", where, float)
    rot = m.get("rot")
    dims = _get(rot, "dims", where + "rot.")
    _get(rot, "base", where + "rot.", float)
    if dims % 2:
        raise ConfigError(f"config.json: '{where}rot.dims' must be even (entries are turned in pairs), got {dims}")
    if dims > dim:
        raise ConfigError(f"config.json: '{where}rot.dims' {dims} exceeds '{where}dim' {dim}")


def _mlp(mlp, where: str) -> None:
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        _get(mlp, "ff", where)
    elif kind == "moe":
        _get(mlp.get("expert"), "ff", where + "expert.")
        r = mlp.get("router")
        experts, top = _get(r, "experts", where + "router."), _get(r, "top", where + "router.")
        if top > experts:
            raise ConfigError(f"config.json: '{where}router.top' {top} exceeds the {experts} experts that can be chosen")
        if mlp.get("shared") is not None:
            _get(mlp["shared"], "ff", where + "shared.")
    else:
        raise ConfigError(f"config.json: '{where}kind' must be 'dense' or 'moe' (or 'mlp' null)")


@dataclass
class SizitarConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]] = field(default_factory=list)
    loop: Optional[Dict[str, int]] = None
    logit_scale: float = 1.0
    norm_eps: float = 1e-6

    ARCHITECTURE = "Sizitar"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SizitarConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        cfg = cls(vocab=_get(d, "vocab", ""), width=_get(d, "width", ""), layers=copy.deepcopy(layers),
                  loop=copy.deepcopy(d.get("loop")), logit_scale=_get(d, "logit_scale", "", float),
                  norm_eps=_get(d.get("norm"), "eps", "norm.", float))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{where}type' must be one of {list(MIXER_TYPES)}, "
                                  f"got {layer.get('type') if isinstance(layer, dict) else layer!r}")
            if not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"config.json: required key '{where}mixer' is missing")
            _mixer(layer["mixer"], where + "mixer.", layer["type"])
            if layer.get("mlp") is not None:
                _mlp(layer["mlp"], where + "mlp.")
        if self.loop is not None:
            for key in ("start", "stop", "times"):
                v = self.loop.get(key) if isinstance(self.loop, dict) else None
                if isinstance(v, bool) or not isinstance(v, int) or v < 0:
                    raise ConfigError(f"config.json: 'loop.{key}' must be a count, got {v!r}")
            if not self.loop["start"] <= self.loop["stop"] <= len(self.layers):
                raise ConfigError(f"config.json: 'loop' names layers {self.loop['start']} to {self.loop['stop']}, "
                                  f"the model has {len(self.layers)}")
            if self.loop["times"] < 1:
                raise ConfigError(f"config.json: 'loop.times' must be at least 1, got {self.loop['times']}")

    def run_order(self) -> List[int]:
        """The layers in the order in which they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def to_dict(self) -> Dict[str, Any]:
        """The config.json this configuration is read back from."""
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "loop": copy.deepcopy(self.loop),
                "layers": copy.deepcopy(self.layers)}

    # the names the command line tools read from any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def stop_ids(self) -> List[int]:
        return []
