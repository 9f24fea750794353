"""Typed configuration of the Fuzazen decoder, read from its own `config.json` layout:

    architecture, vocab, width, embedding.scale, norm.eps, residual_mult, logit_softcap (null: no cap),
    layers: [{type: "attention", mixer: {...}, mlp: {kind: "dense", ff} | null, weights_of: j (optional)}, ...]

    attention mixer:  heads, kv_heads, dim, vdim, scale, mask.size, rot.{dims, base}

A layer with `weights_of` j runs with layer j's tensors and keeps a cache of its own; the rest of its
entry equals layer j's.  Every size and every constant that may differ between models of the design is
read here and nowhere else; a key that is wrong or missing is named in the error.  The design states no
largest position: a request is as long as the cache pool lets it be.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..errors import ConfigError
from .dopudra import _get

MIXER_TYPES = ("attention",)


def _attention(m, where: str) -> None:
    heads, kv = _get(m, "heads", where), _get(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: '{where}heads' {heads} is not a multiple of '{where}kv_heads' {kv}")
    dim = _get(m, "dim", where)
    _get(m, "vdim", where)
    _get(m, "scale", where, float)
    _get(m.get("mask"), "size", where + "mask.")
    rot = m.get("rot")
    dims = _get(rot, "dims", where + "rot.")
    _get(rot, "base", where + "rot.", float)
    if dims % 2:
        raise ConfigError(f"config.json: '{where}rot.dims' must be even (entries are turned in pairs), got {dims}")
    if dims > dim:
        raise ConfigError(f"config.json: '{where}rot.dims' {dims} exceeds '{where}dim' {dim}")


@dataclass
class FuzazenConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]] = field(default_factory=list)
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_softcap: Optional[float] = None
    norm_eps: float = 1e-6

    ARCHITECTURE = "Fuzazen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "FuzazenConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        if "logit_softcap" not in d:
            raise ConfigError("config.json: required key 'logit_softcap' is missing (null: no cap)")
        cap = None if d["logit_softcap"] is None else _get(d, "logit_softcap", "", float)
        cfg = cls(vocab=_get(d, "vocab", ""), width=_get(d, "width", ""), layers=copy.deepcopy(layers),
                  embedding_scale=_get(d.get("embedding"), "scale", "embedding.", float),
                  residual_mult=_get(d, "residual_mult", "", float), logit_softcap=cap,
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
            _attention(layer["mixer"], where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: '{where}mlp.kind' must be 'dense' (or 'mlp' null)")
                _get(mlp, "ff", where + "mlp.")
        for i in range(len(self.layers)):
            self.source(i)

    def source(self, i: int) -> int:
        """The layer whose tensors layer i runs with: itself, or the one its `weights_of` leads to."""
        start, seen = i, {i}
        while self.layers[i].get("weights_of") is not None:
            src = self.layers[i]["weights_of"]
            where = f"layers[{i}]."
            if isinstance(src, bool) or not isinstance(src, int) or not (0 <= src < len(self.layers)):
                raise ConfigError(f"config.json: '{where}weights_of' must name another layer, got {src!r}")
            if src in seen:
                raise ConfigError(f"config.json: '{where}weights_of' leads back to layer {src}: no layer of the chain has tensors")
            for key in ("type", "mixer", "mlp"):
                if self.layers[src].get(key) != self.layers[start].get(key):
                    raise ConfigError(f"config.json: 'layers[{start}].{key}' differs from layer {src}, whose tensors it uses")
            seen.add(src)
            i = src
        return i

    def to_dict(self) -> Dict[str, Any]:
        """The config.json this configuration is read back from."""
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap, "layers": copy.deepcopy(self.layers)}

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
