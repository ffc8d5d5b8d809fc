"""Typed configuration of the Vivepel decoder, read from its config.json.

The file gives ``width``, ``vocab``, ``norm`` (``eps``, ``groups``) and ``layers``. A layer names its mixer (``type``: "attention"),
the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: an object of kind "dense", or null for a layer without
one). Every size and constant is taken from the file; nothing is assumed equal between layers. What a file may leave out:
``norm.groups`` (1), an attention's ``mask`` (every earlier position is seen), ``rot`` (no rotation), ``softcap`` (none), ``vdim``
(the values are the keys, so it can only be ``dim``). ``max_position`` (the longest sequence the engine plans for) is optional.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Tuple

from .bapavik import _need, _positive
from .base import ConfigError, ModelConfig
from .gebilorn import _check_rot, _number


def _check_attention(m, where: str) -> None:
    _need(m, ("heads", "kv_heads", "dim", "scale"), where)
    _positive(m, ("heads", "kv_heads", "dim"), where)
    _number(m, ("scale",), where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
    if m.get("vdim", m["dim"]) != m["dim"]:
        raise ConfigError(f"{where}.vdim must equal dim: the values are the keys")
    if m.get("softcap") is not None:
        _number(m, ("softcap",), where)
    if m.get("mask") is not None:
        _need(m["mask"], ("size",), where + ".mask")
        _positive(m["mask"], ("size",), where + ".mask")
    if m.get("rot") is not None:
        _check_rot(m["rot"], m["dim"], where + ".rot")
        if m["rot"].get("scaling") is not None:
            raise ConfigError(f"{where}.rot: this design has no scaled frequencies")


@dataclass(frozen=True)
class VivepelConfig(ModelConfig):
    width: int
    vocab: int
    eps: float
    groups: int
    layers: Tuple[Dict[str, Any], ...]
    max_position: int = 1 << 17

    architecture = "Vivepel"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VivepelConfig":
        _need(d, ("width", "vocab", "norm", "layers"), "config.json")
        _positive(d, ("width", "vocab"), "config.json")
        _need(d["norm"], ("eps",), "norm")
        _number(d["norm"], ("eps",), "norm")
        groups = d["norm"].get("groups")
        if groups is not None:
            _positive(d["norm"], ("groups",), "norm")
        groups = int(groups or 1)
        if d["width"] % groups:
            raise ConfigError(f"norm.groups: a width of {d['width']} cannot be cut into {groups} equal parts")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, layer in enumerate(d["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] != "attention":
                raise ConfigError(f"{where}: type {layer['type']!r} is not known (attention)")
            _check_attention(layer["mixer"], where + ".mixer")
            f = layer.get("mlp")
            if f is not None:
                _need(f, ("kind",), where + ".mlp")
                if f["kind"] != "dense":
                    raise ConfigError(f"{where}.mlp.kind {f['kind']!r} is not known (dense)")
                _need(f, ("ff",), where + ".mlp")
                _positive(f, ("ff",), where + ".mlp")
            layers.append(copy.deepcopy({"type": layer["type"], "mixer": layer["mixer"], "mlp": f}))
        return cls(width=int(d["width"]), vocab=int(d["vocab"]), eps=float(d["norm"]["eps"]), groups=groups, layers=tuple(layers),
                   max_position=int(d.get("max_position") or (1 << 17)))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps, "groups": self.groups},
                "layers": copy.deepcopy(list(self.layers)), "max_position": self.max_position}
