"""Typed configuration of the Filezen decoder, read from its config.json.

The file gives ``width``, ``vocab``, ``norm.eps``, ``embedding.scale``, ``residual_mult`` and ``layers``. A layer names its mixer
(``type``: "latent_attention" or "retention"), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: an object of
kind "dense" or "moe", or null for a layer without one). Every size and constant is taken from the file; nothing is assumed equal
between layers. A latent attention with ``kv_from`` reads the rows of the layer it names. What a file may leave out:
``embedding.scale`` and ``residual_mult`` (1), an attention's ``mask`` (every earlier position is seen), its ``rot.dims`` (it can only
be ``rot_dim``), ``rot.scaling`` (frequencies as they are), a retention's ``rot`` (no rotation), a router's ``groups`` (any expert can
be chosen), an expert layer's ``shared``. ``max_position`` (the longest sequence the engine plans for) is optional.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Tuple

from .bapavik import _need, _positive
from .base import ConfigError, ModelConfig
from .gebilorn import _number

SCALING = ("factor", "original", "fast", "slow")


def _check_rot(rot, limit: int, where: str, scaling_allowed: bool) -> None:
    _need(rot, ("base",), where)
    _number(rot, ("base",), where)
    dims = rot.get("dims", limit)
    if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > limit:
        raise ConfigError(f"{where}.dims must be even and at most {limit}")
    if rot.get("scaling") is None:
        return
    if not scaling_allowed:
        raise ConfigError(f"{where}.scaling: this mixer has no scaled frequencies")
    _need(rot["scaling"], SCALING, where + ".scaling")
    _number(rot["scaling"], SCALING, where + ".scaling")
    if rot["base"] == 1:
        raise ConfigError(f"{where}.base must not be 1 with scaled frequencies")


def _check_latent(m, where: str) -> None:
    _need(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"), where)
    _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank"), where)
    _number(m, ("scale",), where, positive=False)
    if m["rot_dim"] % 2:
        raise ConfigError(f"{where}.rot_dim must be even")
    _check_rot(m["rot"], m["rot_dim"], where + ".rot", True)
    if m["rot"].get("dims", m["rot_dim"]) != m["rot_dim"]:
        raise ConfigError(f"{where}.rot.dims must be rot_dim: the whole rotated part turns")
    if m.get("mask") is not None:
        _need(m["mask"], ("size",), where + ".mask")
        _positive(m["mask"], ("size",), where + ".mask")


def _check_retention(m, where: str) -> None:
    _need(m, ("heads", "dim", "vdim", "decay"), where)
    _positive(m, ("heads", "dim", "vdim"), where)
    decay = m["decay"]
    if not isinstance(decay, list) or len(decay) != m["heads"] or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
        raise ConfigError(f"{where}.decay must list one number for each of the {m['heads']} heads")
    if m.get("rot") is not None:
        _check_rot(m["rot"], m["dim"], where + ".rot", False)


def _check_source(layers, i: int, where: str) -> None:
    """A layer that reads another's rows: the other comes before it, makes rows of its own, and makes them alike."""
    m, j = layers[i]["mixer"], layers[i]["mixer"]["kv_from"]
    if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < i:
        raise ConfigError(f"{where}.kv_from must name an earlier layer, got {j!r}")
    source = layers[j]
    if source["type"] != "latent_attention" or source["mixer"].get("kv_from") is not None:
        raise ConfigError(f"{where}.kv_from: layer {j} makes no rows of its own")
    key = lambda x: (x["kv_rank"], x["rot_dim"], x["rot"]["base"], x["rot"].get("scaling"))
    if key(source["mixer"]) != key(m):
        raise ConfigError(f"{where}.kv_from: kv_rank, rot_dim and rotation must be those of layer {j}")


def _check_mlp(f, where: str) -> None:
    _need(f, ("kind",), where)
    if f["kind"] == "dense":
        _need(f, ("ff",), where)
        _positive(f, ("ff",), where)
    elif f["kind"] == "moe":
        _need(f, ("expert", "router"), where)
        _need(f["expert"], ("ff",), where + ".expert")
        _need(f["router"], ("experts", "top"), where + ".router")
        _positive(f["expert"], ("ff",), where + ".expert")
        r = f["router"]
        _positive(r, ("experts", "top"), where + ".router")
        open_ = r["experts"]
        if r.get("groups") is not None:
            g = r["groups"]
            _need(g, ("count", "keep"), where + ".router.groups")
            _positive(g, ("count", "keep"), where + ".router.groups")
            if r["experts"] % g["count"] or g["keep"] > g["count"]:
                raise ConfigError(f"{where}.router.groups: {r['experts']} experts, {g['count']} equal groups, {g['keep']} of them kept")
            open_ = g["keep"] * (r["experts"] // g["count"])
        if r["top"] > open_:
            raise ConfigError(f"{where}.router: top exceeds the experts that can be chosen")
        if f.get("shared") is not None:
            _need(f["shared"], ("ff",), where + ".shared")
            _positive(f["shared"], ("ff",), where + ".shared")
    else:
        raise ConfigError(f"{where}.kind {f['kind']!r} is not known (dense, moe)")


@dataclass(frozen=True)
class FilezenConfig(ModelConfig):
    width: int
    vocab: int
    eps: float
    embedding_scale: float
    residual_mult: float
    layers: Tuple[Dict[str, Any], ...]
    max_position: int = 1 << 17

    architecture = "Filezen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "FilezenConfig":
        _need(d, ("width", "vocab", "norm", "layers"), "config.json")
        _positive(d, ("width", "vocab"), "config.json")
        _need(d["norm"], ("eps",), "norm")
        _number(d["norm"], ("eps",), "norm")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, layer in enumerate(d["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] == "latent_attention":
                _check_latent(layer["mixer"], where + ".mixer")
            elif layer["type"] == "retention":
                _check_retention(layer["mixer"], where + ".mixer")
            else:
                raise ConfigError(f"{where}: type {layer['type']!r} is not known (latent_attention, retention)")
            f = layer.get("mlp")
            if f is not None:
                _check_mlp(f, where + ".mlp")
            layers.append(copy.deepcopy({"type": layer["type"], "mixer": layer["mixer"], "mlp": f}))
            if layer["type"] == "latent_attention" and layer["mixer"].get("kv_from") is not None:
                _check_source(layers, i, where + ".mixer")
        scale = mult = 1.0
        emb = d.get("embedding") or {}
        if emb.get("scale") is not None:
            _number(emb, ("scale",), "embedding", positive=False)
            scale = float(emb["scale"])
        if d.get("residual_mult") is not None:
            _number(d, ("residual_mult",), "config.json", positive=False)
            mult = float(d["residual_mult"])
        return cls(width=int(d["width"]), vocab=int(d["vocab"]), eps=float(d["norm"]["eps"]), embedding_scale=scale, residual_mult=mult,
                   layers=tuple(layers), max_position=int(d.get("max_position") or (1 << 17)))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
                "layers": copy.deepcopy(list(self.layers)), "max_position": self.max_position}
