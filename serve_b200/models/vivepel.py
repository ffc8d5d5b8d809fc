"""The Vivepel decoder as a layer description.

x = embed[token]. A layer has a norm before and a norm after each of its two sub-layers, and a learned scale per element behind the
latter: x += s1 * n1b(mixer(n1(x))), then x += s2 * n2b(ff(n2(x))); every norm divides equal parts of the vector by their own root
mean square. The mixer is attention with biased queries and keys, the keys as projected for values, a per-head query/key norm before
a partial rotation, capped scores, keys of the query's own block of positions only, one added to the softmax's denominator, and
weights that an H x H matrix mixes over the heads. The feed-forward is dense without a gate, its activation a polynomial of
normalised powers; a layer may have none. Final norm, an output head of its own. Tensor names: "embed", "final.norm", "head", and
under "l<i>." the layer's "norm1", "norm1b", "ls1", "mix.*" and "norm2", "norm2b", "ls2", "mlp.*".
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..config.vivepel import VivepelConfig


def _mixer_spec(m: dict, width: int, eps: float, prefix: str) -> PartSpec:
    rot = m.get("rot")
    position = PartSpec("none") if not rot or not rot["dims"] else PartSpec(
        "rotary", {"rotary_dim": rot["dims"], "theta": rot["base"], "pairing": "half"})
    return PartSpec("talking_attention", {
        "hidden": width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "scale": m["scale"], "bias": True,
        "keys_are_values": True, "head_norm_eps": eps, "softcap": m.get("softcap"), "chunk": (m.get("mask") or {}).get("size"),
        "sink_score": 0.0, "position": position}, prefix)


def _feed_forward_spec(f: dict, width: int, eps: float, prefix: str) -> PartSpec:
    return PartSpec("plain_dense", {"hidden": width, "intermediate": f["ff"], "activation": "poly_norm", "eps": eps}, prefix)


def vivepel_spec(cfg: VivepelConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.eps

    def norm(name, prefix="", scale=None):
        return PartSpec("grouped_rms", {"size": width, "groups": cfg.groups, "eps": eps, "weight_name": name, "scale_name": scale}, prefix)

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": norm("norm1", p), "mixer": _mixer_spec(layer["mixer"], width, eps, p + "mix."),
                 "mixer_post_norm": norm("norm1b", p, "ls1")}
        if layer["mlp"] is not None:
            parts.update(feed_forward_norm=norm("norm2", p), feed_forward=_feed_forward_spec(layer["mlp"], width, eps, p + "mlp."),
                         feed_forward_post_norm=norm("norm2b", p, "ls2"))
        layers.append(LayerSpec(PartSpec("sandwich_norm"), parts))
        schedule.append(ScheduleEntry(i))
    spec = ModelSpec(
        architecture=VivepelConfig.architecture, hidden_size=width, vocab_size=cfg.vocab,
        embedding=PartSpec("table", {"vocab": cfg.vocab, "hidden": width, "name": "embed"}), layers=layers, schedule=schedule,
        final_norm=norm("final.norm"), head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": width, "name": "head"}),
        max_position=cfg.max_position)
    spec.validate()
    return spec


register_architecture(VivepelConfig.architecture, VivepelConfig, vivepel_spec)
