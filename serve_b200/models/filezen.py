"""The Filezen decoder as a layer description.

x = embed[token] * scale. A layer's sub-layers read the stream as it is, and only what they give back is normalised:
x += m * n1(mixer(x)), then x += m * n2(ff(x)), m one constant of the model: an arrangement with a norm on both sides whose front
norms are the identity. The mixer is "latent_attention" (queries straight from the stream, keys and values read out of one
normalised low-rank vector per token plus one rotated key part that all heads share, frequencies scaled by a ramp over the pairs, a
sliding window; ``kv_from``: the rows of an earlier layer, read through this layer's own queries, read-outs and mask) or "retention"
(a matrix state per head with a fixed decay, rotated queries and keys, the read-out normalised per head without a weight and gated
by silu). The feed-forward is dense and gated with silu, a mixture of silu-gated experts (softmax router, the choice limited to the
best groups, weights = chosen scores over their sum, an ungated shared expert), or absent. Final norm, the embedding table as head.
Tensor names: "embed", "final.norm", and under "l<i>." the layer's "norm1", "norm2", "mix.*", "mlp.*".
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.filezen import FilezenConfig
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..parts.latent_attention import LatentAttention

# added to the sum the chosen experts' scores are divided by
WEIGHT_SUM_EPS = 1e-20


def _mixer_spec(kind: str, m: dict, width: int, eps: float, prefix: str, row_of=None, row_shared: bool = False) -> PartSpec:
    if kind == "retention":
        rot = m.get("rot")
        dims = rot.get("dims", m["dim"]) if rot else 0
        position = PartSpec("rotary", {"rotary_dim": dims, "theta": rot["base"], "pairing": "half"}) if dims else PartSpec("none")
        return PartSpec("retention", {"hidden": width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "decay": list(m["decay"]),
                                      "eps": eps, "position": position}, prefix)
    sc = m["rot"].get("scaling")
    return PartSpec("latent_attention", {
        "hidden": width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
        "scale": m["scale"], "rot_base": m["rot"]["base"], "rot_dims": m["rot_dim"], "pairing": "half", "eps": eps,
        "rot_scaling": dict(sc, kind="yarn") if sc else None, "window": (m.get("mask") or {}).get("size"), "row_of": row_of,
        "row_shared": row_shared}, prefix)


def _feed_forward_spec(f: dict, width: int, prefix: str) -> PartSpec:
    if f["kind"] == "dense":
        return PartSpec("swiglu", {"hidden": width, "intermediate": f["ff"], "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix)
    r = f["router"]
    return PartSpec("routed_experts", {
        "hidden": width, "experts": r["experts"], "top": r["top"], "ff": f["expert"]["ff"], "score": "softmax", "renormalise": True,
        "renormalise_eps": WEIGHT_SUM_EPS, "scale_input": False, "activation": "swiglu", "groups": r.get("groups"),
        "shared": {"ff": f["shared"]["ff"]} if f.get("shared") is not None else None}, prefix)


def filezen_spec(cfg: FilezenConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.eps

    def norm(name, prefix="", multiplier=None):
        return PartSpec("grouped_rms", {"size": width, "eps": eps, "weight_name": name, "multiplier": multiplier}, prefix)

    source = [layer["mixer"].get("kv_from") if layer["type"] == "latent_attention" else None for layer in cfg.layers]
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m, j = f"l{i}.", layer["mixer"], source[i]
        parts = {"mixer_norm": PartSpec("identity", {"size": width}),
                 "mixer": _mixer_spec(layer["type"], m, width, eps, p + "mix.", None if j is None else f"l{j}.mix.", i in source),
                 "mixer_post_norm": norm("norm1", p, cfg.residual_mult)}
        if layer["mlp"] is not None:
            parts.update(feed_forward_norm=PartSpec("identity", {"size": width}),
                         feed_forward=_feed_forward_spec(layer["mlp"], width, p + "mlp."), feed_forward_post_norm=norm("norm2", p, cfg.residual_mult))
        layers.append(LayerSpec(PartSpec("sandwich_norm"), parts))
        # cached rows are read where the other layer wrote them; keys and values cached per head are this layer's own
        reads = j is not None and not LatentAttention.caches_per_head(m["kv_rank"], m["rot_dim"])
        schedule.append(ScheduleEntry(i, j if reads else None))
    spec = ModelSpec(
        architecture=FilezenConfig.architecture, hidden_size=width, vocab_size=cfg.vocab,
        embedding=PartSpec("table", {"vocab": cfg.vocab, "hidden": width, "name": "embed", "scale": cfg.embedding_scale}), layers=layers,
        schedule=schedule, final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": width, "name": "head", "tied_to": "embed"}), max_position=cfg.max_position)
    spec.validate()
    return spec


register_architecture(FilezenConfig.architecture, FilezenConfig, filezen_spec)
