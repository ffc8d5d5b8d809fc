"""Shared by the Vivepel tests: small configurations of their own, seeded weights, engines on either backend.

Two backends: "emu" runs the engine's own parts, cache manager and step function on the CPU over the torch stand-ins of
tests/emu_kernels.py (no GPU needed, float32); "cuda" runs the real kernels. The oracle is tests/plain/vivepel_plain.py
in float64.
"""
from __future__ import annotations

import torch

from tests.bapavik_cases import BACKENDS, compare_rows, make_engine, runtime_for, write_model  # noqa: F401
from tests.plain import vivepel_plain as P


def ATT(heads, kv, dim, scale, cap, size, base, dims):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "softcap": cap, "mask": {"size": size},
         "rot": {"base": base, "dims": dims}}
    if cap is None:
        del m["softcap"]                    # a file may leave the cap out,
    if size is None:
        del m["mask"]                       # the mask (every earlier position is seen)
    if dims is None:
        del m["rot"]                        # and the rotation
    return m


def LAYER(att, ff):
    return {"type": "attention", "mixer": att, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


# Sizes differ between layers and from each other wherever the design allows: one key/value head per query head, one for two
# and one for all; a single head (a 1 x 1 mixing matrix); more heads than one product tile of the mixing holds; head sizes that
# are and are not multiples of 16; rotation of a part of a head, of all of it and none; blocks of positions shorter than a page,
# longer than several, of one position, and none; caps that bend the scores and caps that hardly do; layers without a
# feed-forward; norms over one, two, three, five and eight parts of the row.
CONFIGS = {
    "a": {"architecture": "Vivepel", "width": 64, "vocab": 150, "norm": {"eps": 1e-5, "groups": 2}, "layers": [
        LAYER(ATT(4, 2, 24, 0.3, 5.0, 20, 10000.0, 16), 96), LAYER(ATT(2, 2, 16, 0.4, 30.0, 33, 500.0, 16), None),
        LAYER(ATT(8, 1, 32, 0.2, 2.0, 20, 10000.0, 8), 160), LAYER(ATT(1, 1, 16, 0.3, 15.0, 7, 300.0, 4), 48)]},
    # sizes that are multiples of nothing: no vector load, no tensor-core tile and no padded head fits them exactly
    "o": {"architecture": "Vivepel", "width": 105, "vocab": 131, "norm": {"eps": 3e-5, "groups": 5}, "layers": [
        LAYER(ATT(5, 5, 12, 0.5, 4.0, 11, 3000.0, 10), 70), LAYER(ATT(6, 1, 20, 0.3, None, None, None, None), 33),
        LAYER(ATT(3, 3, 22, 0.35, 9.0, 50, 70.0, 22), 101)]},
    "q": {"architecture": "Vivepel", "width": 48, "vocab": 97, "norm": {"eps": 1e-6, "groups": 3}, "layers": [
        LAYER(ATT(20, 5, 16, 0.4, 6.0, 64, 100.0, 8), 64), LAYER(ATT(6, 3, 8, 0.6, 12.0, 1, 100.0, 8), 40),
        LAYER(ATT(36, 2, 16, 0.4, 20.0, 44, 1000.0, 4), None)]},
}
# Layers as wide as a real model's: heads of 128 and 64, widths that are multiples of 64.
CONFIGS["wide"] = {"architecture": "Vivepel", "width": 512, "vocab": 300, "norm": {"eps": 1e-5, "groups": 8}, "layers": [
    LAYER(ATT(8, 2, 128, 0.09, 20.0, 160, 200000.0, 64), 1024), LAYER(ATT(16, 4, 64, 0.125, 50.0, None, 10000.0, 64), 2048)]}


def make_weights(cfg: dict, seed: int):
    """float32 weights by name, sized so that every layer's output matters."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in P.tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        rnd = torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm2", "norm1b", "norm2b", "norm"):
            t = 1.0 + 0.2 * rnd
        elif leaf in ("ls1", "ls2"):
            t = 0.7 + 0.2 * rnd
        elif leaf == "b":
            t = 0.3 * rnd
        elif leaf == "talk":
            t = 0.7 * torch.eye(shape[0]) + 0.5 * rnd / shape[0] ** 0.5
        elif leaf == "act":
            t = torch.tensor([0.8, -0.5, 0.4, 0.15]) + 0.1 * rnd
        elif leaf == "embed":
            t = rnd
        else:
            t = rnd * 1.5 / shape[-1] ** 0.5
        w[name] = t.bfloat16().float()          # values that a bfloat16 file holds exactly
    return w


def plain_logits(w, cfg, tokens, streams=None):
    with torch.no_grad():
        return P.forward(tokens, {k: v.double() for k, v in w.items()}, cfg, streams).float()
