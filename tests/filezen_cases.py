"""Shared by the Filezen tests: small configurations of their own, seeded weights, engines on either backend.

Two backends: "emu" runs the engine's own parts, cache manager and step function on the CPU over the torch stand-ins of
tests/emu_kernels.py (no GPU needed, float32); "cuda" runs the real kernels. The oracle is tests/plain/filezen_plain.py
in float64.
"""
from __future__ import annotations

import torch

from tests.bapavik_cases import BACKENDS, make_engine, runtime_for, tolerance, write_model  # noqa: F401
from tests.gebilorn_cases import compare_rows  # noqa: F401
from tests.plain import filezen_plain as P


def LAT(heads, dim, rot, vdim, rank, scale, size, base, scaling=None, kv_from=None):
    """``scaling``: (factor, original, fast, slow) or None; ``size``: the window, or None for every earlier position."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if size is not None:
        m["mask"] = {"size": size}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def RET(dim, vdim, decay, base=None, dims=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if base is not None:
        m["rot"] = {"base": base, "dims": dims}
    return m


DENSE = lambda ff: {"kind": "dense", "ff": ff}


def MOE(experts, top, ff, groups=None, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


LATENT = lambda mixer, mlp: {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
RETENTION = lambda mixer, mlp: {"type": "retention", "mixer": mixer, "mlp": mlp}
YARN = (4.0, 64, 8.0, 1.0)

# Sizes differ between layers and from each other wherever the design allows: value heads smaller and larger than the keys';
# readers of another layer's rows with more and fewer heads, other head sizes, scales and windows (shorter and longer than the
# maker's, and none); two layers that make rows and one behind another that read them; windows shorter than a page and longer
# than several; ramps of frequencies and none; matrix states with more and fewer value than key channels, wholly, partly and
# not rotated, with fast and slow and no decay; every kind of feed-forward behind every kind of mixer, and none; routers with
# one and several kept groups, one group, and groups of one expert.
CONFIGS = {
    "a": {"architecture": "Filezen", "width": 64, "vocab": 150, "norm": {"eps": 1e-5}, "embedding": {"scale": 6.0}, "residual_mult": 0.7,
          "layers": [
              RETENTION(RET(16, 24, [0.9, 0.99], 10000.0, 16), MOE(6, 2, 32, groups=(3, 2), shared=48)),
              LATENT(LAT(4, 16, 8, 24, 40, 0.2, 20, 10000.0, YARN), DENSE(96)),
              LATENT(LAT(2, 24, 8, 16, 40, 0.3, 33, 10000.0, YARN, kv_from=1), MOE(4, 1, 48)),
              RETENTION(RET(24, 16, [0.5, 0.97, 1.0]), None),
              LATENT(LAT(3, 8, 8, 8, 40, 0.25, 7, 10000.0, YARN, kv_from=1), MOE(4, 2, 24, groups=(4, 2))),
          ]},
    # sizes that are multiples of nothing: no vector load, no tensor-core tile and no padded head fits them exactly
    "o": {"architecture": "Filezen", "width": 100, "vocab": 131, "norm": {"eps": 3e-5}, "embedding": {"scale": 5.5}, "residual_mult": 1.3,
          "layers": [
              LATENT(LAT(5, 12, 6, 10, 30, 0.22, None, 3000.0), MOE(9, 3, 22, groups=(3, 1), shared=30)),
              RETENTION(RET(20, 12, [0.8, 0.95, 0.999], 500.0, 10), DENSE(70)),
              LATENT(LAT(3, 20, 14, 18, 17, 0.25, 50, 3000.0, (8.0, 32, 4.0, 0.5)), None),
              LATENT(LAT(1, 6, 14, 34, 17, 0.3, 60, 3000.0, (8.0, 32, 4.0, 0.5), kv_from=2), MOE(5, 5, 30)),
              LATENT(LAT(7, 12, 6, 10, 30, 0.2, 9, 3000.0, kv_from=0), DENSE(33)),
          ]},
    # latent rows wider than the attention kernels take (keys and values cached per head), and narrow ones beside them
    "q": {"architecture": "Filezen", "width": 48, "vocab": 97, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "residual_mult": 1.0,
          "layers": [
              LATENT(LAT(3, 8, 8, 16, 264, 0.25, 44, 100.0, (2.0, 16, 8.0, 1.0)), MOE(8, 2, 16, groups=(2, 1), shared=16)),
              RETENTION(RET(32, 16, [0.96], 100.0, 8), DENSE(64)),
              LATENT(LAT(2, 16, 8, 8, 264, 0.3, 64, 100.0, (2.0, 16, 8.0, 1.0), kv_from=0), MOE(4, 4, 16, groups=(2, 2))),
              LATENT(LAT(6, 8, 4, 8, 12, 0.4, 17, 200.0), None),
          ]},
}

# Layers as wide as a real model's: heads of 64 + 64, latent rows of 192 + 64, experts and dense widths that are multiples of
# 64, so the bfloat16 products run on the tensor-core tiles and the attention on its widest head size.
CONFIGS["wide"] = {"architecture": "Filezen", "width": 512, "vocab": 300, "norm": {"eps": 1e-5}, "embedding": {"scale": 12.0}, "residual_mult": 0.6,
                   "layers": [
                       LATENT(LAT(8, 64, 64, 64, 192, 0.088, 96, 10000.0, (8.0, 128, 16.0, 1.0)), MOE(16, 2, 128, groups=(4, 2), shared=128)),
                       RETENTION(RET(64, 128, [0.97, 0.98, 0.99, 0.998], 10000.0, 64), DENSE(1024)),
                       LATENT(LAT(4, 128, 64, 128, 192, 0.07, 160, 10000.0, (8.0, 128, 16.0, 1.0), kv_from=0), MOE(16, 2, 128, groups=(2, 1))),
                   ]}


def make_weights(cfg: dict, seed: int, expert_gain: float = 1.0):
    """float32 weights by name, sized so that every layer's output matters."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in P.tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "embed":
            t = torch.randn(shape, generator=g) / cfg["embedding"]["scale"]
        else:
            t = torch.randn(shape, generator=g) * 1.5 / shape[-1] ** 0.5
        if leaf == "down" and ".e" in name:
            t = t * expert_gain
        w[name] = t.bfloat16().float()          # values that a bfloat16 file holds exactly
    return w


def plain_logits(w, cfg, tokens, streams=None):
    with torch.no_grad():
        return P.forward(tokens, {k: v.double() for k, v in w.items()}, cfg, streams).float()


def row_error(row, ref) -> float:
    """Root mean square of the difference over the vocabulary (means taken off), as a share of the reference row's own."""
    d = row - ref
    return float((d - d.mean()).pow(2).mean().sqrt() / (ref - ref.mean()).pow(2).mean().sqrt())


def rounding_limits(w, cfg, requests, plain, draws: int = 2):
    """{request: a limit on every row's ``row_error`` in bfloat16}. A state that a query hardly meets is divided by its own size,
    and a router's close call can fall the other way, so what rounding does differs from row to row. It is measured on the plain
    model: weights moved at random by up to a bfloat16 rounding move every product about as far as rounding its result does. A
    row may go four times as far as the furthest of ``draws`` such models, and 8 % in any case."""
    g = torch.Generator().manual_seed(1)
    moved = [{k: v * (1.0 + 2.0 ** -8 * (torch.rand(v.shape, generator=g) - 0.5)) for k, v in w.items()} for _ in range(draws)]
    return {rid: [max([0.08] + [4.0 * row_error(m[p], plain[rid][p]) for m in runs]) for p in range(len(toks))]
            for rid, toks in requests.items() for runs in [[plain_logits(mw, cfg, toks) for mw in moved]]}


def compare_with_limits(got, plain, backend, limits, allow: int = 0) -> None:
    """float32: ``compare_rows``. bfloat16: every row finite, at most one in ten (or two, or ``allow``) beyond its limit (one close
    call of a router moves the tokens behind it too), and half of all rows within 6 %."""
    if backend[1] == "float32":
        compare_rows(got, plain, backend)
        return
    errors = {}
    for (rid, pos), row in got.items():
        assert bool(torch.isfinite(row).all()), f"request {rid!r} position {pos}: not finite"
        errors[(rid, pos)] = row_error(row, plain[rid][pos])
    over = [(key, e, limits[key[0]][key[1]]) for key, e in errors.items() if e > limits[key[0]][key[1]]]
    assert len(over) <= max(2, allow, len(errors) // 10), f"{len(over)} of {len(errors)} rows beyond their limits, the first: {over[:3]}"
    assert sorted(errors.values())[len(errors) // 2] <= 0.06
