"""The Filezen decoder in the engine against the plain implementation of tests/plain/filezen_plain.py.

Every test runs on the CPU over the torch stand-ins of the kernels (which checks the parts, the cache manager, the step
function and the scheduler) and, marked gpu, on the real kernels in float32 and bfloat16.
"""
import copy
import json
import math
import os
import random
import subprocess
import sys

import pytest
import torch

from serve_b200.cache import CacheManager
from serve_b200.config import ConfigError, PartSpec, build_spec, config_from_dict
from serve_b200.parts import DeferredNorm, build_part
from tests import helpers
from tests.filezen_cases import (BACKENDS, CONFIGS, DENSE, LAT, LATENT, MOE, RET, RETENTION, YARN, compare_with_limits, make_engine,
                                 make_weights, plain_logits, rounding_limits, runtime_for, write_model)
from tests.plain import filezen_plain as P
from tests.test_bapavik import _ctx, _run_part, _tol

LENGTHS = {"a": [1, 5, 23, 49, 75, 130], "o": [3, 40, 90, 17], "q": [2, 9, 31, 64, 101]}
PAGE = {"a": 8, "o": 4, "q": 16}
F64 = lambda w: {k: v.double() for k, v in w.items()}


# ---- configuration and description ----------------------------------------------------------------------------
def test_configuration_is_read_from_the_file_and_describes_every_layer():
    from serve_b200.weights.random_init import model_tensor_decls

    for name, raw in CONFIGS.items():
        cfg = config_from_dict(copy.deepcopy(raw))
        assert type(cfg).__name__ == "FilezenConfig" and cfg.width == raw["width"] and cfg.vocab == raw["vocab"]
        assert cfg.embedding_scale == raw["embedding"]["scale"] and cfg.residual_mult == raw["residual_mult"]
        spec = build_spec(cfg)
        assert spec.embedding.params["scale"] == raw["embedding"]["scale"] and spec.head.params["tied_to"] == "embed"
        assert len(spec.layers) == len(raw["layers"]) == len(spec.schedule)
        for i, (layer, ls, entry) in enumerate(zip(raw["layers"], spec.layers, spec.schedule)):
            m, p = layer["mixer"], ls.parts["mixer"].params
            assert ls.block.kind == "sandwich_norm" and ls.parts["mixer"].kind == layer["type"]
            assert ls.parts["mixer_norm"].kind == "identity" and ls.parts["mixer_post_norm"].params["multiplier"] == raw["residual_mult"]
            assert ("feed_forward" in ls.parts) == (layer["mlp"] is not None)
            if layer["type"] == "latent_attention":
                j, wide = m.get("kv_from"), m["kv_rank"] + m["rot_dim"] > 256
                assert p["window"] == (m.get("mask") or {}).get("size") and (p["rot_scaling"] is None) == ("scaling" not in m["rot"])
                assert p["row_of"] == (None if j is None else f"l{j}.mix.") and entry.cache_of == (None if wide else j)
            else:
                assert p["decay"] == m["decay"] and p["position"].params.get("rotary_dim", 0) == (m.get("rot") or {}).get("dims", 0)
            if layer["mlp"] and layer["mlp"]["kind"] == "moe":
                f = ls.parts["feed_forward"].params
                assert f["groups"] == layer["mlp"]["router"].get("groups") and (f["shared"] is None) == ("shared" not in layer["mlp"])
        assert {n: tuple(d.shape) for n, d in model_tensor_decls(cfg).items()} == P.tensor_shapes(raw)
        assert config_from_dict(cfg.to_dict()) == cfg


@pytest.mark.parametrize("breaker", [
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"].update(rot_dim=7),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0),
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][2]["mixer"].update(kv_from=0),        # makes no rows
    lambda c: c["layers"][2]["mixer"].update(kv_from=2),        # itself
    lambda c: c["layers"][4]["mixer"].update(kv_from=2),        # reads rows, makes none
    lambda c: c["layers"][2]["mixer"].update(kv_rank=32),
    lambda c: c["layers"][2]["mixer"]["rot"].update(base=500.0),
    lambda c: c["layers"][0]["mixer"].update(decay=[0.9]),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
    lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 2.0, "original": 8, "fast": 2.0, "slow": 1.0}),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5),    # two groups of two are open
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["norm"].update(eps=0.0),
    lambda c: c.update(residual_mult="half"),
    lambda c: c.pop("vocab"),
])
def test_configuration_refuses_what_it_cannot_run(breaker):
    raw = copy.deepcopy(CONFIGS["a"])
    breaker(raw)
    with pytest.raises(ConfigError):
        config_from_dict(raw)


# ---- whole models ---------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """{config name: {dtype: (weights, requests, plain logits, limits in bfloat16, model folder)}}."""
    out = {}
    for name in LENGTHS:
        cfg = CONFIGS[name]
        reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=20 + i) for i, n in enumerate(LENGTHS[name])}
        w = make_weights(cfg, 100 + len(name), expert_gain=0.5)
        plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
        limits = rounding_limits(w, cfg, reqs, plain) if torch.cuda.is_available() else None
        out[name] = {dt: (w, reqs, plain, limits, write_model(str(tmp_path_factory.mktemp(f"{name}-{dt}")), cfg, w, getattr(torch, dt)))
                     for dt in ("float32", "bfloat16")}
    return out


def test_plain_layers_feed_one_another(models):
    """The oracle's own premise: every layer changes the residual stream, and the last positions depend on the first token."""
    for name in LENGTHS:
        w, reqs, plain, _, _ = models[name]["float32"]
        cfg, toks = CONFIGS[name], reqs["r2"]
        layers = []
        plain_logits(w, cfg, toks, layers)
        for a, b in zip(layers, layers[1:]):
            assert float((a - b).abs().max()) > 1e-2
        other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
        assert float((plain_logits(w, cfg, other)[-1] - plain["r2"][-1]).abs().max()) > 1e-4


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["a", "o", "q"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "pairs", "single_tokens"])
def test_cuts_match_plain(models, name, backend, cut):
    w, reqs, plain, limits, folder = models[name][backend[1]]
    page = PAGE[name]
    eng = make_engine(folder, backend, page, num_pages=-(-160 // page) * 2, graphs=(cut == "tail_decode"))
    if cut == "single_tokens":
        steps = helpers.trace_tail_decode({k: v for k, v in reqs.items() if len(v) <= 50}, tail=10 ** 6)
    else:
        make = {"whole": helpers.trace_whole, "tail_decode": lambda r: helpers.trace_tail_decode(r, tail=40),
                "portions": lambda r: helpers.trace_portions(r, sizes=(7, 2, 19, 1, 3, 2, 33, 5, 2, 11)),
                "pairs": lambda r: helpers.trace_portions({k: v for k, v in r.items() if len(v) <= 80}, sizes=(2,))}[cut]
        steps = make(reqs)
    with torch.inference_mode():
        got = helpers.replay(eng, steps)
    eng.kernels.check_errors()
    compare_with_limits(got, plain, backend, limits)
    eng.cache.check()
    assert eng.cache.live == 0


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["a", "o", "q"])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, backend):
    """Unequal requests side by side, portions beside single tokens, fewer slots and pages than the requests need in
    all: every row must equal the request run alone. Pages are poisoned first, so that a page that is read without
    having been written shows; a slot's matrix states are the next request's whoever had the slot before."""
    w, reqs, plain, limits, folder = models[name][backend[1]]
    page = PAGE[name]
    steps = helpers.trace_mixed(reqs, live=3, seed=7)
    need = helpers.tokens_needed(steps, page) // page
    assert need < sum(-(-len(t) // page) for t in reqs.values())
    eng = make_engine(folder, backend, page, num_pages=need, max_slots=3, context=160)
    for view in eng.stepper.views:
        if view is not None and view.k is not None:
            view.k.fill_(float("nan"))
            view.v.fill_(float("nan"))
    with torch.inference_mode():
        got = helpers.replay(eng, steps)
    eng.kernels.check_errors()
    compare_with_limits(got, plain, backend, limits)
    eng.cache.check()
    assert eng.cache.live == 0 and eng.cache.free_slots == 3
    assert max(g.pool.high_water for g in eng.cache.groups) <= need


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["a", "q"])
def test_long_decoding_side_by_side(models, backend, name):
    """Two requests decoded one token at a time for 120 steps after short prompts (from CUDA graphs on the GPU): the windows
    pass over decoded tokens, pages are crossed and given back many times, the matrix states travel from replay to replay,
    and rows that one layer makes are read by others inside the graph."""
    cfg = CONFIGS[name]
    w, _, _, _, folder = models[name][backend[1]]
    seqs = {f"d{i}": helpers.random_tokens(cfg["vocab"], 140 - 9 * i, seed=60 + i) for i in range(2)}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in seqs.items()}
    limits = rounding_limits(w, cfg, seqs, plain) if backend[1] == "bfloat16" else None
    eng = make_engine(folder, backend, 16, num_pages=20, graphs=True)
    steps = [{"step": 0, "entries": [{"id": rid, "tokens": t[:11 + 6 * i], "want": [10 + 6 * i]} for i, (rid, t) in enumerate(seqs.items())], "end": []}]
    at = {rid: 11 + 6 * i for i, rid in enumerate(seqs)}
    while any(at[rid] < len(seqs[rid]) for rid in seqs):
        entries = [{"id": rid, "tokens": [t[at[rid]]], "want": [0]} for rid, t in seqs.items() if at[rid] < len(t)]
        for e in entries:
            at[e["id"]] += 1
        steps.append({"step": len(steps), "entries": entries, "end": []})
    with torch.inference_mode():
        got = helpers.replay(eng, steps)
    eng.kernels.check_errors()
    if backend[0] == "cuda":
        assert eng.stepper.launched_graphs > 80
    compare_with_limits(got, plain, backend, limits)


@pytest.mark.parametrize("backend", BACKENDS)
def test_greedy_generation_through_the_scheduler(models, backend):
    """generate(): the engine's own entry point, scheduler and sampler. Every generated token must be (within the tolerance)
    the best one of the plain model given the tokens before it."""
    from serve_b200.run import Request, generate

    cfg = CONFIGS["a"]
    w, reqs, _, _, folder = models["a"][backend[1]]
    eng = make_engine(folder, backend, 8, num_pages=40, max_slots=3, budget=32)
    prompts = [reqs["r1"], reqs["r2"], reqs["r3"][:30], reqs["r0"]]
    out = generate(eng, [Request(torch.tensor(p), len(p), 12) for p in prompts], temperature=0.0, eos_token_id=None)
    for p, r in zip(prompts, out):
        new = r.generated_tokens.tolist()
        assert len(new) == 12
        logits = plain_logits(w, cfg, p + new)
        tol = float(logits.abs().max()) * (2e-4 if backend[1] == "float32" else 2.0 ** -4)
        for i, tok in enumerate(new):
            row = logits[len(p) - 1 + i]
            assert float(row[tok]) >= float(row.max()) - 2 * tol, f"token {i} of a request is not the plain model's choice"
    assert eng.cache.live == 0


# ---- each mechanism alone ---------------------------------------------------------------------------------------
CUTS = [[57], [30, 1, 1, 2, 5, 17, 1], [1] * 57]


def _single(kind, mixer=None, mlp=None, width=64, eps=1e-5):
    """A one-layer configuration around the mechanism under test."""
    return {"architecture": "Filezen", "width": width, "vocab": 50, "norm": {"eps": eps}, "embedding": {"scale": 4.0}, "residual_mult": 1.0,
            "layers": [{"type": kind, "mixer": mixer, "mlp": mlp}]}


def _plain_mixer(kind, x, w64, m, eps, p="l0.mix."):
    if kind == "retention":
        return P.retention_mixer(x, w64, p, m, eps)
    return P.latent_mixer(x, w64, p, m, *P.latent_row(x, w64, p, m, eps))


def _mixer_alone(backend, cfg, cuts, seed=5, x=None, tweak=None, page=8, loose=1.0):
    from serve_b200.models.filezen import _mixer_spec

    layer = cfg["layers"][0]
    w = make_weights(cfg, seed)
    if tweak is not None:
        tweak(w, "l0.mix.")
    if x is None:
        x = torch.randn(sum(cuts), cfg["width"], generator=torch.Generator().manual_seed(seed + 1))
    x = x.bfloat16().float()
    spec = _mixer_spec(layer["type"], layer["mixer"], cfg["width"], cfg["norm"]["eps"], "l0.mix.")
    want = _plain_mixer(layer["type"], x.double(), F64(w), layer["mixer"], cfg["norm"]["eps"]).float()
    got = _run_part(backend, "mixer", spec, w, x, cuts, page=page)
    torch.testing.assert_close(got, want, atol=_tol(backend, want) * loose, rtol=0)
    return got, want, w


# Also: no mask and no scaling in the file; a window of one key (the query's own); one head; more rotated than plain
# elements; a ramp that ends inside, before and after the pairs there are; a factor of one (nothing changes) and below one
# (frequencies rise, vectors shorten); a latent row wider than the attention kernels take.
LATS = [LAT(4, 16, 8, 24, 40, 0.2, 20, 10000.0, YARN), LAT(5, 12, 6, 10, 30, 0.22, None, 3000.0), LAT(3, 8, 16, 16, 24, 0.25, 1, 100.0, (16.0, 16, 2.0, 1.0)),
        LAT(1, 24, 4, 16, 20, 0.19, 33, 500.0, (1.0, 64, 8.0, 1.0)), LAT(2, 16, 32, 40, 24, 0.2, 57, 1000.0, (0.5, 4096, 32.0, 1.0)),
        LAT(2, 16, 8, 16, 264, 0.2, 12, 100.0, (4.0, 32, 4.0, 1.0)), LAT(2, 16, 8, 16, 264, 0.2, None, 100.0)]
RETS = [RET(16, 24, [0.9, 0.99], 10000.0, 16), RET(20, 12, [0.8, 0.95, 0.999], 500.0, 10), RET(32, 16, [0.5]), RET(8, 40, [1.0, 0.0, 0.97, 0.25], 100.0, 2),
        RET(64, 64, [0.97, 0.996], 1e6, 64), RET(128, 72, [0.98], 10000.0, 64)]
WIDTHS = (64, 100, 48, 40, 72, 56, 64)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", CUTS, ids=["whole", "portions", "tokens"])
@pytest.mark.parametrize("which", range(len(LATS)))
def test_latent_attention_alone(backend, cuts, which):
    _mixer_alone(backend, _single("latent_attention", LATS[which], width=WIDTHS[which]), cuts, loose=2.0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", CUTS + [[33, 2, 130, 1, 64, 40]], ids=["whole", "portions", "tokens", "long-portions"])
@pytest.mark.parametrize("which", range(len(RETS)))
def test_retention_alone(backend, cuts, which):
    """Also: a head that never forgets, one that sees the current token only; a state taller than wide and wider than tall;
    rotation of the whole head, a part of it, one pair, none. The read-out is divided by its own size, so a token whose query
    happens to meet nothing in the state carries its rounding along: eps is the size of such a read-out's square."""
    _mixer_alone(backend, _single("retention", RETS[which], width=WIDTHS[which], eps=1e-2), cuts, loose=2.0)


def test_frequencies_on_the_ramp_and_the_lengthening():
    """The oracle's frequencies: kept before the ramp, divided by the factor behind it, blended on it; the engine's table and
    its factor on cosines and sines equal them. A ramp of no width is a step."""
    from serve_b200.parts.rotary import rotary_inv_freq, rotary_length

    for dims, base, sc in ((32, 10000.0, (4.0, 64, 8.0, 0.5)), (16, 100.0, (2.0, 16, 8.0, 1.0)), (8, 10000.0, YARN), (64, 1e6, (32.0, 4096, 32.0, 1.0)),
                           (4, 500.0, (0.5, 8, 1.0, 1.0))):
        rot = {"base": base, "dims": dims, "scaling": dict(zip(("factor", "original", "fast", "slow"), sc))}
        plain = P.frequencies(rot)
        raw = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        mine = rotary_inv_freq(dims, base, dict(rot["scaling"], kind="yarn"))
        torch.testing.assert_close(mine.double(), torch.tensor(plain, dtype=torch.float64), rtol=1e-6, atol=0)
        assert abs(rotary_length(dict(rot["scaling"], kind="yarn")) - P.lengthening(rot)) < 1e-12
        if dims == 32:
            kinds = {"kept" if f == r else "slowed" if abs(f - r / sc[0]) < 1e-12 else "between" for f, r in zip(plain, raw)}
            assert kinds == {"kept", "slowed", "between"}
    assert rotary_length(None) == 1.0 and rotary_length({"kind": "linear", "factor": 4.0}) == 1.0


@pytest.mark.parametrize("backend", BACKENDS)
def test_lengthened_rotation_changes_the_scores_of_the_rotated_part_only(backend):
    """With a factor of e^10 the rotated vectors double, so their share of a score is four times as large, the plain share is
    as it was: compared with a mixer whose frequencies are the scaled ones but whose vectors keep their length."""
    m = LAT(2, 8, 8, 16, 24, 0.3, 40, 100.0, (math.exp(10.0), 4096, 1e-9, 1e-10))       # (the ramp lies behind every pair: frequencies stay)
    got, want, w = _mixer_alone(backend, _single("latent_attention", m), [40], loose=2.0)
    plain = {k: v for k, v in m.items() if k != "rot"}
    for stretch, same in ((2.0, True), (1.0, False)):
        w2 = F64(w)
        w2["l0.mix.q"] = w2["l0.mix.q"].view(2, 16, 64).clone()
        w2["l0.mix.q"][:, 8:] *= stretch
        w2["l0.mix.q"] = w2["l0.mix.q"].view(32, 64)
        w2["l0.mix.dkv"] = torch.cat([w2["l0.mix.dkv"][:24], w2["l0.mix.dkv"][24:] * stretch])
        x = torch.randn(40, 64, generator=torch.Generator().manual_seed(6)).bfloat16().double()
        other = _plain_mixer("latent_attention", x, w2, dict(plain, rot={"base": 100.0, "dims": 8}), 1e-5).float()
        assert (float((other - want).abs().max()) < 1e-4 * float(want.abs().max())) == same


def _ff_alone(backend, f, width, seed=11, tweak=None, n=40):
    from serve_b200.models.filezen import _feed_forward_spec

    cfg = _single("retention", RETS[0], f, width)
    w = make_weights(cfg, seed)
    if tweak is not None:
        tweak(w)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(seed + 1)).bfloat16().float()
    got = _run_part(backend, "feed_forward", _feed_forward_spec(f, width, "l0.mlp."), w, x, [n - 7, 1, 6])
    want = P.feed_forward(x.double(), F64(w), "l0.mlp.", f).float()
    return got, want, w, x


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("ff,width", [(96, 64), (70, 100), (1, 48)])
def test_dense_feed_forward_alone(backend, ff, width):
    got, want, _, _ = _ff_alone(backend, DENSE(ff), width)
    torch.testing.assert_close(got, want, atol=2 * _tol(backend, want), rtol=0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("f,width", [(MOE(6, 2, 32, groups=(3, 2), shared=48), 64), (MOE(9, 3, 22, groups=(3, 1), shared=30), 100), (MOE(4, 1, 48), 48),
                                     (MOE(4, 2, 24, groups=(4, 2)), 40), (MOE(5, 5, 30), 40), (MOE(1, 1, 16, shared=8), 32),
                                     (MOE(96, 4, 16, groups=(8, 3)), 64), (MOE(8, 4, 16, groups=(1, 1)), 32)])
def test_experts_alone(backend, f, width):
    """Also: one choice (whose weight is then one), every expert chosen, one expert in all, groups of one expert, one group of
    all, groups across the lanes of a warp, the choice taking up all that the kept groups have. The router's rows are spread so
    that no two scores lie within a rounding."""
    def spread(w):
        w["l0.mlp.router"] = (w["l0.mlp.router"] * 3.0).bfloat16().float()
    got, want, w, x = _ff_alone(backend, f, width, tweak=spread)
    if backend[1] == "float32":
        torch.testing.assert_close(got, want, atol=2 * _tol(backend, want), rtol=0)
    else:
        bad = ((got - want).abs().amax(1) > 4 * _tol(backend, want)).sum()
        assert int(bad) <= 2
    idx, wt = P.chosen_experts(x.double(), F64(w), "l0.mlp.", f)
    assert float((wt.sum(-1) - 1.0).abs().max()) < 1e-6


def test_the_groups_of_the_plain_router_close_experts_that_score_high():
    """The oracle's premise: the second best expert of all is passed over when its group is not kept, and a group counts by its
    best expert, not by the sum of its experts."""
    f = MOE(6, 2, 8, groups=(2, 1))
    w = {"r.router": torch.eye(6).double()}
    for scores, want in (([5.0, 0.0, 0.1, 4.9, 4.8, 4.7], [0, 2]), ([0.0, 1.0, 2.0, 2.1, -9.0, -9.5], [3, 4])):
        idx, _ = P.chosen_experts(torch.tensor([scores]).double(), w, "r.", f)
        assert idx[0].tolist() == want


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("top,groups,keep,experts", [(2, 2, 1, 6), (3, 4, 2, 8), (4, 16, 3, 128), (1, 3, 1, 9), (8, 4, 4, 32), (6, 2, 1, 512)])
def test_expert_choice_with_groups_on_given_scores(backend, top, groups, keep, experts):
    """The choice and its weights alone: every expert gives back the sum of its token times a number of its own, so the output
    names the experts that were chosen and how they were weighed. The scores are far apart, and in half of the tokens the
    best experts are spread over the groups so that most of them are closed."""
    rt, dev = runtime_for(backend)
    g = torch.Generator().manual_seed(experts)
    t, n = 64, 16
    z = torch.stack([torch.randperm(experts, generator=g) for _ in range(t)]).float() * (24.0 / experts)
    for i in range(0, t, 2):
        order = torch.arange(experts).view(groups, -1).T.reshape(-1)           # neighbours in score lie in different groups
        z[i, order] = torch.arange(experts, 0, -1).float() * (24.0 / experts)
    h = torch.zeros(t, n)
    h[:, 0] = 1.0
    w_gu = torch.zeros(experts, 2, n)
    w_gu[:, 0, 0], w_gu[:, 1, 0] = 4.0, 1.0 / (4.0 / (1.0 + math.exp(-4.0)))
    w_down = torch.zeros(experts, n, 1)
    for e in range(experts):
        w_down[e, e % n, 0] = 1.0 + (e // n)
    act = rt.act_dtype
    out = torch.empty(t, n, dtype=act, device=dev)
    with torch.inference_mode():
        rt.kernels.routed_experts(h.to(dev).to(act), z.to(dev), w_gu.to(dev).to(act), w_down.to(dev).to(act), top, out, score="softmax",
                                  renormalise=True, scale_input=False, activation="swiglu", outputs=experts, renormalise_eps=1e-20,
                                  groups=groups, keep_groups=keep)
    f = MOE(experts, top, 1, groups=(groups, keep))
    idx, wt = P.chosen_experts(z.double(), {"r.router": torch.eye(experts).double()}, "r.", f)
    want = torch.zeros(t, n).double()
    for i in range(t):
        for e, c in zip(idx[i].tolist(), wt[i]):
            want[i, e % n] += c * (1.0 + e // n)
    torch.testing.assert_close(out.float().cpu(), want.float(), atol=(1e-4 if backend[1] == "float32" else 0.02) * float(want.max()), rtol=0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width", [64, 100, 1024, 1030])
def test_norm_behind_the_sublayer_joins_the_stream_in_the_reader(backend, width):
    """x += m * rms(a) * w inside the step that hands the stream on: as it is (the sub-layers' reader) and normalised (the final
    one, for chosen rows, the stream left alone). Also with nothing pending, a plain tensor pending and another norm's output."""
    rt, dev = runtime_for(backend)
    g = torch.Generator().manual_seed(width)
    eps, mult, t = 1e-3, 0.37, 9
    post = build_part("norm", PartSpec("grouped_rms", {"size": width, "eps": eps, "weight_name": "n", "multiplier": mult}), rt)
    final = build_part("norm", PartSpec("grouped_rms", {"size": width, "eps": eps, "weight_name": "f"}), rt)
    reader = build_part("norm", PartSpec("identity", {"size": width}), rt)
    wt = {n: (1.0 + 0.3 * torch.randn(width, generator=g)).bfloat16().float() for n in "nf"}
    for part in (post, final):
        part.load({n: v.to(dev).to(rt.act_dtype) for n, v in wt.items()})
    x0 = torch.randn(t, width, generator=g) * 3.0
    a = (torch.randn(t, width, generator=g) * 0.05).bfloat16().float()
    joined = x0.double() + mult * P.unit_rms(a.double(), eps) * wt["n"].double()
    tol = (3e-6 if backend[1] == "float32" else 2.0 ** -8) * float(joined.abs().max())
    act = lambda v: v.to(dev).to(rt.act_dtype)
    x = x0.clone().to(dev)
    torch.testing.assert_close(reader.forward(x, None, None).float().cpu(), x0, atol=tol, rtol=0)
    out = reader.forward(x, DeferredNorm(act(a), post), None)
    torch.testing.assert_close(out.float().cpu(), joined.float(), atol=tol, rtol=0)
    torch.testing.assert_close(x.cpu(), joined.float(), atol=3e-6 * float(joined.abs().max()), rtol=0)      # the stream itself stays in 32-bit
    x = x0.clone().to(dev)
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device=dev)
    got = final.forward_rows(x, DeferredNorm(act(a), post), rows, None).float().cpu()
    torch.testing.assert_close(got, (P.unit_rms(joined, eps) * wt["f"].double())[[7, 0, 3]].float(), atol=tol, rtol=0)
    torch.testing.assert_close(reader.forward_rows(x, DeferredNorm(act(a), post), rows, None).float().cpu(), joined[[7, 0, 3]].float(), atol=tol, rtol=0)
    assert torch.equal(x.cpu(), x0)
    torch.testing.assert_close(reader.forward(x, act(a), None).float().cpu(), x0 + a, atol=tol, rtol=0)


# ---- rows of another layer ------------------------------------------------------------------------------------------
def _pair(maker, reader, width=32, between=None):
    layers = [LATENT(maker, None)] + ([between] if between else []) + [LATENT(dict(reader, kv_from=0), None)]
    return {"architecture": "Filezen", "width": width, "vocab": 60, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0}, "residual_mult": 0.8, "layers": layers}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("rank", [24, 260], ids=["cached-rows", "per-head"])
@pytest.mark.parametrize("s1,s2", [(5, 40), (40, 5), (9, None), (None, 9), (16, 16)])
def test_a_reader_with_a_mask_of_its_own(tmp_path, backend, rank, s1, s2):
    """A layer that reads another's rows through a shorter, a longer, no and the same window: the owner keeps the pages that
    either can still see. Other heads, head sizes and scales; a retention layer in between. Pages of 8, poisoned, two requests
    side by side in portions and decoded tokens."""
    cfg = _pair(LAT(3, 16, 8, 8, rank, 0.3, s1, 100.0, YARN), LAT(2, 8, 8, 24, rank, 0.4, s2, 100.0, YARN),
                between=RETENTION(RET(8, 8, [0.9], 100.0, 8), None))
    w = make_weights(cfg, 3)
    assert "l2.mix.dkv" not in w and "l2.mix.uk" in w
    folder = write_model(str(tmp_path / "m"), cfg, w, getattr(torch, backend[1]))
    reqs = {f"r{i}": helpers.random_tokens(60, n, seed=i) for i, n in enumerate((75, 41, 20))}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    limits = rounding_limits(w, cfg, reqs, plain) if backend[1] == "bfloat16" else None
    steps = helpers.trace_mixed(reqs, live=2, seed=5, decode_tail=12)
    eng = make_engine(folder, backend, 8, num_pages=helpers.tokens_needed(steps, 8) // 8, max_slots=2)
    for view in eng.stepper.views:
        if view is not None and view.k is not None:
            view.k.fill_(float("nan"))
            view.v.fill_(float("nan"))
    with torch.inference_mode():
        got = helpers.replay(eng, steps)
    eng.kernels.check_errors()
    compare_with_limits(got, plain, backend, limits)
    eng.cache.check()
    if rank == 24:
        assert len(eng.cache.groups) == 1 and eng.cache.groups[0].window == (None if None in (s1, s2) else max(s1, s2))


def test_plain_reader_depends_on_the_makers_rows():
    """The oracle's premise: changing only the maker's down projection changes what the reader gives back."""
    cfg = _pair(LAT(3, 16, 8, 8, 24, 0.3, 9, 100.0), LAT(2, 8, 8, 24, 24, 0.4, 20, 100.0))
    w = F64(make_weights(cfg, 3))
    x = torch.randn(30, 32, generator=torch.Generator().manual_seed(1)).double()
    m = cfg["layers"][1]["mixer"]
    a = P.latent_mixer(x, w, "l1.mix.", m, *P.latent_row(x, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5))
    w["l0.mix.dkv"] = w["l0.mix.dkv"].roll(5, 0)
    b = P.latent_mixer(x, w, "l1.mix.", m, *P.latent_row(x, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5))
    assert float((a - b).abs().max()) > 0.1 * float(a.abs().max())


# ---- what a key far away, at a page's or a window's edge does --------------------------------------------------------
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", [[300], [255, 1, 1, 43], [130] + [1] * 170], ids=["prompt", "portions", "decoded"])
@pytest.mark.parametrize("at,size,rank", [(3, 64, 16), (63, 200, 16), (64, 200, 16), (127, 150, 16), (0, 32, 16), (40, 300, 16), (5, 256, 16), (20, 65, 16),
                                          (100, 128, 250), (10, 2, 16)])
def test_one_key_far_back_at_edges_of_pages_and_windows(backend, cuts, at, size, rank):
    """One key carries a value nobody else has and takes nearly all the weight of every query that sees it. Queries for which it
    lies just inside the window must find it, the next ones must not: both compared with the plain attention, whose difference
    between the two kinds of rows is checked to be large. Pages of 64: the key sits on the last row of a page, the first of the
    next, and hundreds of positions back; rows read as they are cached, and read out per head."""
    m = LAT(2, 16, 8, 16, rank, 0.9, size, 10000.0, (4.0, 64, 8.0, 1.0))
    cfg = _single("latent_attention", m, width=32)
    n = sum(cuts)
    x = torch.randn(n, 32, generator=torch.Generator().manual_seed(at + size)) * 0.5
    x[:, 0] = 0.0
    x[at] = 0.0
    x[at, 0] = 6.0                         # the loud key: one direction, which no other token's input has
    x[:, 1] = 3.0                          # and every query listens through another
    x[at, 1] = 0.0

    def tweak(w, p):
        w[p + "q"][:, :2] = 0.0
        w[p + "q"].view(2, 24, 32)[:, 0, 1] = 3.0          # the first plain channel of every head
        w[p + "dkv"][:, :2] = 0.0
        w[p + "dkv"][0, 0] = 4.0                           # the direction fills the latent's first channel
        w[p + "uk"][:, 0] = 0.0
        w[p + "uk"].view(2, 16, rank)[:, 0, :] = 0.0
        w[p + "uk"].view(2, 16, rank)[:, 0, 0] = 1.0
        w[p + "uv"].view(2, 16, rank)[:, :, 0] = 1.5

    got, want, _ = _mixer_alone(backend, cfg, cuts, x=x, tweak=tweak, page=64, loose=2.0)
    seen = [i for i in range(at + 1, n) if P.visible(i, at, size)]
    unseen = [i for i in range(at + 1, n) if not P.visible(i, at, size)]
    assert seen, "the case has no query that sees the key"
    if unseen:      # (against the float32 bound: that run is the sharp one)
        assert float((want[seen[-1]] - want[unseen[0]]).abs().max()) > 100 * _tol(("", "float32"), want), "the key does not stand out"


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", [[200], [128, 2, 1, 69], [64] + [1] * 136], ids=["prompt", "portions", "decoded"])
def test_a_state_remembers_a_token_far_back(backend, cuts):
    """A head with a decay of one reads, 190 tokens later, what one loud token left; a head with a fast decay has lost it. The
    first tokens of the sequence, whose state is almost empty, are compared too."""
    m = RET(16, 16, [1.0, 0.8], 1e6, 4)
    cfg = _single("retention", m, width=32, eps=1e-2)
    n = sum(cuts)
    x = torch.randn(n, 32, generator=torch.Generator().manual_seed(4)) * 0.5
    x[:, :2] = 0.0
    x[:, 1] = 2.0
    x[9, 0] = 8.0

    def tweak(w, p):
        for name in ("q", "k", "v"):
            w[p + name][:, :2] = 0.0
        w[p + "q"][8::16, 1] = 2.0             # an element beyond the rotated ones
        w[p + "k"][8::16, 0] = 2.0
        w[p + "v"][:, 0] = 1.0

    got, want, w = _mixer_alone(backend, cfg, cuts, x=x, tweak=tweak, loose=2.0)
    y = x.clone()
    y[9, 0] = 0.0
    other = P.retention_mixer(y.bfloat16().double(), F64(w), "l0.mix.", m, 1e-2).float()
    assert float((want[-1] - other[-1]).abs().max()) > 100 * _tol(("", "float32"), want)


@pytest.mark.parametrize("backend", BACKENDS)
def test_states_of_a_slot_are_the_next_requests(backend):
    """Retention over a sequence, after another one ran in the same slot and was closed: the matrix state of the earlier one
    (three times as loud) must not reach the later one."""
    from serve_b200.models.filezen import _mixer_spec

    m = RETS[0]
    w = make_weights(_single("retention", m), 8)
    rt, dev = runtime_for(backend)
    part = build_part("mixer", _mixer_spec("retention", m, 64, 1e-2, "l0.mix."), rt)
    part.load({d.name: w[d.name].to(dev).to(rt.act_dtype) for d in part.tensor_decls()})
    mgr = CacheManager([part.cache_need()], [None], 8, 16, 1, 256, device=dev, kv_dtype=rt.act_dtype)
    view = mgr.views()[0]
    x = torch.randn(40, 64, generator=torch.Generator().manual_seed(9)).bfloat16().float()
    outs = []
    with torch.inference_mode():
        for rid, rows in (("first", x * 3.0), ("second", x)):
            mgr.open(rid)
            outs.append(part.forward(rows.to(dev).to(rt.act_dtype), _ctx(rt, dev, [40], [0], [mgr.slot(rid)], mgr, [rid]), view).float().cpu())
            mgr.commit(rid, 40)
            mgr.close(rid)
    want = _plain_mixer("retention", x.double(), F64(w), m, 1e-2).float()
    torch.testing.assert_close(outs[1], want, atol=2 * _tol(backend, want), rtol=0)


# ---- the chunked form of the recurrence -----------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("listed", [True, False], ids=["rows-by-length", "rows-in-order"])
@pytest.mark.parametrize("lens,heads,dk,dv,rot,decay", [
    ([100, 1, 33, 64, 65, 2, 300, 32], 3, 32, 32, 32, [0.97, 0.9, 0.999]), ([40], 2, 64, 96, 16, [1.0, 0.0]), ([200, 70], 2, 20, 24, 8, [0.5, 0.99]),
    ([90, 33], 1, 128, 72, 64, [0.98]), ([500, 1, 1], 4, 16, 16, 0, [0.9, 0.99, 0.999, 1.0]), ([129, 32], 2, 8, 100, 8, [0.8, 0.2]),
    ([128, 257], 2, 128, 128, 128, [0.99, 0.9995])])
def test_recurrence_chunk_by_chunk_in_one_batch(lens, heads, dk, dv, rot, decay, listed):
    """A ragged step on states that hold something already, positions that do not start at zero, slots in another order than
    the rows: read-outs and last states equal the recurrence in float64 on the same bfloat16 operands, for lengths below, at and
    just above the threshold, one and several chunks, and chunks that are filled partly. What enters the recurrence is not rounded
    again, so the agreement is that of 32-bit sums."""
    from types import SimpleNamespace

    from serve_b200.engine.step import BatchShape
    from serve_b200.kernels import load_kernels

    k, dev = load_kernels("cuda:0"), "cuda:0"
    g = torch.Generator().manual_seed(sum(lens))
    t, rows = sum(lens), len(lens)
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    starts = [11 * i + 3 for i in range(rows)]
    proj = torch.randn(t, 2 * heads * dk + 2 * heads * dv, generator=g).bfloat16()
    state0 = torch.randn(rows, heads, dk, dv, generator=g)
    inv = torch.tensor([100.0 ** (-2.0 * i / max(rot, 1)) for i in range(max(rot // 2, 1))])
    order = sorted(range(rows), key=lambda i: -lens[i])
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    shape = BatchShape(rows, t, max(lens), min(lens), 4096, False, rows_by_q=i32(order) if listed else None,
                       neg_q_sorted=tuple(-lens[i] for i in order) if listed else None)
    slots = list(range(rows))[::-1]
    ctx = SimpleNamespace(shape=shape, positions=i32([s + j for n, s in zip(lens, starts) for j in range(n)]),
                          token_row=i32([i for i, n in enumerate(lens) for _ in range(n)]), cu_q=i32(cu), slots=i32(slots), memo={})
    q, kk, v = proj[:, : heads * dk], proj[:, heads * dk: 2 * heads * dk], proj[:, 2 * heads * dk: 2 * heads * dk + heads * dv]
    on = proj.to(dev)
    part = lambda a, n: on[:, a: a + n]
    state = state0.to(dev)
    out = torch.full((t, heads * dv), float("nan"), device=dev)
    before = k.launches
    k.linear_recurrence("retention", part(0, heads * dk), part(heads * dk, heads * dk), part(2 * heads * dk, heads * dv), state, ctx, out, heads, heads,
                        dk, dv, decay=torch.tensor(decay, device=dev), inv_freq=inv.to(dev), rot_dims=rot, k_scale=dk ** -0.5)
    assert k.launches - before == 3 + (1 if rot else 0) + (2 if min(lens) <= k.CHUNKED_FROM else 0)
    for r, n in enumerate(lens):
        sl = slice(cu[r], cu[r + 1])
        ang = (torch.arange(n) + starts[r]).float()[:, None] * inv[None, : rot // 2]          # (angles are 32-bit)
        c, sn = ang.double().cos()[:, None], ang.double().sin()[:, None]

        def turn(z):
            z = z[sl].double().view(n, heads, dk)
            a, b = z[..., : rot // 2], z[..., rot // 2: rot]
            return torch.cat([a * c - b * sn, b * c + a * sn, z[..., rot:]], -1)

        qq, ke, ve = turn(q), turn(kk) * dk ** -0.5, v[sl].double().view(n, heads, dv)
        S = state0[slots[r]].double()
        want = torch.zeros(n, heads, dv).double()
        for i in range(n):
            S = torch.tensor(decay).double()[:, None, None] * S + ke[i][:, :, None] * ve[i][:, None, :]
            want[i] = torch.einsum("hkv,hk->hv", S, qq[i])
        torch.testing.assert_close(out[sl].cpu().double(), want.view(n, heads * dv), atol=3e-5 * float(want.abs().max()), rtol=0)
        torch.testing.assert_close(state[slots[r]].cpu().double(), S, atol=2e-5 * float(S.abs().max()), rtol=0)


# ---- the sizes of a real layer, and the programs a user starts ----------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_as_wide_as_a_real_models(tmp_path, dtype):
    """Heads of 64 and 128, a latent row of 192 + 64, experts and dense widths that are multiples of 64: the products take
    the tensor-core paths, the attention its widest heads; prompts of several hundred tokens, portions and decoded tails."""
    cfg = CONFIGS["wide"]
    w = make_weights(cfg, 31, expert_gain=0.3)
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=40 + i) for i, n in enumerate([300, 130, 17])}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    limits = rounding_limits(w, cfg, reqs, plain) if dtype == "bfloat16" else None
    folder = write_model(str(tmp_path / "wide"), cfg, w, getattr(torch, dtype))
    backend = ("cuda", dtype)
    for steps, graphs in ((helpers.trace_whole(reqs), False), (helpers.trace_tail_decode(reqs, tail=40), True),
                          (helpers.trace_portions(reqs, sizes=(64, 2, 130, 1, 33)), False)):
        eng = make_engine(folder, backend, 64, num_pages=16, graphs=graphs, budget=1024, context=512)
        with torch.inference_mode():
            got = helpers.replay(eng, steps)
        eng.kernels.check_errors()
        compare_with_limits(got, plain, backend, limits)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_folder_of_this_design(tmp_path, dtype):
    import numpy as np

    cfg = CONFIGS["q"]
    w = make_weights(cfg, 17, expert_gain=0.5)
    folder = write_model(str(tmp_path / "m"), cfg, w, torch.bfloat16)
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=70 + i) for i, n in enumerate([70, 9, 33, 150, 2])}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    limits = rounding_limits(w, cfg, reqs, plain) if dtype == "bfloat16" else None
    steps = helpers.trace_mixed(reqs, live=4, seed=3)
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                           "--max-tokens", str(helpers.tokens_needed(steps, 64))],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    got, at = {}, {}
    for s in steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        i = 0
        for e in s["entries"]:
            for wnt in e["want"]:
                got[(e["id"], at.get(e["id"], 0) + wnt)] = torch.from_numpy(rows[i].copy())
                i += 1
            at[e["id"]] = at.get(e["id"], 0) + len(e["tokens"])
    compare_with_limits(got, plain, ("cuda", dtype), limits)


# ---- configurations nobody chose ---------------------------------------------------------------------------------
def _random_config(rng) -> dict:
    """A model of this design drawn at random: widths and vocabularies that are no power of two, 3 to 6 layers in any order with
    at least one of each mixer, head sizes that are and are not multiples of 16, value heads smaller and larger than the keys',
    latent rows from 20 numbers to more than the attention kernels take, readers of any earlier layer's rows, windows from one
    key to longer than the prompts, scaled and plain frequencies, states of 8 to 128 rows wholly, partly and not rotated, 2 to 64
    experts with 1 to 8 choices, with and without groups and a shared expert, layers without a feed-forward."""
    def lat(made):
        if made and rng.random() < 0.5:
            j = rng.choice(list(made))
            like = made[j]
        else:
            j, like = None, None
        rot = like["rot_dim"] if like else rng.choice([4, 8, 16, 32, 64])
        m = {"heads": rng.choice([1, 2, 3, 4, 8]), "dim": rng.choice([16, 32, 64]), "rot_dim": rot, "vdim": rng.choice([16, 24, 64, 80]),
             "kv_rank": like["kv_rank"] if like else rng.choice([16, 24, 40, 64, 100, 192, 288])}
        m["scale"] = rng.choice([1.0, 2.0]) / (m["dim"] + rot) ** 0.5
        m["rot"] = copy.deepcopy(like["rot"]) if like else {"base": rng.choice([100.0, 10000.0]), "dims": rot}
        if like is None and rng.random() < 0.7:
            m["rot"]["scaling"] = {"factor": rng.choice([2.0, 8.0, 32.0]), "original": rng.choice([16, 64, 2048]), "fast": rng.choice([8.0, 32.0]), "slow": 1.0}
        if rng.random() < 0.85:
            m["mask"] = {"size": rng.choice([1, 7, 38, 64, 65, 130, 1000])}
        if j is not None:
            m["kv_from"] = j
        return m

    def ret():
        dim, heads = rng.choice([8, 16, 20, 32, 64, 128]), rng.choice([1, 2, 3, 4])
        m = {"heads": heads, "dim": dim, "vdim": rng.choice([dim, 16, 40, 64]), "decay": [rng.choice([0.5, 0.9, 0.97, 0.99, 0.999]) for _ in range(heads)]}
        if rng.random() < 0.85:
            m["rot"] = {"base": rng.choice([100.0, 10000.0, 1e6]), "dims": rng.choice([d for d in (4, 8, 16, 32, 64) if d <= dim] + [dim])}
        return m

    def mlp():
        r = rng.random()
        if r < 0.15:
            return None
        if r < 0.4:
            return DENSE(rng.choice([64, 90, 128, 333]))
        experts = rng.choice([2, 4, 6, 8, 16, 64])
        count = rng.choice([g for g in (1, 2, 4, 8) if experts % g == 0])
        keep = rng.randint(1, count)
        top = rng.choice([t for t in (1, 2, 3, 4, 8) if t <= keep * (experts // count)])
        return MOE(experts, top, rng.choice([16, 24, 64]), (count, keep) if rng.random() < 0.8 else None, rng.choice([None, 16, 96]))

    kinds = ["latent", "retention"] + [rng.choice(["latent", "latent", "retention"]) for _ in range(rng.randint(1, 4))]
    rng.shuffle(kinds)
    layers, made = [], {}
    for i, k in enumerate(kinds):
        if k == "latent":
            layers.append(LATENT(lat(made), mlp()))
            if "kv_from" not in layers[-1]["mixer"]:
                made[i] = layers[-1]["mixer"]
        else:
            layers.append(RETENTION(ret(), mlp()))
    return {"architecture": "Filezen", "width": rng.choice([72, 96, 100, 128, 136, 200, 264]), "vocab": rng.choice([131, 257, 500, 1000]),
            "norm": {"eps": rng.choice([1e-3, 1e-5])}, "embedding": {"scale": rng.choice([1.0, 2.5, 8.0])},
            "residual_mult": rng.choice([0.3, 0.7, 1.0]), "layers": layers}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_random_configuration(tmp_path, seed, dtype):
    """Five requests of 2 to 330 tokens in pages of 64, whole, with decoded tails from CUDA graphs, in portions and as mixed batches
    of four live requests on a pool without a spare page, against the plain implementation."""
    rng = random.Random(seed)
    cfg = _random_config(rng)
    w = make_weights(cfg, seed, expert_gain=0.3)
    folder = write_model(str(tmp_path / "m"), cfg, w, getattr(torch, dtype))
    lens = [rng.choice([2, 3, 17, 64, 65, 130, 200, 257, 330]) for _ in range(5)]
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=seed * 10 + i) for i, n in enumerate(lens)}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    limits = rounding_limits(w, cfg, reqs, plain) if dtype == "bfloat16" else None
    backend = ("cuda", dtype)
    cuts = {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_tail_decode(r, tail=70),
            "portions": lambda r: helpers.trace_portions(r, sizes=(64, 2, 130, 1, 33, 5)), "mixed": lambda r: helpers.trace_mixed(r, live=4, seed=seed)}
    for cut, make in cuts.items():
        steps = make(reqs)
        pages = helpers.tokens_needed(steps, 64) // 64
        eng = make_engine(folder, backend, 64, num_pages=pages, max_slots=4, graphs=(cut == "tail"), budget=max(512, pages * 64), context=pages * 64)
        for v in eng.stepper.views:
            if v is not None and v.k is not None:
                v.k.fill_(float("nan"))
                v.v.fill_(float("nan"))
        with torch.inference_mode():
            got = helpers.replay(eng, steps)
        eng.kernels.check_errors()
        try:
            compare_with_limits(got, plain, backend, limits, allow=len(got) // 8)
        except AssertionError as e:
            raise AssertionError(f"{cut}: {json.dumps(cfg)}: {e}") from None
        assert eng.cache.live == 0
