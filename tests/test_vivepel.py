"""The Vivepel decoder in the engine against the plain implementation of tests/plain/vivepel_plain.py.

Every test runs on the CPU over the torch stand-ins of the kernels (which checks the parts, the cache manager, the step
function and the scheduler) and, marked gpu, on the real kernels in float32 and bfloat16.
"""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

from serve_b200.config import ConfigError, PartSpec, build_spec, config_from_dict
from serve_b200.parts import DeferredNorm, build_part
from tests import helpers
from tests.plain import vivepel_plain as P
from tests.test_bapavik import _ctx, _run_part, _tol
from tests.vivepel_cases import ATT, BACKENDS, CONFIGS, LAYER, compare_rows, make_engine, make_weights, plain_logits, runtime_for, write_model

LENGTHS = {"a": [1, 5, 23, 49, 75, 130], "o": [3, 40, 90, 17], "q": [2, 9, 31, 64, 101]}
PAGE = {"a": 8, "o": 4, "q": 16}
F64 = lambda w: {k: v.double() for k, v in w.items()}
CUDA = [b for b in BACKENDS if b.id != "emu"]


# ---- configuration and description ----------------------------------------------------------------------------
def test_configuration_is_read_from_the_file_and_describes_every_layer():
    for raw in CONFIGS.values():
        cfg = config_from_dict(copy.deepcopy(raw))
        assert type(cfg).__name__ == "VivepelConfig" and (cfg.width, cfg.vocab, cfg.groups) == (raw["width"], raw["vocab"], raw["norm"]["groups"])
        spec = build_spec(cfg)
        assert len(spec.layers) == len(raw["layers"]) == len(spec.schedule) and not spec.head.params.get("tied_to")
        for layer, ls in zip(raw["layers"], spec.layers):
            assert ls.block.kind == "sandwich_norm" and ("feed_forward" in ls.parts) == (layer["mlp"] is not None)
            p, m = ls.parts["mixer"].params, layer["mixer"]
            assert (p["heads"], p["kv_heads"], p["dim"], p["scale"]) == (m["heads"], m["kv_heads"], m["dim"], m["scale"])
            assert p["softcap"] == m.get("softcap") and p["chunk"] == (m.get("mask") or {}).get("size") and p["sink_score"] == 0.0
            assert p["position"].kind == ("rotary" if m.get("rot") else "none")
            assert ls.parts["mixer_post_norm"].params["scale_name"] == "ls1" and ls.parts["mixer_norm"].params["groups"] == raw["norm"]["groups"]
        assert config_from_dict(cfg.to_dict()) == cfg


@pytest.mark.parametrize("breaker", [
    lambda c: c["layers"][0].update(type="conv"),
    lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"].update(heads=3),
    lambda c: c["layers"][0]["mixer"].update(vdim=16),
    lambda c: c["layers"][0]["mixer"].update(softcap=-1.0),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26),
    lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 2.0, "low": 1.0, "high": 4.0, "original": 64}),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][0]["mlp"].pop("ff"),
    lambda c: c["norm"].update(groups=3),
    lambda c: c["norm"].update(eps=0.0),
    lambda c: c.pop("vocab"),
    lambda c: c.update(layers=[]),
])
def test_configuration_refuses_what_it_cannot_run(breaker):
    raw = copy.deepcopy(CONFIGS["a"])
    breaker(raw)
    with pytest.raises(ConfigError):
        config_from_dict(raw)


# ---- whole models ---------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """{config name: {dtype: (weights, requests, plain logits, model folder)}}."""
    out = {}
    for name in LENGTHS:
        cfg = CONFIGS[name]
        reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=20 + i) for i, n in enumerate(LENGTHS[name])}
        w = make_weights(cfg, 100 + len(name))
        plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
        out[name] = {dt: (w, reqs, plain, write_model(str(tmp_path_factory.mktemp(f"{name}-{dt}")), cfg, w, getattr(torch, dt)))
                     for dt in ("float32", "bfloat16")}
    return out


def test_plain_layers_feed_one_another(models):
    """The oracle's own premise: every layer changes the residual stream, and the last position of a block depends on the block's
    first token."""
    for name in LENGTHS:
        w, reqs, plain, _ = models[name]["float32"]
        cfg, toks = CONFIGS[name], reqs["r2"]
        layers = []
        plain_logits(w, cfg, toks, layers)
        for a, b in zip(layers, layers[1:]):
            assert float((a - b).abs().max()) > 1e-2
        other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
        assert float((plain_logits(w, cfg, other)[6] - plain["r2"][6]).abs().max()) > 1e-3


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["a", "o", "q"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "pairs", "single_tokens"])
def test_cuts_match_plain(models, name, backend, cut):
    w, reqs, plain, folder = models[name][backend[1]]
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
    compare_rows(got, plain, backend)
    eng.cache.check()
    assert eng.cache.live == 0


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["a", "o", "q"])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, backend):
    """Unequal requests side by side, portions beside single tokens, fewer slots and pages than the requests need in all: every
    row must equal the request run alone. Pages are poisoned first, so that a page that is read without having been written shows."""
    w, reqs, plain, folder = models[name][backend[1]]
    page = PAGE[name]
    steps = helpers.trace_mixed(reqs, live=3, seed=7)
    need = helpers.tokens_needed(steps, page) // page
    assert need < sum(-(-len(t) // page) for t in reqs.values())
    eng = make_engine(folder, backend, page, num_pages=need, max_slots=3, context=160)
    for view in eng.stepper.views:
        view.k.fill_(float("nan"))
        view.v.fill_(float("nan"))
    with torch.inference_mode():
        got = helpers.replay(eng, steps)
    eng.kernels.check_errors()
    compare_rows(got, plain, backend)
    eng.cache.check()
    assert eng.cache.live == 0 and eng.cache.free_slots == 3
    assert max(g.pool.high_water for g in eng.cache.groups) <= need


def test_pages_behind_a_block_of_positions_are_given_back(models):
    """A request of 130 tokens in blocks of at most 33 positions and pages of 8 never holds more pages than a block and a portion
    can touch."""
    w, reqs, plain, folder = models["a"]["float32"]
    eng = make_engine(folder, ("emu", "float32"), 8, num_pages=40)
    with torch.inference_mode():
        got = helpers.replay(eng, helpers.trace_portions({"r5": reqs["r5"]}, sizes=(7, 1, 2)))
    compare_rows(got, plain, ("emu", "float32"))
    for g in eng.cache.groups:
        assert g.pool.high_water <= (g.chunk + 7 - 2) // 8 + 2 < 130 // 8


@pytest.mark.parametrize("backend", BACKENDS)
def test_long_decoding_side_by_side(models, backend):
    """Two requests decoded one token at a time for 120 steps after short prompts (from CUDA graphs on the GPU): block after block
    of positions begins and ends on decoded tokens, pages are crossed and given back."""
    cfg = CONFIGS["a"]
    w, _, _, folder = models["a"][backend[1]]
    seqs = {f"d{i}": helpers.random_tokens(cfg["vocab"], 140 - 9 * i, seed=60 + i) for i in range(2)}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in seqs.items()}
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
    compare_rows(got, plain, backend)


@pytest.mark.parametrize("backend", BACKENDS)
def test_greedy_generation_through_the_scheduler(models, backend):
    """generate(): the engine's own entry point, scheduler and sampler. Every generated token must be (within the tolerance) the
    best one of the plain model given the tokens before it."""
    from serve_b200.run import Request, generate

    cfg = CONFIGS["a"]
    w, reqs, _, folder = models["a"][backend[1]]
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


# ---- the attention alone ----------------------------------------------------------------------------------------
CUTS = [[57], [30, 1, 1, 2, 5, 17, 1], [1] * 57]


def _mixer_alone(backend, m, cuts, width=64, seed=5, x=None, tweak=None, page=8, loose=1.0, pages=128, eps=1e-5):
    from serve_b200.models.vivepel import _mixer_spec

    cfg = {"architecture": "Vivepel", "width": width, "vocab": 50, "norm": {"eps": eps, "groups": 1}, "layers": [LAYER(m, None)]}
    w = make_weights(cfg, seed)
    if tweak is not None:
        tweak(w, "l0.mix.")
    if x is None:
        x = torch.randn(sum(cuts), width, generator=torch.Generator().manual_seed(seed + 1))
    x = x.bfloat16().float()
    want = P.attention_mixer(x.double(), F64(w), "l0.mix.", m, eps).float()
    got = _run_part(backend, "mixer", _mixer_spec(m, width, eps, "l0.mix."), w, x, cuts, page=page, pages=pages)
    torch.testing.assert_close(got, want, atol=_tol(backend, want) * loose, rtol=0)
    return got, want, w


# One head; as many key/value heads as heads, one for all; 17 and 40 heads (more than one, more than two product tiles of the
# mixing matrix; groups of more than 16 heads, whose decoding steps take the prompts' kernels); head sizes that are no multiple
# of 16, an odd multiple of 16, and the largest; no rotation, all of a head; no cap, a cap that bends everything; no mask, blocks
# of one, two, a page, and more positions than there are.
ATTS = [ATT(4, 2, 24, 0.3, 5.0, 20, 10000.0, 16), ATT(1, 1, 16, 0.4, 8.0, 13, 100.0, 16), ATT(5, 5, 12, 0.5, 1.0, 8, 3000.0, 10),
        ATT(6, 1, 48, 0.2, None, None, None, None), ATT(17, 17, 16, 0.3, 12.0, 2, 100.0, 4), ATT(40, 2, 16, 0.3, 30.0, 1000, 700.0, 8),
        ATT(40, 10, 32, 0.25, 3.0, 64, 700.0, 32), ATT(2, 1, 256, 0.06, 20.0, 30, 500.0, 64), ATT(3, 1, 80, 0.1, 0.5, 1, 500.0, 80),
        ATT(70, 7, 16, 0.3, 6.0, 33, 90.0, 6), ATT(8, 8, 112, 0.1, 25.0, None, 10000.0, 28)]
WIDTHS = (64, 100, 48, 40, 72, 56, 64, 80, 36, 96, 64)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", CUTS, ids=["whole", "portions", "tokens"])
@pytest.mark.parametrize("which", range(len(ATTS)))
def test_attention_alone(backend, cuts, which):
    _mixer_alone(backend, ATTS[which], cuts, width=WIDTHS[which])


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("page", [4, 16, 48, 64, 128])
def test_pages_of_other_sizes(backend, page):
    _mixer_alone(backend, ATT(6, 2, 32, 0.25, 9.0, 90, 10000.0, 16), [150, 1, 30, 2, 1, 1, 70], page=page)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size", [None, 700], ids=["all-keys", "blocks-of-700"])
def test_hundreds_of_keys_with_few_rows(backend, size):
    """A decoded token, two and three tokens over several hundred keys: the keys of a step with few rows are dealt to several thread
    blocks whose sums are merged."""
    _mixer_alone(backend, ATT(4, 2, 32, 0.3, 10.0, size, 10000.0, 16), [611, 1, 1, 2, 3, 1, 90, 1, 2], page=64, pages=32)


def _loud_key(x, at, rows, gain=6.0):
    """Make position ``at`` a key that the queries of ``rows`` put nearly all their weight on if they see it: its input is one
    direction that the key projection maps to a large key, and those queries' inputs share it."""
    direction = torch.zeros(x.shape[1])
    direction[0] = 1.0
    x[at] = direction * gain
    for r in rows:
        x[r] = x[r] * 0.3 + direction * gain


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", [[300], [255, 1, 1, 43], [130] + [1] * 170], ids=["prompt", "portions", "decoded"])
@pytest.mark.parametrize("at,size", [(3, 64), (63, 64), (64, 65), (127, 150), (149, 150), (150, 151), (40, None), (0, 299), (100, 101)])
def test_one_key_at_the_edges_of_blocks_and_pages(backend, cuts, at, size):
    """One key carries a value nobody else has. Queries of its block (to the block's last position) must find it, those from the next
    block's first position on must not, although the next block's queries ask for it as loudly. Pages of 64: the key sits on the last
    row of a page, the first of the next, on a block's last and first position, and hundreds of positions back."""
    m = ATT(2, 1, 16, 1.2, 25.0, size, 10000.0, 8)
    n = sum(cuts)
    x = torch.randn(n, 32, generator=torch.Generator().manual_seed(at)) * 0.5
    _loud_key(x, at, [r for r in range(at + 1, n)])
    for r in range(at + 1, n):
        x[r, 1:] = 0.5 * x[r, 1:]

    def tweak(w, p):
        for name in ("q", "k"):
            w[p + name + ".b"].zero_()
            w[p + name][:, 0] = 0.0
            w[p + name][9::16, 0] = 1.0        # a channel that is not rotated listens to the direction
            w[p + name][9::16, 1:] = 0.0
        w[p + "k"][12, :] = 0.0
        x[at, 2] = 8.0
        w[p + "k"][12, 2] = 3.0               # and this one's value nobody else has
        x[at + 1:, 2] = 0.0

    _, want, _ = _mixer_alone(backend, m, cuts, width=32, x=x, tweak=tweak, page=64)
    seen = [i for i in range(at + 1, n) if P.visible(i, at, size)]
    unseen = [i for i in range(at + 1, n) if not P.visible(i, at, size)]
    if seen and unseen:      # (against the float32 bound: that run is the sharp one)
        assert float((want[seen[-1]] - want[unseen[0]]).abs().max()) > 30 * _tol(("", "float32"), want), "the key does not stand out"


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("cuts", [[40], [1] * 40], ids=["prompt", "decoded"])
def test_one_is_added_to_the_denominator(backend, cuts):
    """Scores pushed far below zero leave nearly all weight with the added one (the heads' outputs all but vanish: the softmax without
    it would not notice); pushed far above, it takes nothing, and the first token's output is its own value."""
    m = ATT(2, 2, 16, 1.0, 40.0, 30, 10000.0, 8)
    outs = {}
    for name, sign in (("low", -1.0), ("high", 1.0)):
        def tweak(w, p, sign=sign):
            w[p + "talk"] = torch.eye(2)
            w[p + "o"] = torch.eye(32)
            for n in ("q", "k"):
                w[p + n].mul_(0.1)                      # the biases decide: every query meets every key alike
                w[p + n + ".b"].zero_()
                w[p + n + ".b"][10::16] = 4.0 * (sign if n == "q" else 1.0)
        # (scores of -16: the low outputs are e^-16 of a value, and the error of the exponent shows in all of their digits)
        outs[name] = _mixer_alone(backend, m, cuts, width=32, tweak=tweak, loose=1.0 if name == "high" else 8.0)[1]
    assert float(outs["low"].abs().max()) < 0.02 * float(outs["high"].abs().max())
    assert float(outs["high"][0, 10]) > 3.5             # (the value of the first key as projected, not the normalised key)


@pytest.mark.parametrize("backend", BACKENDS)
def test_values_are_the_keys_as_projected(backend):
    """A key norm weight scaled per element and rotated keys change the scores, never the values: with the mixing matrix at the identity
    and scores all alike (a cap near zero), a head's output is the mean of the biased projections, weighed 1 / (n + 1)."""
    m = ATT(2, 1, 16, 1.0, 1e-3, 50, 10.0, 16)

    def tweak(w, p):
        w[p + "talk"] = torch.eye(2)
        w[p + "o"] = torch.eye(32)
        w[p + "k.norm"] = torch.linspace(0.25, 4.0, 16).bfloat16().float()
    got, want, w = _mixer_alone(backend, m, [20, 1, 9], width=32, tweak=tweak)
    x = torch.randn(30, 32, generator=torch.Generator().manual_seed(6)).bfloat16().double()
    v = x @ w["l0.mix.k"].double().T + w["l0.mix.k.b"].double()
    mean = v.cumsum(0) / torch.arange(2, 32)[:, None]
    torch.testing.assert_close(want[:, :16].double(), mean, atol=3e-3 * float(mean.abs().max()), rtol=0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("heads,kv", [(4, 2), (20, 4), (33, 3)])
def test_mixing_moves_weights_between_heads(backend, heads, kv):
    """A mixing matrix with one entry per row, off the diagonal, with signs and sizes of their own: head h carries another head's weights
    (from another key/value head, too) to the values of its own key/value head. The transposed matrix gives something else."""
    m = ATT(heads, kv, 16, 0.8, 15.0, 40, 10000.0, 8)
    perm = [(5 * h + 3) % heads for h in range(heads)] if heads % 5 else [(7 * h + 3) % heads for h in range(heads)]
    assert sorted(perm) == list(range(heads))
    gain = [(-1.0) ** h * (0.5 + h / heads) for h in range(heads)]

    def tweak(w, p):
        t = torch.zeros(heads, heads)
        for h in range(heads):
            t[h, perm[h]] = gain[h]
        w[p + "talk"] = t.bfloat16().float()
    _, want, w = _mixer_alone(backend, m, [50, 1, 1, 9], tweak=tweak)
    other = F64(w)
    other["l0.mix.talk"] = other["l0.mix.talk"].T
    x = torch.randn(61, 64, generator=torch.Generator().manual_seed(6)).bfloat16().double()
    assert float((P.attention_mixer(x, other, "l0.mix.", m, 1e-5).float() - want).abs().max()) > 0.1 * float(want.abs().max())


@pytest.mark.parametrize("backend", CUDA)
def test_runs_of_tokens_in_a_bounded_scratch_buffer(backend, monkeypatch):
    """A scratch buffer that holds a few tokens only: the step runs in pieces that end inside portions, tiles and requests of few
    rows, with the same result."""
    from serve_b200.kernels import CudaKernels

    m = ATT(6, 2, 32, 0.3, 10.0, 90, 10000.0, 16)
    cuts = [150, 2, 3, 1, 70]
    whole = _mixer_alone(backend, m, cuts, page=64)[0]
    for tokens in (1, 7, 40):
        monkeypatch.setattr(CudaKernels, "TALK_SCRATCH_BYTES", tokens * 6 * 192 * 9)
        torch.testing.assert_close(_mixer_alone(backend, m, cuts, page=64)[0], whole, atol=0, rtol=0)


@pytest.mark.parametrize("backend", CUDA)
@pytest.mark.parametrize("heads,kv,dim,chunk,ps,cap,gain", [
    (8, 2, 64, 100, 32, 8.0, 2.0), (32, 8, 128, 0, 32, 0.0, 2.0), (5, 1, 48, 64, 32, 8.0, 2.0), (40, 2, 16, 130, 32, 100.0, 2.0),
    (16, 4, 128, 65, 16, 50.0, 1.0), (6, 2, 64, 0, 256, 8.0, 30.0), (4, 4, 64, 64, 8, 100.0, 30.0), (12, 1, 128, 150, 64, 3.0, 2.0),
    (34, 2, 64, 90, 128, 0.0, 30.0)])
def test_a_batch_of_unequal_requests_is_each_alone(backend, heads, kv, dim, chunk, ps, cap, gain):
    """The kernels themselves on a batch of decoded tokens, short and long portions (some shapes take the prompts' kernels, some the
    decoding ones), against the stand-in; and the same rows for every request whatever stands beside it. Caps that bound every
    exponential, caps that do not, none; scores far inside a cap, at it, and (gain 30) far beyond what an exponential holds."""
    from serve_b200.engine.step import BatchShape
    from tests.emu_kernels import EmuKernels

    rt, dev = runtime_for(backend)
    q_lens, lens = [1, 290, 3, 1, 17, 2, 1, 70], [200, 340, 64, 33, 17, 129, 1, 70]
    g = torch.Generator().manual_seed(3)
    pages = [-(-n // ps) for n in lens]
    order = torch.randperm(sum(pages), generator=g).tolist()
    width = max(pages)
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    for r, n in enumerate(pages):
        for b in range(n):
            table[r, b] = order.pop()
    rnd = lambda *s: torch.randn(*s, generator=g).to(rt.act_dtype)
    kc, vc = rnd(sum(pages), kv, ps, dim), rnd(sum(pages), kv, ps, dim)
    for r, n in enumerate(lens):                 # what lies in a page behind a sequence's end is no number
        kc[table[r, pages[r] - 1], :, n - (pages[r] - 1) * ps:] = float("nan")
        vc[table[r, pages[r] - 1], :, n - (pages[r] - 1) * ps:] = float("nan")
    q = rnd(sum(q_lens), heads * dim)
    talk = (torch.eye(heads) + 0.3 * torch.randn(heads, heads, generator=g)).to(rt.act_dtype)
    if rt.act_dtype == torch.bfloat16:
        n = 16 * -(-heads // 16)
        padded = torch.zeros(n, n, dtype=talk.dtype)
        padded[:heads, :heads] = talk
        talk = padded
    sinks = torch.randn(heads, generator=g)

    def run(rows, kernels, device):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)
        at = [sum(q_lens[:r]) for r in rows]
        ql, kl = [q_lens[r] for r in rows], [lens[r] for r in rows]
        cu = [0]
        for n in ql:
            cu.append(cu[-1] + n)
        pos = [kl[i] - ql[i] + j for i in range(len(rows)) for j in range(ql[i])]
        qq = torch.cat([q[a: a + n] for a, n in zip(at, ql)]).to(device)
        by_q = sorted(range(len(rows)), key=lambda i: -ql[i])
        shape = BatchShape(len(rows), len(pos), max(ql), min(ql), max(kl), False, rows_by_q=i32(by_q), neg_q_sorted=tuple(-ql[i] for i in by_q))
        out = torch.full((len(pos), heads * dim), float("nan"), dtype=rt.act_dtype, device=device)
        kernels.talking_attention(qq, kc.to(device), vc.to(device), table[rows].to(device), i32(cu), i32(kl), i32(pos), heads, kv, dim, ps,
                                  gain / dim ** 0.5, talk.to(device), out, shape, chunk=chunk, softcap=cap, sinks=sinks.to(device))
        return out.float().cpu()

    every = run(list(range(len(lens))), rt.kernels, dev)
    want = run(list(range(len(lens))), EmuKernels("cpu", torch.float64), "cpu")
    torch.testing.assert_close(every, want, atol=_tol(backend, want), rtol=0)
    rt.kernels.check_errors()
    alone = torch.cat([run([r], rt.kernels, dev) for r in range(len(lens))])
    torch.testing.assert_close(every, alone, atol=_tol(backend, want), rtol=0)


# ---- norms and the activation ---------------------------------------------------------------------------------
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size,groups", [(48, 1), (96, 2), (105, 5), (64, 64), (4096, 8), (9000, 3), (20480, 1), (12, 4)])
def test_norm_over_equal_parts_alone_and_behind_another(backend, size, groups):
    """The norm of the stream; with a sub-layer's output added that goes through a norm with a layer scale first, in one kernel; with a
    plain delta; for picked rows; and of a sub-layer's output alone. Parts of very different size must not see one another."""
    rt, dev = runtime_for(backend)
    g = torch.Generator().manual_seed(size)
    x = torch.randn(9, size, generator=g) * torch.repeat_interleave(10.0 ** torch.linspace(-2, 2, groups), size // groups)
    a = (torch.randn(9, size, generator=g) * torch.repeat_interleave(10.0 ** torch.linspace(1, -2, groups), size // groups)).bfloat16().float()
    w = {n: (1.0 + 0.3 * torch.randn(size, generator=g)).bfloat16().float() for n in ("n", "nb", "ls")}
    load = {n: t.to(dev).to(rt.act_dtype) for n, t in w.items()}
    norm = build_part("norm", PartSpec("grouped_rms", {"size": size, "groups": groups, "eps": 1e-4, "weight_name": "n"}), rt)
    post = build_part("norm", PartSpec("grouped_rms", {"size": size, "groups": groups, "eps": 1e-4, "weight_name": "nb", "scale_name": "ls"}), rt)
    norm.load(load), post.load(load)
    n64 = lambda v, name: P.grouped_norm(v, w[name].double(), groups, 1e-4)
    ad = a.to(dev).to(rt.act_dtype)
    added = n64(a.double(), "nb") * w["ls"].double()
    for delta, x_want in ((None, x.double()), (DeferredNorm(ad, post), x.double() + added), (ad, x.double() + a.double())):
        xs = x.clone().to(dev)
        got = norm.forward(xs, delta, None).float().cpu()
        want = n64(x_want, "n").float()
        torch.testing.assert_close(got, want, atol=_tol(backend, want), rtol=0)
        torch.testing.assert_close(xs.cpu(), x_want.float(), atol=1e-5, rtol=1e-5)
        xs = x.clone().to(dev)
        rows = torch.tensor([7, 0, 3], dtype=torch.int32, device=dev)
        got = norm.forward_rows(xs, delta, rows, None).float().cpu()
        torch.testing.assert_close(got, want[[7, 0, 3]], atol=_tol(backend, want), rtol=0)
        assert torch.equal(xs.cpu(), x)
    torch.testing.assert_close(post.apply(ad).cpu(), added.float(), atol=1e-5 * float(added.abs().max()), rtol=1e-5)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("ff,width", [(96, 64), (70, 105), (1, 48), (1000, 64), (5000, 32), (17000, 16), (40000, 16)])
def test_feed_forward_alone(backend, ff, width):
    """Also: one value (N of it is its sign, nearly), and rows longer than a block's registers hold."""
    from serve_b200.models.vivepel import _feed_forward_spec

    g = torch.Generator().manual_seed(ff)
    f = {"kind": "dense", "ff": ff}
    w = {"l0.mlp.up": torch.randn(ff, width, generator=g) * 1.5 / width ** 0.5, "l0.mlp.down": torch.randn(width, ff, generator=g) / ff ** 0.5,
         "l0.mlp.act": torch.tensor([0.7, -0.6, 0.5, 0.2])}
    w = {k: v.bfloat16().float() for k, v in w.items()}
    x = torch.randn(24, width, generator=g).bfloat16().float()
    got = _run_part(backend, "feed_forward", _feed_forward_spec(f, width, 1e-5, "l0.mlp."), w, x, [17, 1, 6])
    want = P.feed_forward(x.double(), F64(w), "l0.mlp.", f, 1e-5).float()
    torch.testing.assert_close(got, want, atol=2 * _tol(backend, want), rtol=0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("coef", [(1.0, 0.0, 0.0, 0.0), (0.0, 1.0, 0.0, 0.0), (0.0, 0.0, 1.0, 0.0), (0.0, 0.0, 0.0, 1.0)], ids=["z", "z2", "z3", "one"])
def test_each_power_of_the_activation(backend, coef):
    """Each term alone, on rows whose values span four orders of magnitude (a cube's root mean square is that of the largest value)."""
    rt, dev = runtime_for(backend)
    g = torch.Generator().manual_seed(1)
    z = (torch.randn(5, 264, generator=g) * 10.0 ** (4 * torch.rand(5, 264, generator=g) - 2)).bfloat16().float()
    z[4] *= 1e-3                                   # small enough for the constant under the root to matter
    want = P.poly_norm(z.double(), torch.tensor(coef).double(), 1e-5).float()
    buf = z.to(dev).to(rt.act_dtype)
    rt.kernels.poly_norm(buf, torch.tensor(coef, device=dev), 1e-5, buf)
    torch.testing.assert_close(buf.float().cpu(), want, atol=_tol(backend, want), rtol=2.0 ** -7 if backend[1] == "bfloat16" else 1e-4)


# ---- the sizes of a real layer, and the programs a user starts ----------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_as_wide_as_a_real_models(tmp_path, dtype):
    cfg = CONFIGS["wide"]
    w = make_weights(cfg, 31)
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=40 + i) for i, n in enumerate([420, 130, 17])}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    folder = write_model(str(tmp_path / "wide"), cfg, w, getattr(torch, dtype))
    backend = ("cuda", dtype)
    for steps, graphs in ((helpers.trace_whole(reqs), False), (helpers.trace_tail_decode(reqs, tail=40), True),
                          (helpers.trace_portions(reqs, sizes=(64, 2, 130, 1, 33)), False), (helpers.trace_mixed(reqs, live=3, seed=4), False)):
        eng = make_engine(folder, backend, 64, num_pages=20, graphs=graphs, budget=1024, context=512)
        with torch.inference_mode():
            got = helpers.replay(eng, steps)
        eng.kernels.check_errors()
        compare_rows(got, plain, backend)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_folder_of_this_design(tmp_path, dtype):
    import numpy as np

    cfg = CONFIGS["q"]
    w = make_weights(cfg, 17)
    folder = write_model(str(tmp_path / "m"), cfg, w, torch.bfloat16)
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=70 + i) for i, n in enumerate([70, 9, 33, 150, 2])}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
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
    compare_rows(got, plain, ("cuda", dtype))


# ---- configurations nobody chose ---------------------------------------------------------------------------------
def _random_config(rng) -> dict:
    """A model of this design drawn at random: widths and vocabularies that are no power of two, 2 to 6 layers that differ in every
    size, 1 to 5 key/value heads for up to 40 heads, head sizes that are and are not multiples of 16, blocks from one position to
    longer than the prompts and none, partial, full and no rotation, caps and none, layers without a feed-forward."""
    width, groups = rng.choice([(72, 3), (96, 2), (105, 7), (128, 1), (136, 4), (200, 5), (264, 8)])

    def att():
        kv = rng.choice([1, 2, 3, 4, 5])
        dim = rng.choice([8, 16, 24, 32, 40, 64, 80, 128])
        dims = rng.choice([d for d in (2, 4, 8, 16, 32, 64) if d <= dim] + [dim, None])
        return ATT(kv * rng.choice([1, 2, 3, 8]), kv, dim, rng.choice([1.0, 1.5, 2.5]) / dim ** 0.5, rng.choice([None, 3.0, 15.0, 50.0]),
                   rng.choice([None, 1, 7, 38, 64, 65, 130, 1000]), rng.choice([100.0, 10000.0, 500000.0]), dims)

    return {"architecture": "Vivepel", "width": width, "vocab": rng.choice([131, 257, 500, 640, 1000]),
            "norm": {"eps": rng.choice([1e-5, 1e-6]), "groups": groups},
            "layers": [LAYER(att(), rng.choice([None, 64, 90, 128, 333])) for _ in range(rng.randint(2, 6))]}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_random_configuration(tmp_path, seed, dtype):
    """Five requests of 2 to 330 tokens in pages of 64, whole, with decoded tails from CUDA graphs, in portions and as mixed batches
    of four live requests on a pool without a spare page, against the plain implementation."""
    import random

    rng = random.Random(seed)
    cfg = _random_config(rng)
    w = make_weights(cfg, seed)
    folder = write_model(str(tmp_path / "m"), cfg, w, getattr(torch, dtype))
    lens = [rng.choice([2, 3, 17, 64, 65, 130, 200, 257, 330]) for _ in range(5)]
    reqs = {f"r{i}": helpers.random_tokens(cfg["vocab"], n, seed=seed * 10 + i) for i, n in enumerate(lens)}
    plain = {rid: plain_logits(w, cfg, toks) for rid, toks in reqs.items()}
    backend = ("cuda", dtype)
    cuts = {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_tail_decode(r, tail=70),
            "portions": lambda r: helpers.trace_portions(r, sizes=(64, 2, 130, 1, 33, 5)), "mixed": lambda r: helpers.trace_mixed(r, live=4, seed=seed)}
    for cut, make in cuts.items():
        steps = make(reqs)
        pages = helpers.tokens_needed(steps, 64) // 64
        eng = make_engine(folder, backend, 64, num_pages=pages, max_slots=4, graphs=(cut == "tail"), budget=max(512, pages * 64), context=pages * 64)
        for v in eng.stepper.views:
            v.k.fill_(float("nan"))
            v.v.fill_(float("nan"))
        with torch.inference_mode():
            got = helpers.replay(eng, steps)
        eng.kernels.check_errors()
        try:
            compare_rows(got, plain, backend)
        except AssertionError as e:
            raise AssertionError(f"{cut}: {json.dumps(cfg)}: {e}") from None
        assert eng.cache.live == 0
