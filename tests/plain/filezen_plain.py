"""The Filezen decoder, whole sequences at a time, in plain torch on the CPU: one function per mechanism.

A slow restatement of the design's equations that shares no code with the engine; the tests compare the engine
with it. Every function takes one sequence ([T, ...] tensors, position 0 first) and works in the dtype of its
inputs (the tests use float64). Notation: T tokens, W width, H heads.

The design: x_t = embed[tok_t] * s. A layer's two sub-layers read the stream as it is, and only what they give back is
normalised: x += m n1(mixer(x)), x += m n2(ff(x)), n(a) = a / rms(a) * w. Two mixers: "latent_attention" (queries
straight from the stream; keys and values read out of one normalised low-rank vector per token plus one rotated key part
that all heads share; frequencies scaled by a ramp over the pair index, rotated vectors lengthened by a constant; a
sliding window; a layer may take the low-rank vector and the rotated key part of an earlier layer instead of making its
own) and "retention" (a matrix state per head with a fixed decay, S <- d S + k v^T, read out after the update, divided by
its root mean square per head and gated by silu; queries and keys rotated). The feed-forward is dense and gated with
silu, or a mixture of silu-gated experts (softmax router, only the experts of the best groups can be chosen, weights =
chosen scores over their sum, a shared expert added for every token), or absent. Final norm, the embedding table as head.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F


# ---- small pieces -------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(rot: dict) -> List[float]:
    """One frequency per rotated pair: base^(-2i/dims); with a scaling, pair i keeps 1 - r_i of its frequency and takes r_i
    of it divided by the factor, r a ramp over i between the pairs that turn ``fast`` and ``slow`` times in ``original``
    positions."""
    dims, base = rot["dims"], rot["base"]
    sc = rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            pair = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
            lo, hi = max(math.floor(pair(sc["fast"])), 0), min(math.ceil(pair(sc["slow"])), dims - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * r + f * (1.0 - r)
        out.append(f)
    return out


def lengthening(rot: dict) -> float:
    """What a scaled rotation multiplies its cosines and sines by."""
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1.0 if rot.get("scaling") else 1.0


def rotate(x, rot: Optional[dict]):
    """x [T, heads, D]: element i < dims/2 of a head pairs with element i + dims/2; the pair at position p turns by
    p * f_i. Elements from ``dims`` on pass unchanged."""
    if not rot or not rot.get("dims"):
        return x
    t, half, long = x.shape[0], rot["dims"] // 2, lengthening(rot)
    out = x.clone()
    pos = torch.arange(t, dtype=x.dtype)
    for i, f in enumerate(frequencies(rot)):
        c, s = (torch.cos(pos * f) * long)[:, None], (torch.sin(pos * f) * long)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def visible(i: int, j: int, size: Optional[int]) -> bool:
    """May position i read position j? Not the future, and nothing ``size`` or more positions back."""
    return j <= i and (size is None or i - j < size)


# ---- mixers ---------------------------------------------------------------------------------------------------
def latent_row(h, w, p, m, eps):
    """What a token leaves for later ones: the normalised low-rank vector c [T, rank] and the shared rotated key part [T, rd]."""
    rank, rd = m["kv_rank"], m["rot_dim"]
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    rot = dict(m["rot"], dims=rd)
    return c, rotate(down[:, rank:].view(h.shape[0], 1, rd), rot)[:, 0]


def latent_mixer(h, w, p, m, c, k_rot):
    heads, dim, rd, vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    t = h.shape[0]
    q = (h @ w[p + "q"].T).view(t, heads, dim + rd)
    q_plain, q_rot = q[..., :dim], rotate(q[..., dim:], dict(m["rot"], dims=rd))
    k_plain = (c @ w[p + "uk"].T).view(t, heads, dim)
    v = (c @ w[p + "uv"].T).view(t, heads, vdim)
    size = (m.get("mask") or {}).get("size")
    allowed = torch.zeros(t, t, dtype=torch.bool)
    for i in range(t):
        allowed[i, [j for j in range(0 if size is None else max(0, i - size), i + 1) if visible(i, j, size)]] = True
    out = torch.zeros(t, heads, vdim, dtype=h.dtype)
    for n in range(heads):
        s = (q_plain[:, n] @ k_plain[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]
        out[:, n] = torch.softmax(s.masked_fill(~allowed, -math.inf), -1) @ v[:, n]
    return out.reshape(t, heads * vdim) @ w[p + "o"].T


def retention_mixer(h, w, p, m, eps):
    """S_t = d_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head."""
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    t = h.shape[0]
    q = rotate((h @ w[p + "q"].T).view(t, heads, dim), m.get("rot"))
    k = rotate((h @ w[p + "k"].T).view(t, heads, dim), m.get("rot")) * dim ** -0.5
    v = (h @ w[p + "v"].T).view(t, heads, vdim)
    out = torch.zeros(t, heads, vdim, dtype=h.dtype)
    decay = torch.tensor(m["decay"], dtype=h.dtype)[:, None, None]
    S = torch.zeros(heads, dim, vdim, dtype=h.dtype)
    for i in range(t):
        S = decay * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = (S * q[i][:, :, None]).sum(1)
    y = unit_rms(out, eps).reshape(t, heads * vdim) * F.silu(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------
def gated_ff(h, w, p):
    return (F.silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def chosen_experts(h, w, p, f):
    """[T, top] indices of the experts with the largest scores among those of the best groups (lowest index first on ties),
    and their weights. A group of neighbours is as good as its best expert."""
    s = torch.softmax(h @ w[p + "router"].T, -1)
    r = f["router"]
    open_ = torch.ones_like(s, dtype=torch.bool)
    if r.get("groups"):
        n = r["groups"]["count"]
        best = s.view(s.shape[0], n, -1).amax(-1)
        kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, : r["groups"]["keep"]]
        mark = torch.zeros(s.shape[0], n, dtype=torch.bool).scatter(1, kept, True)
        open_ = mark.repeat_interleave(s.shape[1] // n, dim=1)
    idx = torch.sort(s.masked_fill(~open_, -1.0), dim=-1, descending=True, stable=True).indices[:, : r["top"]]
    wt = torch.gather(s, 1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20)


def expert_ff(h, w, p, f):
    idx, wt = chosen_experts(h, w, p, f)
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        rows, place = (idx == e).nonzero(as_tuple=True)          # the tokens that chose this expert
        if len(rows):
            out[rows] += wt[rows, place][:, None] * gated_ff(h[rows], w, f"{p}e{e}.")
    if f.get("shared") is not None:
        out = out + gated_ff(h, w, p + "shared.")
    return out


def feed_forward(h, w, p, f):
    return gated_ff(h, w, p) if f["kind"] == "dense" else expert_ff(h, w, p, f)


# ---- the model ------------------------------------------------------------------------------------------------
def forward(tokens, w: Dict[str, torch.Tensor], cfg: dict, streams: Optional[list] = None):
    """Logits [T, vocab] of one sequence. ``streams``, if given, receives the residual stream after every layer."""
    tokens = [int(t) for t in tokens]
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = w["embed"][tokens] * (cfg.get("embedding") or {}).get("scale", 1.0)
    left = {}                                                # layer -> what its tokens left for later ones
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                left[i] = latent_row(x, w, p + "mix.", m, eps)
            a = latent_mixer(x, w, p + "mix.", m, *left[i if source is None else source])
        else:
            a = retention_mixer(x, w, p + "mix.", m, eps)
        x = x + mult * (unit_rms(a, eps) * w[p + "norm1"])
        if layer.get("mlp") is not None:
            x = x + mult * (unit_rms(feed_forward(x, w, p + "mlp.", layer["mlp"]), eps) * w[p + "norm2"])
        if streams is not None:
            streams.append(x.clone())
    return (unit_rms(x, eps) * w["final.norm"]) @ w["embed"].T


# ---- tensor names and shapes ------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Every tensor of a model of this configuration."""
    wd = cfg["width"]
    s: Dict[str, tuple] = {"embed": (cfg["vocab"], wd), "final.norm": (wd,)}

    def gated(p, ff):
        s[p + "gate"], s[p + "up"], s[p + "down"] = (ff, wd), (ff, wd), (wd, ff)

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        s[f"l{i}.norm1"] = (wd,)
        heads, hv = m["heads"], m["heads"] * m["vdim"]
        s[p + "o"] = (wd, hv)
        if layer["type"] == "latent_attention":
            s[p + "q"] = (heads * (m["dim"] + m["rot_dim"]), wd)
            if m.get("kv_from") is None:
                s[p + "dkv"], s[p + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], wd), (m["kv_rank"],)
            s[p + "uk"], s[p + "uv"] = (heads * m["dim"], m["kv_rank"]), (hv, m["kv_rank"])
        else:
            s[p + "q"] = s[p + "k"] = (heads * m["dim"], wd)
            s[p + "v"] = s[p + "g"] = (hv, wd)
        f = layer.get("mlp")
        if f is None:
            continue
        s[f"l{i}.norm2"] = (wd,)
        p = f"l{i}.mlp."
        if f["kind"] == "dense":
            gated(p, f["ff"])
        else:
            s[p + "router"] = (f["router"]["experts"], wd)
            for e in range(f["router"]["experts"]):
                gated(f"{p}e{e}.", f["expert"]["ff"])
            if f.get("shared") is not None:
                gated(p + "shared.", f["shared"]["ff"])
    return s
