"""The Vivepel decoder, whole sequences at a time, in plain torch on the CPU: one function per mechanism.

A slow restatement of the design's equations that shares no code with the engine; the tests compare the engine
with it. Every function takes one sequence ([T, ...] tensors, position 0 first) and works in the dtype of its
inputs (the tests use float64). Notation: T tokens, W width, H heads, G key/value heads, d head size.

The design: x = embed[token]; per layer x += s1 * n1b(attention(n1(x))), then x += s2 * n2b(ff(n2(x))), with n a root-mean-square
norm taken over equal groups of the vector, and s a learned scale per element. Attention: biased queries and keys; the values
are the keys as projected; per-head norms with a shared weight, then a partial rotation in the half layout; scores capped by
c * tanh(s / c); a query reads the keys of its own block of positions; one is added to the softmax's denominator; the weights of
the heads are mixed by an H x H matrix before they meet the values. The feed-forward is plain and dense with a polynomial of
normalised powers as activation, or absent. Final norm, an output head of its own.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


# ---- small pieces -------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, weight, groups, eps):
    """Every one of ``groups`` equal consecutive parts of a vector divided by its own root mean square; then the weight."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * weight


def poly_norm(z, coef, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e, N dividing a token's vector by its root mean square."""
    a, b, c, e = coef.unbind()
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z * z * z, eps) + e


def rotate(x, rot: Optional[dict]):
    """x [T, heads, d]: element i < dims/2 of a head pairs with element i + dims/2; the pair at position p turns by
    p * base^(-2i/dims). Elements from ``dims`` on pass unchanged."""
    if not rot or not rot.get("dims"):
        return x
    t, half = x.shape[0], rot["dims"] // 2
    out = x.clone()
    pos = torch.arange(t, dtype=x.dtype)
    for i in range(half):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(pos * f)[:, None], torch.sin(pos * f)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def visible(i: int, j: int, size: Optional[int]) -> bool:
    """May position i read position j? Not the future, and only inside its own block of ``size`` positions."""
    return j <= i and (size is None or i // size == j // size)


def capped(s, cap: Optional[float]):
    return cap * torch.tanh(s / cap) if cap else s


def weights_with_one_more(s):
    """exp(s_j) / (1 + sum_j exp(s_j)) over the last axis (masked scores are -inf)."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def mix_heads(weights, talk):
    """weights [H, T, T]: head h's weights become sum_g talk[h, g] * (head g's)."""
    return torch.einsum("hg,gij->hij", talk, weights)


# ---- sub-layers -----------------------------------------------------------------------------------------------
def attention_mixer(h, w, p, m, eps):
    heads, g, d = m["heads"], m["kv_heads"], m["dim"]
    t = h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(t, heads, d)
    v = (h @ w[p + "k"].T + w[p + "k.b"]).view(t, g, d)
    k = rotate(unit_rms(v, eps) * w[p + "k.norm"], m.get("rot"))
    q = rotate(unit_rms(q, eps) * w[p + "q.norm"], m.get("rot"))
    size = (m.get("mask") or {}).get("size")
    allowed = torch.tensor([[visible(i, j, size) for j in range(t)] for i in range(t)])
    per = heads // g
    weights = torch.zeros(heads, t, t, dtype=h.dtype)
    for n in range(heads):
        s = capped((q[:, n] @ k[:, n // per].T) * m["scale"], m.get("softcap"))
        weights[n] = weights_with_one_more(s.masked_fill(~allowed, float("-inf")))
    weights = mix_heads(weights, w[p + "talk"])
    out = torch.stack([weights[n] @ v[:, n // per] for n in range(heads)], 1)
    return out.reshape(t, heads * d) @ w[p + "o"].T


def feed_forward(h, w, p, f, eps):
    return poly_norm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


# ---- the model ------------------------------------------------------------------------------------------------
def forward(tokens, w: Dict[str, torch.Tensor], cfg: dict, streams: Optional[List] = None):
    """Logits [T, vocab] of one sequence. ``streams``, if given, receives the residual stream after every layer."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups") or 1
    norm = lambda v, name: grouped_norm(v, w[name], groups, eps)
    x = w["embed"][torch.tensor([int(t) for t in tokens])]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = attention_mixer(norm(x, p + "norm1"), w, p + "mix.", layer["mixer"], eps)
        x = x + norm(y, p + "norm1b") * w[p + "ls1"]
        f = layer.get("mlp")
        if f is not None:
            y = feed_forward(norm(x, p + "norm2"), w, p + "mlp.", f, eps)
            x = x + norm(y, p + "norm2b") * w[p + "ls2"]
        if streams is not None:
            streams.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T


# ---- tensor names and shapes ------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Every tensor of a model of this configuration."""
    wd = cfg["width"]
    s: Dict[str, tuple] = {"embed": (cfg["vocab"], wd), "final.norm": (wd,), "head": (cfg["vocab"], wd)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        s[p + "norm1"] = s[p + "norm1b"] = s[p + "ls1"] = (wd,)
        for n, heads in (("q", m["heads"]), ("k", m["kv_heads"])):
            s[p + f"mix.{n}"], s[p + f"mix.{n}.b"], s[p + f"mix.{n}.norm"] = (heads * m["dim"], wd), (heads * m["dim"],), (m["dim"],)
        s[p + "mix.talk"], s[p + "mix.o"] = (m["heads"], m["heads"]), (wd, m["heads"] * m["vdim"])
        if f is not None:
            s[p + "norm2"] = s[p + "norm2b"] = s[p + "ls2"] = (wd,)
            s[p + "mlp.up"], s[p + "mlp.down"], s[p + "mlp.act"] = (f["ff"], wd), (wd, f["ff"]), (4,)
    return s
