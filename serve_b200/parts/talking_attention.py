"""Grouped-query softmax attention whose heads' weights are mixed before they meet the values.

q = W_q h (+ b_q), k = W_k h (+ b_k). With ``keys_are_values`` the values are the keys as projected, before norm and rotation, and
there is no value projection; else v = W_v h (+ b_v). With ``head_norm_eps`` every query and key head is divided by its own root mean
square over ``dim`` elements and multiplied by a weight of that size that all query (all key) heads share ("q.norm", "k.norm"), before
the position part turns the first ``rotary_dim`` elements. score = (q . k) * scale; with ``softcap`` c the score becomes
c * tanh(score / c). Causal; with ``chunk`` position i reads position j only if floor(i / chunk) = floor(j / chunk). With
``sink_score`` s the softmax's denominator also holds exp(s), the same for all heads, without key or value (0: one is added). The heads'
weights are then mixed, weight_h(i, j) <- sum_g T[h, g] weight_g(i, j) with T = "talk" [heads, heads], and head h applies its mixed
weights to the values of its own key/value head. The output projection has no bias.

The cache pages and the kernels have one head size, ``dim`` rounded up to a multiple of 16, and what lies beyond a head's true size
is zero. The projection's sums stay float until bias, norm and rotation are done, so queries and cached keys are rounded once.
"""
from __future__ import annotations

import math

import torch

from .base import CacheNeed, Mixer, TensorDecl, build_part, register_part
from .biased_attention import _pad_heads
from .rotary import PAIRING_HALF


@register_part("mixer", "talking_attention")
class TalkingAttention(Mixer):
    """params: hidden, heads, kv_heads, dim, scale (None: dim**-0.5), bias (bool), keys_are_values (bool), head_norm_eps (None: no norm),
    softcap (None: none), chunk (None: all keys), sink_score (None: no sink), position (PartSpec), names."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.heads, self.kv_heads, self.dim = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"]), int(p["dim"])
        if self.heads % self.kv_heads:
            raise ValueError(f"heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        self.scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.dim)
        self.bias = bool(p.get("bias", False))
        self.keys_are_values = bool(p.get("keys_are_values", False))
        self.head_norm_eps = float(p["head_norm_eps"]) if p.get("head_norm_eps") is not None else None
        self.softcap = float(p["softcap"]) if p.get("softcap") else 0.0
        self.chunk = int(p["chunk"]) if p.get("chunk") else None
        self.sink_score = float(p["sink_score"]) if p.get("sink_score") is not None else None
        self.position = build_part("position", p["position"], runtime)
        if self.position.rotary_dim > self.dim:
            raise ValueError("rotary_dim exceeds the query/key size")
        if self.position.rotary_dim and self.position.pairing != PAIRING_HALF:
            raise ValueError("talking_attention rotates pairs (i, i + rotary_dim / 2)")
        self.names = dict(p.get("names", {}))
        self.head_dim = 16 * -(-self.dim // 16)
        self.mixed_size = self.heads * self.head_dim
        runtime.kernels.check_attention_shape(self.heads, self.kv_heads, self.head_dim)

    def _name(self, key):
        return self.prefix + self.names.get(key, key)

    def kernel_needs(self):
        return {"talking_head_dims": [self.head_dim], "libraries": ["prep"]}

    def _projections(self):
        return [("q", self.heads), ("k", self.kv_heads)] + ([] if self.keys_are_values else [("v", self.kv_heads)])

    def tensor_decls(self):
        decls = [TensorDecl(self._name(n), (h * self.dim, self.hidden)) for n, h in self._projections()]
        if self.bias:
            decls += [TensorDecl(self._name(n + ".b"), (h * self.dim,), role="vector", init="small") for n, h in self._projections()]
        if self.head_norm_eps is not None:
            decls += [TensorDecl(self._name(n + ".norm"), (self.dim,), role="vector", init="norm") for n in ("q", "k")]
        decls += [TensorDecl(self._name("talk"), (self.heads, self.heads)), TensorDecl(self._name("o"), (self.hidden, self.heads * self.dim))]
        return decls

    def load(self, tensors):
        d = self.head_dim
        self.w_in = torch.cat([_pad_heads(tensors[self._name(n)], h, self.dim, d) for n, h in self._projections()], dim=0).contiguous()
        vec = lambda name, h: _pad_heads(tensors[self._name(name)].float().view(-1, 1), h, self.dim, d).view(-1)
        self.b_in = torch.cat([vec(n + ".b", h) for n, h in self._projections()]).contiguous() if self.bias else None
        self.q_norm = self.k_norm = None
        if self.head_norm_eps is not None:
            self.q_norm, self.k_norm = vec("q.norm", 1).contiguous(), vec("k.norm", 1).contiguous()
        w_o = tensors[self._name("o")]
        if self.dim != d:
            padded = w_o.new_zeros((self.hidden, self.heads, d))
            padded[:, :, : self.dim] = w_o.view(self.hidden, self.heads, self.dim)
            w_o = padded.view(self.hidden, self.heads * d)
        self.w_o = w_o.contiguous()
        talk = tensors[self._name("talk")]
        if talk.dtype == torch.bfloat16:
            # the mixing runs as a matrix product on the tensor cores: both sides padded to a multiple of 16
            n = 16 * -(-self.heads // 16)
            padded = talk.new_zeros((n, n))
            padded[: self.heads, : self.heads] = talk
            talk = padded
        self.talk = talk.contiguous()
        self.sinks = None
        if self.sink_score is not None:
            self.sinks = torch.full((self.heads,), self.sink_score, dtype=torch.float32, device=self.w_o.device)

    def cache_need(self):
        return CacheNeed(kv_heads=self.kv_heads, head_dim=self.head_dim, chunk=self.chunk)

    def output_weight(self):
        return self.w_o

    def mix_into(self, h, ctx, cache, out, scale: float = 1.0):
        if scale != 1.0 or not out.is_contiguous():
            raise ValueError("talking_attention writes its heads unscaled into a contiguous buffer")
        if not cache.writes:
            raise ValueError("talking_attention writes the pages it reads")
        k = self.rt.kernels
        t, d = h.shape[0], self.head_dim
        sums = torch.empty((t, self.w_in.shape[0]), dtype=torch.float32, device=h.device)
        k.linear(h, self.w_in, sums)
        table = ctx.block_tables[cache.group]
        q = self.rt.empty_act((t, self.heads * d))
        k.qk_prepare(sums, self.b_in, ctx.positions, ctx.token_row, self.heads, self.kv_heads, d, self.dim, self.q_norm, self.k_norm,
                     self.head_norm_eps or 0.0, self.position.inv_freq, self.position.rotary_dim, q, cache.k, cache.v, table, cache.page_size,
                     head_norm="before" if self.head_norm_eps is not None else False, keys_are_values=self.keys_are_values)
        k.talking_attention(q, cache.k, cache.v, table, ctx.cu_q, ctx.kv_len, ctx.positions, self.heads, self.kv_heads, d, cache.page_size,
                            self.scale, self.talk, out, ctx.shape, chunk=self.chunk or 0, softcap=self.softcap, sinks=self.sinks)

    def forward(self, h, ctx, cache):
        mixed = self.rt.empty_act((h.shape[0], self.mixed_size))
        self.mix_into(h, ctx, cache, mixed)
        out = self.rt.empty_act((h.shape[0], self.hidden))
        self.rt.kernels.linear(mixed, self.w_o, out)
        return out
