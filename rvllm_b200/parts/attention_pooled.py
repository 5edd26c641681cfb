"""Grouped-query attention over a window of tokens and the pooled blocks before it
(`PooledAttentionSpec`).

A query weighs two kinds of rows in the same softmax.  Its own position and the window - 1 before
it are single tokens.  What is older is there as means: every `pool` consecutive positions (0 to
pool - 1, and so on) give one key and one value, the means of what the pages hold for them, and a
query at i takes the first max(0, i - window + 1) // pool of these.  So between the newest mean it
takes and its window up to pool - 1 positions are hidden from it.  Options: a further term
exp(sink_h) in the denominator; capped scores, c tanh(s / c); keys that serve, unrotated, as values.

Two page groups serve a call: the tokens' keys and values, whose pages are given back once they
lie before the window *and* before the newest incomplete block, and one row per block, which is
kept as long as the request lives.  A block's row is formed in the step that brings the block's
last token, always from its tokens' rows as the cache holds them, so it does not depend on how
the block's tokens were cut into steps.

q and k (and v, when it has a projection) are one product; rotation, the cache write and the
blocks' rows are one kernel (`ops.rope_pool_write`).
"""
from __future__ import annotations

import math

import torch

from .base import Mixer, PagedNeed, SeveralNeeds, position_class, register_mixer
from .spec import ParamDecl, PooledAttentionSpec

_LOCAL = ("q", "k", "v", "o", "sink")


class PooledAttention(Mixer):
    @staticmethod
    def _names(spec):
        return {k: spec.names.get(k, k) for k in _LOCAL}

    @staticmethod
    def _check(spec: PooledAttentionSpec):
        if spec.num_heads < 1 or spec.num_kv_heads < 1 or spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"invalid attention head counts: {spec.num_heads} query, "
                             f"{spec.num_kv_heads} KV")
        if spec.v_head_dim and spec.v_head_dim != spec.head_dim:
            raise ValueError("attention_pooled: keys and values have the same size")
        if spec.pool is not None and spec.window is None:
            raise ValueError("attention_pooled: pooled blocks lie before a window")
        if spec.position.kind not in ("rope_partial", "none"):
            raise ValueError("attention_pooled takes a rope_partial rotation or none")
        if spec.softcap is not None and not spec.softcap > 0:
            raise ValueError("attention_pooled: the cap must be positive")

    @staticmethod
    def params(spec: PooledAttentionSpec, owns_cache: bool = True):
        PooledAttention._check(spec)
        n = PooledAttention._names(spec)
        H, G, d = spec.num_heads, spec.num_kv_heads, spec.head_dim
        p = {n["q"]: ParamDecl((H * d, spec.hidden), "linear"),
             n["k"]: ParamDecl((G * d, spec.hidden), "linear"),
             n["o"]: ParamDecl((spec.hidden, H * d), "linear")}
        if not spec.values_are_keys:
            p[n["v"]] = ParamDecl((G * d, spec.hidden), "linear")
        if spec.sinks:
            p[n["sink"]] = ParamDecl((H,), "normal", mean=0.0, std=1.0)
        return p

    @staticmethod
    def cache_need(spec: PooledAttentionSpec):
        tokens = PagedNeed(spec.num_kv_heads, spec.head_dim, spec.window, block=spec.pool)
        if spec.pool is None:
            return SeveralNeeds((tokens, None))
        return SeveralNeeds((tokens, PagedNeed(spec.num_kv_heads, spec.head_dim, every=spec.pool)))

    @staticmethod
    def workspace_bytes(spec: PooledAttentionSpec, ops, max_requests: int, max_context: int) -> int:
        sizer = getattr(ops, "attention_pooled_scratch_bytes", None)
        if sizer is None:
            return 0
        return sizer(max_requests, spec.num_heads, spec.head_dim, max_context, spec.window, spec.pool)

    def __init__(self, spec: PooledAttentionSpec, tensors, ops, dtype):
        self._check(spec)
        self.spec = spec
        self.ops = ops
        self.dtype = dtype
        n = self._names(spec)
        q = tensors[n["q"]]
        keys = ("q", "k") if spec.values_are_keys else ("q", "k", "v")
        self.w_in = torch.cat([tensors[n[k]].to(q.dtype) for k in keys], dim=0).contiguous()
        self.w_out = tensors[n["o"]].contiguous()
        self.sinks = tensors[n["sink"]].to(torch.float32).contiguous() if spec.sinks else None
        self.position = position_class(spec.position.kind)(spec.position, q.device)
        self.scale = spec.scale if spec.scale is not None else 1.0 / math.sqrt(spec.head_dim)

    def forward(self, normed, ctx, cache):
        if cache is None or cache.parts is None:
            raise ValueError("attention_pooled: the call keeps its own tokens and blocks")
        s = self.spec
        H, G, d = s.num_heads, s.num_kv_heads, s.head_dim
        tokens, blocks = cache.parts
        group = ctx.groups[tokens.group]
        rows = self.ops.linear(normed, self.w_in, out_dtype=self.dtype)
        freq, amplitude = None, 1.0
        if s.position.kind == "rope_partial":
            freq, amplitude = self.position.frequencies(), self.position.amplitude
        options = dict(amplitude=amplitude, values_are_keys=s.values_are_keys)
        pooled = None
        if blocks is None:
            self.ops.rope_partial_write(rows, H, G, d, d, freq, ctx.positions, group.slot_mapping,
                                        tokens.k, tokens.v, **options)
        else:
            bgroup = ctx.groups[blocks.group]
            self.ops.rope_pool_write(rows, H, G, d, freq, ctx, group, tokens.k, tokens.v, s.pool,
                                     bgroup.slot_mapping, blocks.k, blocks.v, **options)
            pooled = (blocks.k, blocks.v, bgroup, s.pool)
        out = self.ops.new_rows(normed.shape[0], H * d, self.dtype, normed.device)
        self.ops.paged_attention_pooled(rows, H, G, d, tokens.k, tokens.v, ctx, group, pooled,
                                        self.scale, s.softcap, s.window, self.sinks, out)
        return self.ops.linear(out, self.w_out, out_dtype=self.dtype)


register_mixer("attention_pooled", PooledAttention)
