"""A selective state space with one decay per token and head (`StateSpaceSpec`; "Transformers are
SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality", Dao and
Gu): per head a float32 matrix S [state, v_head_dim] that starts at zero.

For a token with mixer input h, inner = heads * v_head_dim, head j in group j // (heads / groups):

    z | x | B | C | t = W_in h                    inner | inner | groups * state (twice) | heads
    x, B, C <- silu(conv(x, B, C) + b)            causal, per channel
    dt = softplus(t + dt_bias),   a = exp(-exp(A_log) dt)                          per head
    S <- a S + dt B x^T,          y = S^T C + D x                                  per head
    out = W_o [ rms(y * silu(z), in norm_groups equal parts of the row) * norm ]

This is a linear attention whose keys B and queries C are shared by a group's heads, whose values
are x and whose one decay per head is made by every token, so the recurrence runs on the kernels of
`ops.linear_attention`'s family (`ops.state_space`), prompts in chunks.  The request keeps S and the
convolution's last taps-1 inputs in two state records, float32 whatever the compute type.  The
product W_in h stays float32, so the step sizes and decays are 32-bit throughout.
"""
from __future__ import annotations

import torch

from .base import Mixer, SeveralNeeds, StateNeed, register_mixer
from .spec import ParamDecl, StateSpaceSpec

_LOCAL = ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")


class StateSpace(Mixer):
    @staticmethod
    def _names(spec):
        return {k: spec.names.get(k, k) for k in _LOCAL}

    @staticmethod
    def _check(spec: StateSpaceSpec):
        if spec.num_heads < 1 or spec.v_head_dim < 1 or spec.state < 1 or spec.taps < 1:
            raise ValueError("state_space: heads, sizes and taps must be at least 1")
        if spec.groups < 1 or spec.num_heads % spec.groups:
            raise ValueError(f"state_space: {spec.num_heads} heads do not share {spec.groups} "
                             f"groups evenly")
        if spec.norm_groups < 1 or spec.num_heads * spec.v_head_dim % spec.norm_groups:
            raise ValueError("state_space: the norm's parts are not equal")

    @staticmethod
    def channels(spec: StateSpaceSpec) -> int:
        """What the convolution works on: x | B | C."""
        return spec.num_heads * spec.v_head_dim + 2 * spec.groups * spec.state

    @staticmethod
    def params(spec: StateSpaceSpec, owns_cache: bool = True):
        StateSpace._check(spec)
        n = StateSpace._names(spec)
        inner, c, H = spec.num_heads * spec.v_head_dim, StateSpace.channels(spec), spec.num_heads
        return {
            n["in"]: ParamDecl((inner + c + H, spec.hidden), "linear"),
            n["conv"]: ParamDecl((c, spec.taps), "conv"),
            n["conv.b"]: ParamDecl((c,), "bias"),
            n["dt_bias"]: ParamDecl((H,), "normal", mean=-2.0, std=1.0),
            n["A_log"]: ParamDecl((H,), "normal", mean=0.0, std=1.0),
            n["D"]: ParamDecl((H,), "normal", mean=1.0, std=0.2),
            n["norm"]: ParamDecl((inner,), "norm"),
            n["o"]: ParamDecl((spec.hidden, inner), "linear"),
        }

    @staticmethod
    def cache_need(spec: StateSpaceSpec):
        conv = StateNeed((spec.taps - 1, StateSpace.channels(spec))) if spec.taps > 1 else None
        return SeveralNeeds((conv, StateNeed((spec.num_heads * spec.state * spec.v_head_dim,))))

    def __init__(self, spec: StateSpaceSpec, tensors, ops, dtype):
        self._check(spec)
        self.spec = spec
        self.ops = ops
        self.dtype = dtype
        n = self._names(spec)
        w_in = tensors[n["in"]]
        fill = -w_in.shape[0] % 8                  # zero rows, so that the product's rows stay aligned
        if fill:
            w_in = torch.cat([w_in, torch.zeros((fill, spec.hidden), dtype=w_in.dtype,
                                                device=w_in.device)])
        self.w_in = w_in.contiguous()
        self.w_out = tensors[n["o"]].contiguous()
        f32 = lambda k: tensors[n[k]].to(torch.float32).contiguous()
        self.filt, self.conv_bias = f32("conv"), f32("conv.b")
        self.dt_bias, self.a_log, self.skip, self.norm = f32("dt_bias"), f32("A_log"), f32("D"), f32("norm")

    def forward(self, normed, ctx, cache):
        if cache is None or cache.parts is None:
            raise ValueError("state_space: a recurrent state cannot be shared between calls")
        s = self.spec
        conv, memory = cache.parts
        proj = self.ops.linear(normed, self.w_in, out_dtype=torch.float32)
        y = self.ops.new_rows(normed.shape[0], s.num_heads * s.v_head_dim, self.dtype,
                              normed.device)
        self.ops.state_space(proj, self.filt, self.conv_bias, self.dt_bias, self.a_log, self.skip,
                             self.norm, conv.state if conv is not None else None, memory.state,
                             ctx, y, s.num_heads, s.v_head_dim, s.state, s.groups, s.taps,
                             s.norm_groups, s.norm_eps)
        return self.ops.linear(y, self.w_out, out_dtype=self.dtype)


register_mixer("state_space", StateSpace)
