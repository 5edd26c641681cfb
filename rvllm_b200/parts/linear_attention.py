"""Linear attention with decay: a recurrence whose state per head is a matrix S [d, dv],

    S <- diag(a) S + k v^T,   o = S^T q

for a token's query, key (size d) and value (size dv).  The decay a is a constant per head
("lightning" form: "Lightning Attention-2", Qin et al.) or made by every token for every key
channel, a = sigmoid(z)^(1/tau) ("Gated Linear Attention Transformers with Hardware-Efficient
Training", Yang et al.).  q, k and v may pass silu; the read-out passes an RMS norm, over all heads
together or per head, and is multiplied by a gate before the output product:

    y = W_o [ o / sqrt(mean(o^2) + eps) * w * gate(W_g x) ]

S starts at zero and is the request's record in a state slot: float32 whatever the compute type.

W_q | W_k | W_v | W_g are one matrix, whose product has the compute type.  z = W_z x of decays made
by tokens is another product whose result stays float32 (decays are 32-bit throughout).  W_z =
W_a2 W_a1 is formed once when the weights are loaded: the rank of the two factors saves
parameters in the file, but each is a product of a few columns or a few terms, and two of them
take longer than the one.  Activations, decays, recurrence, norm and gate are
`ops.linear_attention`, for any mixture of prompt portions and single tokens.
"""
from __future__ import annotations

import math

import torch

from .base import Mixer, StateNeed, register_mixer
from .spec import LinearAttentionSpec, ParamDecl

_LOCAL = ("q", "k", "v", "g", "o", "norm", "a1", "a2", "a2.b")


class LinearAttention(Mixer):
    ACTIVATIONS = (None, "silu")
    NORMS = ("all", "head")
    GATES = ("sigmoid", "silu")

    @staticmethod
    def _names(spec):
        return {k: spec.names.get(k, k) for k in _LOCAL}

    @staticmethod
    def _check(spec: LinearAttentionSpec):
        if spec.num_heads < 1 or spec.head_dim < 1 or spec.v_head_dim < 1:
            raise ValueError("linear_attention: head count and sizes must be at least 1")
        if spec.decay is not None:
            if len(spec.decay) != spec.num_heads:
                raise ValueError("linear_attention: one decay per head")
        elif spec.decay_rank < 1 or not spec.decay_tau > 0:
            raise ValueError("linear_attention: decays made by tokens need a rank and a positive tau")
        if spec.activation not in LinearAttention.ACTIVATIONS or \
                spec.norm not in LinearAttention.NORMS or spec.gate not in LinearAttention.GATES:
            raise ValueError(f"linear_attention: activation {spec.activation!r}, norm {spec.norm!r} "
                             f"or gate {spec.gate!r} is not known")

    @staticmethod
    def params(spec: LinearAttentionSpec, owns_cache: bool = True):
        LinearAttention._check(spec)
        n = LinearAttention._names(spec)
        w, H, d, dv = spec.hidden, spec.num_heads, spec.head_dim, spec.v_head_dim
        p = {n["q"]: ParamDecl((H * d, w), "linear"), n["k"]: ParamDecl((H * d, w), "linear"),
             n["v"]: ParamDecl((H * dv, w), "linear"), n["g"]: ParamDecl((H * dv, w), "linear"),
             n["norm"]: ParamDecl((H * dv if spec.norm == "all" else dv,), "norm"),
             n["o"]: ParamDecl((w, H * dv), "linear")}
        if spec.decay is None:
            p[n["a1"]] = ParamDecl((spec.decay_rank, w), "linear")
            p[n["a2"]] = ParamDecl((H * d, spec.decay_rank), "normal", mean=0.0, std=0.5)
            p[n["a2.b"]] = ParamDecl((H * d,), "normal", mean=1.0, std=1.0)
        return p

    @staticmethod
    def cache_need(spec: LinearAttentionSpec):
        return StateNeed((spec.num_heads * spec.head_dim * spec.v_head_dim,))

    def __init__(self, spec: LinearAttentionSpec, tensors, ops, dtype):
        self._check(spec)
        self.spec = spec
        self.ops = ops
        self.dtype = dtype
        n = self._names(spec)
        q = tensors[n["q"]]
        parts = [tensors[n[k]].to(q.dtype) for k in ("q", "k", "v", "g")]
        self.log_decay = self.decay_bias = self.w_z = None
        if spec.decay is None:
            wide = torch.float64
            self.w_z = (tensors[n["a2"]].to(wide) @ tensors[n["a1"]].to(wide)).to(q.dtype).contiguous()
            self.decay_bias = tensors[n["a2.b"]].to(torch.float32).contiguous()
        else:
            # a decay of 0 forgets everything: e^-1e4 is 0 in float32, without an infinity whose
            # product with 0 would be no number
            self.log_decay = torch.tensor([math.log(a) if a > 0.0 else -1e4 for a in spec.decay],
                                          dtype=torch.float32, device=q.device)
        self.w_in = torch.cat(parts, dim=0).contiguous()
        norm = tensors[n["norm"]].to(torch.float32)
        if spec.norm == "head":
            norm = norm.repeat(spec.num_heads)
        self.norm = norm.contiguous()                          # [H * dv] either way
        self.w_out = tensors[n["o"]].contiguous()

    def forward(self, normed, ctx, cache):
        if cache is None or not cache.owns:
            raise ValueError("linear_attention: a recurrent state cannot be shared between calls")
        s = self.spec
        rows = self.ops.linear(normed, self.w_in, out_dtype=self.dtype)
        z = self.ops.linear(normed, self.w_z, out_dtype=torch.float32) if self.w_z is not None else None
        y = self.ops.new_rows(normed.shape[0], s.num_heads * s.v_head_dim, self.dtype,
                              normed.device)
        self.ops.linear_attention(rows, z, self.log_decay, self.decay_bias, s.decay_tau, self.norm,
                                  cache.state, ctx, y, s.num_heads, s.head_dim, s.v_head_dim,
                                  s.activation, s.q_scale, s.norm, s.gate, s.norm_eps)
        return self.ops.linear(y, self.w_out, out_dtype=self.dtype)


register_mixer("linear_attention", LinearAttention)
