"""Dopuvik: from its configuration to a `ModelSpec`.

Scaled embedding rows; every layer is a pre-norm block with bias-free layer norms:

    x <- x + mixer(LN(x) g1);   x <- x + moe(LN(x) g2)

The mixer is a selective state space (Mamba-2 form), a latent attention over a sliding window
(queries through a latent of their own; a pairwise, YaRN-scaled rotation of a key part that all
heads share), or two mixers side by side whose outputs are added with two factors: a grouped-query
attention with biases over a window that keeps its first tokens, and a gated delta rule with one
decay per head.  The feed-forward is a mixture of SwiGLU experts and identity experts: softmax
scores, compared with a learned correction within the best groups and weighed without it, not
renormalised.  The head is a matrix of its own; logits are scaled.

Tensor names: `embed`; `l<i>.norm1`, `.norm2`; `l<i>.mix.*` (`.left.*`, `.right.*` in a parallel
layer), `l<i>.mlp.*`; `final.norm`; `head`.
"""
from __future__ import annotations

from ..config.dopuvik import LATENT, MAMBA2, DopuvikConfig
from ..config.registry import register_architecture
from ..parts.spec import (AttentionSpec, BlockSpec, GatedDeltaSpec, LatentAttentionSpec,
                          LayerCall, ModelSpec, MoESpec, NormSpec, ParallelSpec, PositionSpec,
                          StateSpaceSpec)

# the design has no longest context: positions are bounded only by what float32 counts exactly
MAX_POSITION = 1 << 24
UNIT_EPS = 1e-6                # under the root of the delta rule's unit norms

_LATENT_NAMES = {"dkv_norm": "dkv.norm", "dq_norm": "dq.norm"}
_LEFT_NAMES = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "out_proj": "o", "q_bias": "q.b",
               "k_bias": "k.b", "v_bias": "v.b", "out_bias": "o.b"}
_MOE_NAMES = {"expert": "e{e}.{k}"}


def _position(rot, head_dim: int) -> PositionSpec:
    if rot is None:
        return PositionSpec("none")
    return PositionSpec("rope_partial", head_dim=head_dim, theta=rot.base, rot_dims=rot.dims,
                        yarn=rot.yarn)


def _mixer(l, cfg: DopuvikConfig):
    hidden, eps = cfg.width, cfg.norm_eps
    if l.type == MAMBA2:
        m = l.state_space
        return StateSpaceSpec("state_space", hidden, num_heads=m.heads, v_head_dim=m.vdim,
                              state=m.state, groups=m.groups, taps=m.taps,
                              norm_groups=m.norm_groups, norm_eps=eps)
    if l.type == LATENT:
        m = l.latent
        return LatentAttentionSpec(
            "attention_latent", hidden, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
            kv_rank=m.kv_rank, scale=m.scale, norm_eps=eps, q_rank=m.q_rank, rot_dim=m.rot_dim,
            rot_theta=m.rot.base if m.rot is not None else 10000.0, rot_pairs=True,
            rot_yarn=m.rot.yarn if m.rot is not None else None, window=m.window,
            names=_LATENT_NAMES)
    a, b = l.left, l.right
    left = AttentionSpec("attention", hidden, num_heads=a.heads, num_kv_heads=a.kv_heads,
                         head_dim=a.dim, v_head_dim=a.vdim, scale=a.scale, window=a.window,
                         keep_first=a.keep_first, position=_position(a.rot, a.dim), bias=True,
                         out_bias=True, names=_LEFT_NAMES)
    right = GatedDeltaSpec("gated_delta", hidden, num_heads=b.heads, num_kv_heads=b.kv_heads,
                           head_dim=b.dim, v_head_dim=b.vdim, taps=b.taps, norm_eps=eps,
                           unit_eps=UNIT_EPS, decay="head", gate="silu")
    return ParallelSpec("parallel", hidden, branches=(left, right),
                        scales=(l.left_scale, l.right_scale), prefixes=("left.", "right."))


def build_spec(cfg: DopuvikConfig) -> ModelSpec:
    hidden = cfg.width
    norm = NormSpec("layernorm_weight", hidden, cfg.norm_eps)
    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        norms = {"mixer": (norm, p + "norm1")}
        ffn = None
        if l.mlp is not None:
            norms["ffn"] = (norm, p + "norm2")
            f = l.mlp
            ffn = MoESpec("moe", hidden, ffn_dim=f.ff, experts=f.experts, top=f.top,
                          groups=f.groups, keep=f.keep, group_top=1, score="softmax",
                          renormalize=False, route_scale=f.route_scale, choice_bias=True,
                          identity=f.identity, names=_MOE_NAMES)
        layers.append(BlockSpec("pre_norm", _mixer(l, cfg), ffn, norms, mixer_prefix=p + "mix.",
                                ffn_prefix=p + "mlp."))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden=hidden,
        max_position=MAX_POSITION, layers=tuple(layers),
        order=tuple(LayerCall(i) for i in range(len(layers))), final_norm=norm,
        embedding_name="embed", final_norm_name="final.norm", head_name="head",
        embedding_scale=cfg.embedding_scale, logit_scale=cfg.logit_scale)


register_architecture("Dopuvik", DopuvikConfig, build_spec, replace=True)
