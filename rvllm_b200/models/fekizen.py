"""Fekizen: from its configuration to a `ModelSpec`.

The scaled embedding rows plus a learned position vector pass an RMS norm.  A layer is a pre-norm
block whose mixer reads the normed rows moved towards the token before (token shift):

    h = N(x) g1;  h_p <- h_p + (h_(p-1) - h_p) * shift;  x <- x + mixer(h);  x <- x + ff(N(x) g2)

The mixer is a linear attention with a constant decay per head and silu on its projections, read
out through one norm over all heads and a sigmoid gate; or half the sum of two mixers' outputs,
each normed over the model's width: a grouped-query attention whose values are its unrotated
keys (YaRN-scaled rotation, capped scores, a learned sink, a window of tokens and before it one
mean key and value per block), and a linear attention with a decay per key channel, read out
through a norm per head and a silu gate.  The feed-forward is a mixture of gated experts whose
weights come from the chosen experts' logits only, with one more expert for all tokens.  Layers [start, stop) may run several times
with the same weights: every pass has caches of its own, begins by adding its row of `loop.step`
to the stream and, from the second on, the embedding rows once more.  The head is a matrix of
its own.

Tensor names: `embed`, `pos`, `embed.norm`; `loop.step`; `l<i>.norm1`, `.norm2`, `.shift`;
`l<i>.mix.*` (`.left.*`, `.right.*` in a parallel layer), `l<i>.mlp.*`; `final.norm`; `head`.
"""
from __future__ import annotations

from ..config.fekizen import LIGHTNING, FekizenConfig
from ..config.registry import register_architecture
from ..parts.spec import (BlockSpec, LayerCall, LinearAttentionSpec, ModelSpec, MoESpec, NormSpec,
                          ParallelSpec, PooledAttentionSpec, PositionSpec, SwiGLUSpec)

_GLU_NAMES = {"gate": "gate", "up": "up", "down": "down"}
_MOE_NAMES = {"expert": "e{e}.{k}"}
LOOP_STEP = "loop.step"
DEFAULT_RANK = 16          # of the decay product, for random weights of a config without it


def run_order(n_layers: int, loop):
    """The calls in order: layers before the stretch, the stretch `times` times (each pass with
    caches of its own; its first call adds the pass's row of `loop.step` and, from the second
    pass on, the embedding rows), the rest."""
    if loop is None:
        return [LayerCall(i) for i in range(n_layers)]
    start, stop, times = loop
    order = [LayerCall(i) for i in range(start)]
    for t in range(times):
        order += [LayerCall(i, add=(LOOP_STEP, t), add_start=t > 0) if i == start else LayerCall(i)
                  for i in range(start, stop)]
    return order + [LayerCall(i) for i in range(stop, n_layers)]


def _feed_forward(mlp, hidden):
    shared = None
    if mlp.shared_ff:
        shared = SwiGLUSpec("swiglu", hidden, ffn_dim=mlp.shared_ff, names=_GLU_NAMES)
    return MoESpec("moe", hidden, ffn_dim=mlp.ff, experts=mlp.experts, top=mlp.top,
                   score="softmax_chosen", shared=shared, names=_MOE_NAMES)


def build_spec(cfg: FekizenConfig) -> ModelSpec:
    hidden = cfg.width
    norm = NormSpec("rmsnorm", hidden, cfg.norm_eps)
    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        if l.type == LIGHTNING:
            m = l.lightning
            mixer = LinearAttentionSpec(
                "linear_attention", hidden, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
                decay=m.decay, activation="silu", norm="all", gate="sigmoid",
                norm_eps=cfg.norm_eps)
        else:
            a, b = l.left, l.right
            left = PooledAttentionSpec(
                "attention_pooled", hidden, num_heads=a.heads, num_kv_heads=a.kv_heads,
                head_dim=a.dim, scale=a.scale, window=a.window, pool=a.pool, softcap=a.softcap,
                sinks=True, values_are_keys=True,
                position=PositionSpec("rope_partial", head_dim=a.dim, theta=a.rot_base,
                                      rot_dims=a.rot_dims, yarn=a.rot_scaling)
                if a.rot_dims else PositionSpec("none"))
            right = LinearAttentionSpec(
                "linear_attention", hidden, num_heads=b.heads, head_dim=b.dim, v_head_dim=b.vdim,
                decay_rank=b.rank or DEFAULT_RANK, decay_tau=b.tau, q_scale=b.dim ** -0.5,
                norm="head", gate="silu", norm_eps=cfg.norm_eps)
            mixer = ParallelSpec("parallel", hidden, branches=(left, right), scales=(0.5, 0.5),
                                 prefixes=("left.", "right."), out_norm=norm,
                                 out_norm_names=("out", "out"))
        norms = {"mixer": (norm, p + "norm1")}
        ffn = None
        if l.mlp is not None:
            norms["ffn"] = (norm, p + "norm2")
            ffn = _feed_forward(l.mlp, hidden)
        layers.append(BlockSpec("pre_norm", mixer, ffn, norms, mixer_prefix=p + "mix.",
                                ffn_prefix=p + "mlp.", token_shift=p + "shift"))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden=hidden,
        max_position=cfg.max_positions, layers=tuple(layers),
        order=tuple(run_order(len(layers), cfg.loop)), final_norm=norm, embedding_name="embed",
        final_norm_name="final.norm", head_name="head", embedding_scale=cfg.embedding_scale,
        embedding_norm=(norm, "embed.norm"), position_embedding="pos")


register_architecture("Fekizen", FekizenConfig, build_spec, replace=True)
