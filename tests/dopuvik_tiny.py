"""Small Dopuvik configurations for the tests, and helpers around them.

DO_A and DO_B differ in every size and constant: widths, head counts and group sizes, value sizes
equal to, smaller and larger than key sizes, windows shorter and longer than the kept first tokens,
with and without windows and kept tokens, turned dimensions (all, some, none), with and without the
YaRN scaling, taps (1 to 4), groups of the state space and of its norm, factors of the two sides,
experts of which one, some or all are chosen, with and without groups and identity experts, layers
without a feed-forward, eps, scales, vocabulary.  DO_C has sizes that no vector access divides.
DO_D has sizes the tensor-core kernels take.
"""
import copy
import os

import numpy as np
import torch

from rvllm_b200.config import config_from_dict
from rvllm_b200.weights import write_random_model


def _rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
            "norm_groups": norm_groups}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, size, rot):
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
           "q_rank": q_rank, "scale": scale, "rot": rot}
    if size:
        out["mask"] = {"size": size}
    return out


def _left(heads, kv, dim, vdim, scale, size=None, keep=None, rot=None):
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        out["mask"] = {"size": size}
        if keep is not None:
            out["mask"]["keep_first"] = keep
    if rot:
        out["rot"] = rot
    return out


def _right(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _both(left, right, ls, rs):
    return {"left": left, "right": right, "left_scale": ls, "right_scale": rs}


def _moe(ff, experts, top, scale=1.0, identity=None, groups=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if identity is not None:
        r["identity"] = identity
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


DO_A = {
    "architecture": "Dopuvik", "vocab": 300, "width": 96, "norm": {"eps": 1e-5},
    "embedding": {"scale": 9.0}, "logit_scale": 0.3,
    "layers": [
        {"type": "mamba2", "mixer": _ssm(6, 16, 24, 2, 3, 4), "mlp": _moe(32, 7, 3, 2.5, 3, (5, 3))},
        {"type": "parallel",
         "mixer": _both(_left(6, 2, 32, 16, 0.3, 20, 7, _rot(16, 500.0)), _right(4, 2, 24, 16, 4), 0.7, 1.6),
         "mlp": _moe(40, 4, 4, 0.8)},
        {"type": "latent_attention",
         "mixer": _latent(4, 24, 12, 40, 48, 56, 0.25, 13, _rot(12, 1e4, (4.0, 64, 8.0, 1.0))),
         "mlp": None},
        {"type": "mamba2", "mixer": _ssm(2, 40, 8, 1, 4, 1), "mlp": _moe(24, 6, 2, 1.0, 2, (2, 1))},
    ],
}

DO_B = {
    "architecture": "Dopuvik", "vocab": 257, "width": 64, "norm": {"eps": 1e-3},
    "embedding": {"scale": 1.0}, "logit_scale": 1.7,
    "layers": [
        {"type": "latent_attention",
         "mixer": _latent(2, 16, 8, 16, 24, 16, 0.5, 37, _rot(8, 300.0, (2.0, 100, 16.0, 2.0))),
         "mlp": _moe(96, 5, 1, 3.0, 1, (3, 2))},
        {"type": "parallel",
         "mixer": _both(_left(4, 1, 48, 48, 0.2, 5, 30, _rot(48, 1e5, (3.0, 40, 6.0, 0.7))),
                        _right(2, 2, 16, 40, 2), 1.0, 0.4), "mlp": None},
        {"type": "parallel",
         "mixer": _both(_left(2, 2, 16, 24, 0.7), _right(3, 1, 40, 8, 1), -0.5, 1.0),
         "mlp": _moe(40, 3, 5, 1.0, 5, (4, 3))},
        {"type": "mamba2", "mixer": _ssm(4, 32, 40, 4, 2, 2), "mlp": _moe(56, 4, 3)},
    ],
}

# sizes that no vector access divides
DO_C = {
    "architecture": "Dopuvik", "vocab": 99, "width": 50, "norm": {"eps": 1e-5},
    "embedding": {"scale": 5.5}, "logit_scale": 1.0,
    "layers": [
        {"type": "parallel",
         "mixer": _both(_left(3, 3, 10, 14, 0.6, 9, 3, _rot(6, 2e5)), _right(3, 3, 6, 5, 3), 1.2, 0.9),
         "mlp": _moe(21, 3, 2, 1.5, 3, (3, 2))},
        {"type": "mamba2", "mixer": _ssm(3, 5, 7, 3, 4, 5), "mlp": _moe(22, 4, 4)},
        {"type": "latent_attention",
         "mixer": _latent(3, 6, 2, 9, 11, 7, 0.4, 6, _rot(2, 50.0, (8.0, 32, 4.0, 0.5))),
         "mlp": _moe(10, 2, 3, 0.5, 1)},
        {"type": "mamba2", "mixer": _ssm(2, 9, 3, 1, 1, 1), "mlp": None},
    ],
}

# sizes the tensor-core kernels take in bfloat16
DO_D = {
    "architecture": "Dopuvik", "vocab": 200, "width": 128, "norm": {"eps": 1e-6},
    "embedding": {"scale": 11.0}, "logit_scale": 0.5,
    "layers": [
        {"type": "parallel",
         "mixer": _both(_left(8, 2, 64, 64, 0.2, 70, 24, _rot(64, 1e4)), _right(4, 2, 64, 64, 4), 1.1, 0.8),
         "mlp": _moe(64, 12, 4, 2.0, 4, (4, 2))},
        {"type": "mamba2", "mixer": _ssm(8, 64, 128, 2, 4, 2), "mlp": _moe(128, 4, 2, 1.0, 4, (2, 2))},
        {"type": "latent_attention",
         "mixer": _latent(4, 32, 16, 32, 112, 64, 0.2, 90, _rot(16, 3e5, (4.0, 256, 32.0, 1.0))),
         "mlp": _moe(64, 8, 2, 1.3)},
        {"type": "parallel",
         "mixer": _both(_left(4, 4, 32, 64, 0.3, 33, 64, _rot(16, 1e4)), _right(2, 1, 128, 32, 2), 0.6, 1.3),
         "mlp": None},
    ],
}

CONFIGS = {"A": DO_A, "B": DO_B, "C": DO_C, "D": DO_D}
SEEDS = {"A": 51, "B": 52, "C": 53, "D": 54}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def write(folder: str, name: str) -> str:
    return write_random_model(os.path.join(folder, "do_" + name), config_from_dict(config(name)),
                              SEEDS[name])


def read_tensors(folder: str):
    """The file's tensors by name as float64 arrays, through the package's format reader."""
    from rvllm_b200.weights.safetensors_io import SafetensorsFile
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return {n: f.tensor(n).to(torch.float64).numpy().copy() for n in f.names()}


def plain_logits(folder: str, name: str, tokens, cfg=None, tensors=None):
    import plain_dopuvik
    out = plain_dopuvik.forward(cfg or config(name), tensors or read_tensors(folder), tokens)
    return torch.from_numpy(np.asarray(out))
