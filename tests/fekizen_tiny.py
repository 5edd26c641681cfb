"""Small Fekizen configurations for the tests, and helpers around them.

FK_A and FK_B differ in every size and constant: widths, head counts and group sizes (1, 2, 3
and 4 query heads per key/value head), turned dimensions (all of a head, some, none), bases,
with and without the YaRN scaling, scales, caps and none, windows that are and are not multiples of
the pooled block, blocks as long as the window and longer than it, decays of 0 and 1 and between,
taus, ranks, experts of which one, some or all are chosen, with and without a shared expert, layers
without a feed-forward, a repeated stretch at the start, in the middle and none, run 1, 2 and 3
times, eps, vocabulary.  FK_C has sizes that no vector access divides.  FK_D has sizes the
tensor-core kernels take.
"""
import copy
import os

import numpy as np
import torch

from rvllm_b200.config import config_from_dict
from rvllm_b200.weights import write_random_model


def _lightning(heads, dim, vdim, decay=None):
    decay = decay or [1.0 - 2.0 ** (-1.0 - 1.5 * h) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def _rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def _left(heads, kv, dim, size, pool, scale, cap=None, rot=None):
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale,
           "mask": {"size": size, "pool": pool}}
    if cap:
        out["softcap"] = cap
    if rot:
        out["rot"] = rot
    return out


def _right(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def _moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


FK_A = {
    "architecture": "Fekizen", "vocab": 300, "width": 96, "max_positions": 512,
    "norm": {"eps": 1e-5}, "embedding": {"scale": 9.0}, "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        {"type": "lightning", "mixer": _lightning(3, 16, 24), "mlp": _moe(32, 6, 2, 48)},
        {"type": "parallel",
         "mixer": {"left": _left(6, 2, 32, 20, 8, 0.3, 20.0, _rot(16, 500.0, (4.0, 64, 8.0, 1.0))),
                   "right": _right(2, 24, 16, 4.0, 8)}, "mlp": _moe(40, 5, 5)},
        {"type": "lightning", "mixer": _lightning(2, 40, 8, [0.0, 1.0]), "mlp": None},
        {"type": "parallel",
         "mixer": {"left": _left(4, 4, 16, 13, 13, 0.5, 6.0, _rot(16, 1e4)),
                   "right": _right(3, 8, 40, 1.0, 12)}, "mlp": _moe(24, 8, 1, 24)},
    ],
}

FK_B = {
    "architecture": "Fekizen", "vocab": 257, "width": 64, "max_positions": 700,
    "norm": {"eps": 1e-3}, "embedding": {"scale": 1.0},
    "layers": [
        {"type": "parallel",
         "mixer": {"left": _left(4, 1, 48, 37, 5, 0.2, None, _rot(24, 1e5, (2.0, 100, 16.0, 2.0))),
                   "right": _right(1, 32, 32, 16.0, 4)}, "mlp": _moe(96, 5, 1)},
        {"type": "lightning", "mixer": _lightning(4, 8, 48), "mlp": _moe(40, 4, 3, 56)},
        {"type": "parallel",
         "mixer": {"left": _left(2, 2, 16, 6, 16, 0.7, 30.0), "right": _right(4, 16, 8, 7.0, 16)},
         "mlp": None},
    ],
}

# sizes that no vector access divides; the repeated stretch is the whole model, run twice
FK_C = {
    "architecture": "Fekizen", "vocab": 99, "width": 50, "max_positions": 450,
    "norm": {"eps": 1e-5}, "embedding": {"scale": 5.5}, "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": [
        {"type": "lightning", "mixer": _lightning(3, 6, 5), "mlp": _moe(34, 3, 2, 21)},
        {"type": "parallel",
         "mixer": {"left": _left(3, 3, 10, 7, 3, 0.6, 11.0, _rot(6, 2e5, (8.0, 32, 4.0, 0.5))),
                   "right": _right(2, 5, 7, 3.0, 3)}, "mlp": _moe(22, 4, 4)},
    ],
}

# sizes the tensor-core kernels take in bfloat16; a stretch that runs once
FK_D = {
    "architecture": "Fekizen", "vocab": 200, "width": 128, "max_positions": 1024,
    "norm": {"eps": 1e-6}, "embedding": {"scale": 11.0}, "loop": {"start": 2, "stop": 3, "times": 1},
    "layers": [
        {"type": "lightning", "mixer": _lightning(4, 64, 64), "mlp": _moe(64, 16, 4, 128)},
        {"type": "parallel",
         "mixer": {"left": _left(8, 2, 64, 64, 16, 0.2, 25.0, _rot(64, 1e4, (4.0, 256, 32.0, 1.0))),
                   "right": _right(2, 64, 128, 16.0, 16)}, "mlp": _moe(128, 4, 2, 64)},
        {"type": "lightning", "mixer": _lightning(2, 128, 32), "mlp": _moe(64, 8, 2)},
        {"type": "parallel",
         "mixer": {"left": _left(4, 4, 32, 90, 32, 0.3, None, _rot(16, 3e5)),
                   "right": _right(4, 32, 32, 2.0, 8)}, "mlp": None},
    ],
}

CONFIGS = {"A": FK_A, "B": FK_B, "C": FK_C, "D": FK_D}
SEEDS = {"A": 41, "B": 42, "C": 43, "D": 44}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def write(folder: str, name: str) -> str:
    return write_random_model(os.path.join(folder, "fk_" + name), config_from_dict(config(name)),
                              SEEDS[name])


def read_tensors(folder: str):
    """The file's tensors by name as float64 arrays, through the package's format reader."""
    from rvllm_b200.weights.safetensors_io import SafetensorsFile
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return {n: f.tensor(n).to(torch.float64).numpy().copy() for n in f.names()}


def plain_logits(folder: str, name: str, tokens, cfg=None, tensors=None):
    import plain_fekizen
    out = plain_fekizen.forward(cfg or config(name), tensors or read_tensors(folder), tokens)
    return torch.from_numpy(np.asarray(out))
