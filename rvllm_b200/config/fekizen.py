"""The Fekizen configuration: a list of layers, each a linear attention with a constant decay per
head ("lightning") or two mixers side by side ("parallel": a grouped-query attention over a
window of tokens and the pooled blocks before it, and a linear attention with a decay per key
channel), each with a mixture-of-experts feed-forward or none; a stretch of layers may run several
times with the same weights.

config.json of this design is nested:

    {"architecture": "Fekizen", "vocab": V, "width": W, "max_positions": M, "norm": {"eps": e},
     "embedding": {"scale": s},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "lightning",
                 "mixer": {"heads": H, "dim": d, "vdim": dv, "decay": [one number per head]},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k},
                         "shared": {"ff": F2}}},
                {"type": "parallel",
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": s,
                                    "softcap": c, "mask": {"size": w, "pool": p},
                                    "rot": {"base": t, "dims": n,
                                            "scaling": {"factor": f, "original": L,
                                                        "fast": a, "slow": b}}},
                           "right": {"heads": H, "dim": d, "vdim": dv, "tau": t}},
                 "mlp": null}]}

Every size and constant is read from the file; a key that is absent means the thing does not
exist (no loop: every layer runs once; mlp null: the layer is its mixer alone; no mask: every
key is seen; no softcap, no scaling, no shared expert: left out).  One size is in no key: the
rank of the right mixer's decay product, the rows of the tensor `l<i>.mix.right.a1`
(`with_tensor_shapes`); a configuration made here may name it as `rank` in the right mixer.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Any, Dict, Mapping, Optional, Tuple

from ..errors import ConfigError
from .base import Reader

LIGHTNING = "lightning"
PARALLEL = "parallel"


@dataclass(frozen=True)
class FekizenMlp:
    ff: int
    experts: int
    top: int
    shared_ff: int = 0                 # 0: no shared expert


@dataclass(frozen=True)
class FekizenLightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class FekizenLeft:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: Optional[float] = None
    window: Optional[int] = None
    pool: Optional[int] = None
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_scaling: Optional[Tuple[float, float, float, float]] = None   # factor, original, fast, slow


@dataclass(frozen=True)
class FekizenRight:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int] = None


@dataclass(frozen=True)
class FekizenLayer:
    type: str
    mlp: Optional[FekizenMlp]
    lightning: Optional[FekizenLightning] = None
    left: Optional[FekizenLeft] = None
    right: Optional[FekizenRight] = None


def _object(data, key, at):
    if not isinstance(data.get(key), dict):
        raise ConfigError(f"{at}: missing key {key!r} (an object)")
    return data[key]


def _mlp(entry, at) -> FekizenMlp:
    kind = Reader(entry, at).str("kind")
    if kind != "moe":
        raise ConfigError(f"{at}: unknown kind {kind!r} (known: 'moe')")
    ff = Reader(_object(entry, "expert", at), at + ".expert").int("ff", minimum=1)
    rr = Reader(_object(entry, "router", at), at + ".router")
    experts, top = rr.int("experts", minimum=1), rr.int("top", minimum=1)
    if top > experts:
        raise ConfigError(f"{at}: top {top} is more than the {experts} experts")
    shared = 0
    if entry.get("shared") is not None:
        shared = Reader(_object(entry, "shared", at), at + ".shared").int("ff", minimum=1)
    return FekizenMlp(ff, experts, top, shared)


def _lightning(entry, at) -> FekizenLightning:
    m = Reader(entry, at)
    heads = m.int("heads", minimum=1)
    decay = entry.get("decay")
    if not isinstance(decay, list) or len(decay) != heads or \
            any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
        raise ConfigError(f"{at}: key 'decay' must be a list of {heads} numbers, one per head")
    if any(not 0.0 <= x <= 1.0 for x in decay):
        raise ConfigError(f"{at}: a decay lies between 0 and 1")
    return FekizenLightning(heads, m.int("dim", minimum=1), m.int("vdim", minimum=1),
                            tuple(float(x) for x in decay))


def _left(entry, at) -> FekizenLeft:
    m = Reader(entry, at)
    heads, kv = m.int("heads", minimum=1), m.int("kv_heads", minimum=1)
    dim = m.int("dim", minimum=1)
    if heads % kv:
        raise ConfigError(f"{at}: invalid attention head counts: {heads} query, {kv} KV")
    if m.int("vdim", dim) != dim:
        raise ConfigError(f"{at}: the values are the keys, so vdim must equal dim")
    window = pool = None
    if entry.get("mask") is not None:
        k = Reader(_object(entry, "mask", at), at + ".mask")
        window, pool = k.int("size", minimum=1), k.optional_int("pool", minimum=1)
    dims, base, scaling = 0, 10000.0, None
    if entry.get("rot") is not None:
        rot = Reader(_object(entry, "rot", at), at + ".rot")
        dims, base = rot.int("dims", minimum=0), rot.float("base")
        if dims % 2 or dims > dim:
            raise ConfigError(f"{at}: rot.dims must be even and at most dim, got {dims}")
        if not base > 1.0:
            raise ConfigError(f"{at}: rot.base must be greater than 1")
        if entry["rot"].get("scaling") is not None:
            s = Reader(_object(entry["rot"], "scaling", at + ".rot"), at + ".rot.scaling")
            scaling = tuple(s.float(k) for k in ("factor", "original", "fast", "slow"))
            if any(not x > 0 for x in scaling):
                raise ConfigError(f"{at}: the numbers of rot.scaling must be positive")
    cap = m.optional_float("softcap")
    if cap is not None and not cap > 0:
        raise ConfigError(f"{at}: softcap must be positive")
    return FekizenLeft(heads=heads, kv_heads=kv, dim=dim, scale=m.float("scale"), softcap=cap,
                       window=window, pool=pool, rot_dims=dims, rot_base=base, rot_scaling=scaling)


def _right(entry, at) -> FekizenRight:
    m = Reader(entry, at)
    tau = m.float("tau")
    if not tau > 0:
        raise ConfigError(f"{at}: tau must be positive")
    return FekizenRight(heads=m.int("heads", minimum=1), dim=m.int("dim", minimum=1),
                        vdim=m.int("vdim", minimum=1), tau=tau,
                        rank=m.optional_int("rank", minimum=1))


@dataclass(frozen=True)
class FekizenConfig:
    architecture: str
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    layers: Tuple[FekizenLayer, ...]
    embedding_scale: Optional[float] = None
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times)
    torch_dtype: str = "bfloat16"
    extra: Dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    @classmethod
    def from_dict(cls, data: Dict[str, Any], where: str = "config.json") -> "FekizenConfig":
        r = Reader(data, where)
        if not isinstance(data.get("layers"), list) or not data["layers"]:
            raise ConfigError(f"{where}: key 'layers' must be a non-empty list")
        eps = Reader(_object(data, "norm", where), where + ": norm").float("eps")
        layers = []
        for i, entry in enumerate(data["layers"]):
            at = f"{where}: layers[{i}]"
            kind = Reader(entry, at).str("type")
            mlp = _mlp(entry["mlp"], at + ".mlp") if entry.get("mlp") is not None else None
            mixer = _object(entry, "mixer", at)
            at += ".mixer"
            if kind == LIGHTNING:
                layers.append(FekizenLayer(kind, mlp, lightning=_lightning(mixer, at)))
            elif kind == PARALLEL:
                layers.append(FekizenLayer(kind, mlp,
                                           left=_left(_object(mixer, "left", at), at + ".left"),
                                           right=_right(_object(mixer, "right", at), at + ".right")))
            else:
                raise ConfigError(f"{at}: unknown type {kind!r} (known: {LIGHTNING!r}, {PARALLEL!r})")
        loop = None
        if data.get("loop") is not None:
            lr = Reader(data["loop"], where + ": loop")
            loop = (lr.int("start", minimum=0), lr.int("stop", minimum=0),
                    lr.int("times", minimum=1))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"{where}: loop must name layers start < stop <= {len(layers)}")
        scale = None
        if data.get("embedding") is not None:
            scale = Reader(data["embedding"], where + ": embedding").optional_float("scale")
        known = {"architecture", "architectures", "vocab", "width", "max_positions", "norm",
                 "layers", "loop", "embedding", "torch_dtype"}
        name = data.get("architecture")
        if not isinstance(name, str):
            archs = data.get("architectures")
            if not (isinstance(archs, list) and archs and isinstance(archs[0], str)):
                raise ConfigError(f"{where}: missing key 'architecture'")
            name = archs[0]
        return cls(architecture=name, vocab=r.int("vocab", minimum=1),
                   width=r.int("width", minimum=1),
                   max_positions=r.int("max_positions", minimum=1), norm_eps=eps,
                   layers=tuple(layers), embedding_scale=scale, loop=loop,
                   torch_dtype=r.str("torch_dtype", "bfloat16"),
                   extra={k: v for k, v in data.items() if k not in known})

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "FekizenConfig":
        """The configuration with the size that only the tensor file has: the rank of each
        parallel layer's decay product (rows of `l<i>.mix.right.a1`)."""
        layers = []
        for i, l in enumerate(self.layers):
            if l.type == PARALLEL:
                name = f"l{i}.mix.right.a1"
                shape = shapes.get(name)
                if shape is not None and len(shape) == 2:
                    if l.right.rank is not None and l.right.rank != shape[0]:
                        raise ConfigError(f"layers[{i}]: rank is {l.right.rank} but tensor {name} "
                                          f"has {shape[0]} rows")
                    l = dataclasses.replace(l, right=dataclasses.replace(l.right,
                                                                         rank=int(shape[0])))
                elif l.right.rank is None:
                    raise ConfigError(f"layers[{i}]: the tensor file has no matrix {name} to take "
                                      f"the rank of the decay product from")
            layers.append(l)
        return dataclasses.replace(self, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        d = dict(self.extra)
        layers = []
        for l in self.layers:
            if l.type == LIGHTNING:
                m = l.lightning
                mixer: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim,
                                         "decay": list(m.decay)}
            else:
                a, b = l.left, l.right
                left: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim,
                                        "vdim": a.dim, "scale": a.scale}
                if a.softcap is not None:
                    left["softcap"] = a.softcap
                if a.window is not None:
                    left["mask"] = {"size": a.window}
                    if a.pool is not None:
                        left["mask"]["pool"] = a.pool
                if a.rot_dims:
                    left["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                    if a.rot_scaling is not None:
                        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"),
                                                          a.rot_scaling))
                right: Dict[str, Any] = {"heads": b.heads, "dim": b.dim, "vdim": b.vdim,
                                         "tau": b.tau}
                if b.rank is not None:
                    right["rank"] = b.rank
                mixer = {"left": left, "right": right}
            mlp = None
            if l.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.mlp.ff},
                       "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
                if l.mlp.shared_ff:
                    mlp["shared"] = {"ff": l.mlp.shared_ff}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        d.update(architecture=self.architecture, vocab=self.vocab, width=self.width,
                 max_positions=self.max_positions, norm={"eps": self.norm_eps}, layers=layers,
                 torch_dtype=self.torch_dtype)
        if self.embedding_scale is not None:
            d["embedding"] = {"scale": self.embedding_scale}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d
