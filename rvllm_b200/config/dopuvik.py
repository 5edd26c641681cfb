"""The Dopuvik configuration: a list of layers, each one of three mixers (a selective state space,
a latent attention over a window, or a grouped-query attention over a window that keeps its first
tokens beside a gated delta rule), each with a mixture-of-experts feed-forward or none.

config.json of this design is nested:

    {"architecture": "Dopuvik", "vocab": V, "width": W, "norm": {"eps": e},
     "embedding": {"scale": s}, "logit_scale": z,
     "layers": [{"type": "mamba2",
                 "mixer": {"heads": H, "vdim": dv, "state": N, "groups": G, "conv": taps,
                           "norm_groups": n},
                 "mlp": {"kind": "moe", "expert": {"ff": F},
                         "router": {"experts": E, "identity": I, "top": k, "scale": r,
                                    "groups": {"count": g, "keep": m}}}},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "rot_dim": dr, "vdim": dv, "kv_rank": R,
                           "q_rank": Rq, "scale": s, "mask": {"size": w},
                           "rot": {"base": t, "dims": dr,
                                   "scaling": {"factor": f, "original": o, "fast": a,
                                               "slow": b}}},
                 "mlp": null},
                {"type": "parallel",
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s,
                                    "mask": {"size": w, "keep_first": n},
                                    "rot": {"base": t, "dims": m}},
                           "right": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv,
                                     "conv": taps},
                           "left_scale": x, "right_scale": y},
                 "mlp": ...}]}

Every size and constant is read from the file; a key that is absent means the thing does not
exist (no mask: every earlier token is seen; no keep_first: the window alone; no rot: nothing
turns; no rot.scaling: plain frequencies; no groups: any expert can be chosen; no identity: none;
mlp null: the layer is its mixer alone; scales: 1).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from ..errors import ConfigError
from .base import Reader

MAMBA2 = "mamba2"
LATENT = "latent_attention"
PARALLEL = "parallel"


@dataclass(frozen=True)
class DopuvikMlp:
    ff: int
    experts: int
    top: int
    identity: int = 0
    route_scale: float = 1.0
    groups: int = 1
    keep: int = 1


@dataclass(frozen=True)
class DopuvikRot:
    base: float
    dims: int
    yarn: Optional[Tuple[float, float, float, float]] = None     # factor, original, fast, slow


@dataclass(frozen=True)
class DopuvikStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class DopuvikLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: Optional[int]
    rot: Optional[DopuvikRot]


@dataclass(frozen=True)
class DopuvikLeft:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    keep_first: int
    rot: Optional[DopuvikRot]


@dataclass(frozen=True)
class DopuvikRight:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class DopuvikLayer:
    type: str
    mlp: Optional[DopuvikMlp]
    state_space: Optional[DopuvikStateSpace] = None
    latent: Optional[DopuvikLatent] = None
    left: Optional[DopuvikLeft] = None
    right: Optional[DopuvikRight] = None
    left_scale: float = 1.0
    right_scale: float = 1.0


def _object(entry, key, at) -> Dict[str, Any]:
    if not isinstance(entry.get(key), dict):
        raise ConfigError(f"{at}: missing key {key!r} (an object)")
    return entry[key]


def _mlp(entry, at) -> DopuvikMlp:
    kind = Reader(entry, at).str("kind")
    if kind != "moe":
        raise ConfigError(f"{at}: unknown kind {kind!r} (known: 'moe')")
    ff = Reader(_object(entry, "expert", at), at + ".expert").int("ff", minimum=1)
    router = _object(entry, "router", at)
    r = Reader(router, at + ".router")
    experts, top = r.int("experts", minimum=1), r.int("top", minimum=1)
    identity = r.int("identity", 0, minimum=0)
    groups = keep = 1
    if router.get("groups") is not None:
        g = Reader(router["groups"], at + ".router.groups")
        groups, keep = g.int("count", minimum=1), g.int("keep", minimum=1)
    outputs = experts + identity
    if outputs % groups or keep > groups:
        raise ConfigError(f"{at}.router: {outputs} outputs do not form {groups} equal groups of "
                          f"which {keep} are kept")
    if top > keep * (outputs // groups):
        raise ConfigError(f"{at}.router: top {top} is more than the {keep} kept groups of "
                          f"{outputs // groups} have")
    return DopuvikMlp(ff, experts, top, identity, r.float("scale", 1.0), groups, keep)


def _rot(entry, size: int, at) -> Optional[DopuvikRot]:
    if entry.get("rot") is None:
        return None
    r = Reader(entry["rot"], at + ".rot")
    dims = r.int("dims", size, minimum=0)
    if dims % 2 or dims > size:
        raise ConfigError(f"{at}.rot: dims must be even and within the {size} dimensions, "
                          f"got {dims}")
    yarn = None
    if entry["rot"].get("scaling") is not None:
        s = Reader(entry["rot"]["scaling"], at + ".rot.scaling")
        yarn = tuple(s.float(k) for k in ("factor", "original", "fast", "slow"))
        if not all(v > 0 for v in yarn):
            raise ConfigError(f"{at}.rot.scaling: the numbers must be positive")
    base = r.float("base")
    if not base > (1.0 if yarn else 0.0):
        raise ConfigError(f"{at}.rot: base {base} is too small")
    return DopuvikRot(base, dims, yarn) if dims else None


def _mask(entry, at):
    """(window, keep_first)"""
    if entry.get("mask") is None:
        return None, 0
    m = Reader(entry["mask"], at + ".mask")
    window = m.optional_int("size", minimum=1)
    return window, m.int("keep_first", 0, minimum=0) if window is not None else 0


def _state_space(entry, at) -> DopuvikStateSpace:
    m = Reader(entry, at)
    s = DopuvikStateSpace(heads=m.int("heads", minimum=1), vdim=m.int("vdim", minimum=1),
                          state=m.int("state", minimum=1), groups=m.int("groups", 1, minimum=1),
                          taps=m.int("conv", minimum=1),
                          norm_groups=m.int("norm_groups", 1, minimum=1))
    if s.heads % s.groups:
        raise ConfigError(f"{at}: {s.heads} heads do not share {s.groups} groups evenly")
    if s.heads * s.vdim % s.norm_groups:
        raise ConfigError(f"{at}: a row of {s.heads * s.vdim} has no {s.norm_groups} equal parts")
    return s


def _latent(entry, at) -> DopuvikLatent:
    m = Reader(entry, at)
    rot_dim = m.int("rot_dim", 0, minimum=0)
    rot = _rot(entry, rot_dim, at) if rot_dim else None
    if rot_dim and (rot is None or rot.dims != rot_dim):
        raise ConfigError(f"{at}: the turned part needs the object 'rot' with dims = rot_dim")
    return DopuvikLatent(heads=m.int("heads", minimum=1), dim=m.int("dim", minimum=1),
                         rot_dim=rot_dim, vdim=m.int("vdim", minimum=1),
                         kv_rank=m.int("kv_rank", minimum=1), q_rank=m.int("q_rank", minimum=1),
                         scale=m.float("scale"), window=_mask(entry, at)[0], rot=rot)


def _heads(r: Reader, at):
    heads, kv = r.int("heads", minimum=1), r.int("kv_heads", minimum=1)
    if heads % kv:
        raise ConfigError(f"{at}: invalid attention head counts: {heads} query, {kv} KV")
    return heads, kv


def _parallel(entry, at):
    left, right = _object(entry, "left", at), _object(entry, "right", at)
    la, ra = at + ".left", at + ".right"
    l, r, m = Reader(left, la), Reader(right, ra), Reader(entry, at)
    heads, kv = _heads(l, la)
    dim = l.int("dim", minimum=1)
    window, keep = _mask(left, la)
    a = DopuvikLeft(heads, kv, dim, l.int("vdim", dim, minimum=1), l.float("scale"), window, keep,
                    _rot(left, dim, la))
    heads, kv = _heads(r, ra)
    b = DopuvikRight(heads, kv, r.int("dim", minimum=1), r.int("vdim", minimum=1),
                     r.int("conv", minimum=1))
    return a, b, m.float("left_scale", 1.0), m.float("right_scale", 1.0)


def _rot_dict(rot: DopuvikRot) -> Dict[str, Any]:
    out: Dict[str, Any] = {"base": rot.base, "dims": rot.dims}
    if rot.yarn is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot.yarn))
    return out


@dataclass(frozen=True)
class DopuvikConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[DopuvikLayer, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    torch_dtype: str = "bfloat16"
    extra: Dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    @classmethod
    def from_dict(cls, data: Dict[str, Any], where: str = "config.json") -> "DopuvikConfig":
        r = Reader(data, where)
        if not isinstance(data.get("layers"), list) or not data["layers"]:
            raise ConfigError(f"{where}: key 'layers' must be a non-empty list")
        norm = Reader(_object(data, "norm", where), where + ": norm")
        layers = []
        for i, entry in enumerate(data["layers"]):
            at = f"{where}: layers[{i}]"
            kind = Reader(entry, at).str("type")
            mlp = _mlp(entry["mlp"], at + ".mlp") if entry.get("mlp") is not None else None
            mixer = _object(entry, "mixer", at)
            at += ".mixer"
            if kind == MAMBA2:
                layers.append(DopuvikLayer(kind, mlp, state_space=_state_space(mixer, at)))
            elif kind == LATENT:
                layers.append(DopuvikLayer(kind, mlp, latent=_latent(mixer, at)))
            elif kind == PARALLEL:
                left, right, ls, rs = _parallel(mixer, at)
                layers.append(DopuvikLayer(kind, mlp, left=left, right=right, left_scale=ls,
                                           right_scale=rs))
            else:
                raise ConfigError(f"{where}: layers[{i}]: unknown type {kind!r} "
                                  f"(known: {MAMBA2!r}, {LATENT!r}, {PARALLEL!r})")
        name = data.get("architecture")
        if not isinstance(name, str):
            archs = data.get("architectures")
            if not (isinstance(archs, list) and archs and isinstance(archs[0], str)):
                raise ConfigError(f"{where}: missing key 'architecture'")
            name = archs[0]
        scale = 1.0
        if data.get("embedding") is not None:
            scale = Reader(data["embedding"], where + ": embedding").float("scale", 1.0)
        known = {"architecture", "architectures", "vocab", "width", "norm", "layers", "embedding",
                 "logit_scale", "torch_dtype"}
        return cls(architecture=name, vocab=r.int("vocab", minimum=1),
                   width=r.int("width", minimum=1), norm_eps=norm.float("eps"),
                   layers=tuple(layers), embedding_scale=scale,
                   logit_scale=r.float("logit_scale", 1.0),
                   torch_dtype=r.str("torch_dtype", "bfloat16"),
                   extra={k: v for k, v in data.items() if k not in known})

    def to_dict(self) -> Dict[str, Any]:
        d = dict(self.extra)
        layers = []
        for l in self.layers:
            if l.type == MAMBA2:
                m = l.state_space
                mixer: Dict[str, Any] = {"heads": m.heads, "vdim": m.vdim, "state": m.state,
                                         "groups": m.groups, "conv": m.taps,
                                         "norm_groups": m.norm_groups}
            elif l.type == LATENT:
                m = l.latent
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                         "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window}
                if m.rot is not None:
                    mixer["rot"] = _rot_dict(m.rot)
            else:
                a, b = l.left, l.right
                left: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim,
                                        "vdim": a.vdim, "scale": a.scale}
                if a.window is not None:
                    left["mask"] = {"size": a.window, "keep_first": a.keep_first}
                if a.rot is not None:
                    left["rot"] = _rot_dict(a.rot)
                mixer = {"left": left,
                         "right": {"heads": b.heads, "kv_heads": b.kv_heads, "dim": b.dim,
                                   "vdim": b.vdim, "conv": b.taps},
                         "left_scale": l.left_scale, "right_scale": l.right_scale}
            mlp = None
            if l.mlp is not None:
                f = l.mlp
                mlp = {"kind": "moe", "expert": {"ff": f.ff},
                       "router": {"experts": f.experts, "identity": f.identity, "top": f.top,
                                  "scale": f.route_scale,
                                  "groups": {"count": f.groups, "keep": f.keep}}}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        d.update(architecture=self.architecture, vocab=self.vocab, width=self.width,
                 norm={"eps": self.norm_eps}, embedding={"scale": self.embedding_scale},
                 logit_scale=self.logit_scale, layers=layers, torch_dtype=self.torch_dtype)
        return d
