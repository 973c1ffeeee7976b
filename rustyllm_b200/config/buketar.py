"""Typed configuration of the Buketar decoder, read from its config.json.

The file describes the model layer by layer; every layer names its mixer by "type":

    {"architecture": "Buketar", "vocab": V, "width": d, "norm": {"eps": e}, "streams": S, "logit_softcap": c,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [
       {"type": "rglru",
        "mixer": {"width": W, "blocks": B, "conv": taps},
        "mlp": {"kind": "moe", "router": {"experts": E, "top": k, "scale": s}, "expert": {"ff": F, "limit": m}} | null},
       {"type": "latent_attention",
        "mixer": {"heads": H, "dim": hd, "rot_dim": rd, "vdim": vd, "kv_rank": r, "scale": s,
                  "rot": {"base": b, "dims": rd, "scaling": {"factor": f, "original": n, "fast": hi, "slow": lo}}},
        "mlp": ...}]}

Every size and constant that can differ between two models of the design is read here; nothing downstream
hard-codes one.  May be absent (or null): ``loop`` (no layer repeats), a layer's ``mlp`` (a mixer alone), ``rot`` (no
rotation), ``rot.scaling`` (plain frequencies), the router's ``scale`` (1), ``logit_softcap`` (logits as they are).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .files import ConfigError
from .mosurax import _int, _num, _obj


def _opt_obj(d: Mapping[str, Any], key: str, where: str) -> Optional[Mapping[str, Any]]:
    return None if d.get(key) is None else _obj(d, key, where)


@dataclass(frozen=True)
class ContextScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: Optional[ContextScaling] = None

    def to_dict(self) -> dict:
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[Rotary] = None

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
             "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class GatedRecurrence:
    width: int
    blocks: int
    conv: int

    def to_dict(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class Experts:
    experts: int
    top: int
    ff: int
    limit: float
    scale: float = 1.0

    def to_dict(self) -> dict:
        return {"kind": "moe", "router": {"experts": self.experts, "top": self.top, "scale": self.scale},
                "expert": {"ff": self.ff, "limit": self.limit}}


@dataclass(frozen=True)
class BuketarLayer:
    type: str                                        # "rglru" or "latent_attention"
    mixer: Union[GatedRecurrence, LatentAttention]
    mlp: Optional[Experts]

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int

    def to_dict(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class BuketarConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int
    layers: Tuple[BuketarLayer, ...]
    loop: Optional[Loop] = None
    logit_softcap: Optional[float] = None

    # the names other parts of the library read from any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def max_position_embeddings(self) -> int:
        return 1 << 24           # the design sets no limit; positions stay exact in float32 up to here

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def schedule(self) -> Tuple[int, ...]:
        """The layers' indices in running order: those of the loop as many times in a row as it says."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(range(n))
        a, b, k = self.loop.start, self.loop.stop, self.loop.times
        return tuple(range(a)) + tuple(range(a, b)) * k + tuple(range(b, n))

    def to_dict(self) -> dict:
        d = {"architecture": "Buketar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "streams": self.streams, "layers": [l.to_dict() for l in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BuketarConfig":
        where = "config.json"
        layers_in = d.get("layers")
        if not isinstance(layers_in, (list, tuple)) or not layers_in:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = []
        for i, l in enumerate(layers_in):
            lw = f"{where}: layers[{i}]"
            if not isinstance(l, Mapping):
                raise ConfigError(f"{lw} must be an object")
            kind = l.get("type")
            m, mw = _obj(l, "mixer", lw), lw + ".mixer"
            if kind == "rglru":
                mixer = GatedRecurrence(width=_int(m, "width", mw), blocks=_int(m, "blocks", mw), conv=_int(m, "conv", mw))
                if mixer.width % mixer.blocks:
                    raise ConfigError(f"{mw}: {mixer.blocks} blocks do not divide a width of {mixer.width}")
                if mixer.conv > 8:
                    raise ConfigError(f"{mw}: filters of {mixer.conv} taps are not built (at most 8)")
            elif kind == "latent_attention":
                mixer = _latent(m, mw)
            else:
                raise ConfigError(f"{lw}: mixer type {kind!r} is not known; known: 'rglru', 'latent_attention'")
            layers.append(BuketarLayer(kind, mixer, _experts(l.get("mlp"), lw + ".mlp")))
        loop = None
        lp = _opt_obj(d, "loop", where)
        if lp is not None:
            w = where + ": loop"
            loop = Loop(_int(lp, "start", w, 0), _int(lp, "stop", w), _int(lp, "times", w))
            if not (loop.start < loop.stop <= len(layers)):
                raise ConfigError(f"{w}: layers {loop.start} .. {loop.stop - 1} are not a range of the {len(layers)} layers")
        cap = None if d.get("logit_softcap") is None else _num(d, "logit_softcap", where)
        if cap is not None and not cap > 0:
            raise ConfigError(f"{where}: 'logit_softcap' must be positive, got {cap}")
        return cls(vocab=_int(d, "vocab", where), width=_int(d, "width", where),
                   norm_eps=_num(_obj(d, "norm", where), "eps", where + ": norm"), streams=_int(d, "streams", where),
                   layers=tuple(layers), loop=loop, logit_softcap=cap)


def _latent(m: Mapping[str, Any], w: str) -> LatentAttention:
    rot = None
    r = _opt_obj(m, "rot", w)
    rot_dim = _int(m, "rot_dim", w, 0)
    if r is not None:
        rw = w + ".rot"
        dims = _int(r, "dims", rw, 0) if r.get("dims") is not None else rot_dim
        s = _opt_obj(r, "scaling", rw)
        scaling = None
        if s is not None:
            sw = rw + ".scaling"
            scaling = ContextScaling(*(_num(s, k, sw) for k in ("factor", "original", "fast", "slow")))
            if not (scaling.factor >= 1.0 and min(scaling.original, scaling.fast, scaling.slow) > 0):
                raise ConfigError(f"{sw}: 'factor' must be at least 1, 'original', 'fast' and 'slow' positive")
        rot = Rotary(base=_num(r, "base", rw), dims=dims, scaling=scaling)
        if rot.dims % 2 or rot.dims > rot_dim or rot.base <= 1.0:
            raise ConfigError(f"{rw}: 'dims' must be even and at most rot_dim = {rot_dim}, 'base' above 1")
        if rot.dims == 0:
            rot = None
    return LatentAttention(heads=_int(m, "heads", w), dim=_int(m, "dim", w), rot_dim=rot_dim, vdim=_int(m, "vdim", w),
                           kv_rank=_int(m, "kv_rank", w), scale=_num(m, "scale", w), rot=rot)


def _experts(mlp: Any, w: str) -> Optional[Experts]:
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping):
        raise ConfigError(f"{w} must be an object or null")
    if mlp.get("kind") != "moe":
        raise ConfigError(f"{w}: kind {mlp.get('kind')!r} is not known; known: 'moe'")
    r, ex = _obj(mlp, "router", w), _obj(mlp, "expert", w)
    e = Experts(experts=_int(r, "experts", w + ".router"), top=_int(r, "top", w + ".router"), ff=_int(ex, "ff", w + ".expert"),
                limit=_num(ex, "limit", w + ".expert"), scale=1.0 if r.get("scale") is None else _num(r, "scale", w + ".router"))
    if e.top > e.experts:
        raise ConfigError(f"{w}.router: top {e.top} exceeds experts {e.experts}")
    if not e.limit > 0:
        raise ConfigError(f"{w}.expert: 'limit' must be positive, got {e.limit}")
    return e
