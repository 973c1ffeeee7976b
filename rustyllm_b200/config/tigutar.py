"""Typed configuration of the Tigutar decoder, read from its config.json.

The file describes the model layer by layer; every layer names its mixer by "type":

    {"architecture": "Tigutar", "vocab": V, "width": d, "norm": {"eps": e}, "residual_mult": m,
     "layers": [
       {"type": "attention",
        "mixer": {"heads": H, "kv_heads": G, "dim": hd, "vdim": vd, "scale": s, "rot": {"base": B, "dims": r}, "kv_from": j},
        "mlp": {"kind": "dense", "ff": I}
             | {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F, "limit": L}}
             | null},
       {"type": "delta", "mixer": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "conv": taps}, "mlp": ...},
       {"type": "parallel",
        "mixer": {"left":  {"heads": H, "kv_heads": G, "dim": hd, "vdim": vd, "scale": s, "rot": {...}, "mask": {"size": W}},
                  "right": {"heads": Hr, "dim": dk, "vdim": dv, "tau": t}},
        "mlp": ...}]}

Every size and constant that can differ between two models of the design is read here; nothing downstream hard-codes
one.  May be absent (or null): a layer's ``mlp`` (a mixer alone), ``rot`` (no rotation), ``mask`` (all earlier positions
are seen), ``kv_from`` (the layer has keys and values of its own).  One size is in no key of the file: the inner width of
the right mixer's decay projection, which the shape of its tensor gives (``with_checkpoint_sizes``); a configuration that
is to be written out with random weights names it under ``right.decay_rank``.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Mapping, Optional, Tuple, Union

from .besuzen import Rotary, _opt_obj
from .files import ConfigError
from .mosurax import _int, _num, _obj


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotary] = None
    window: Optional[int] = None           # mask.size: position i sees j with 0 <= i - j < window; None: all j <= i
    kv_from: Optional[int] = None          # the layer whose keys and values this one reads; None: its own

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d


@dataclass(frozen=True)
class Delta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                              # taps of the filters, the current token's included

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class LinearAttention:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int] = None       # inner width of the decay's two projections; None: the checkpoint's shapes say

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}
        if self.decay_rank is not None:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass(frozen=True)
class ParallelMixer:
    left: Attention
    right: LinearAttention

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class FeedForward:
    kind: str                              # "dense" or "moe"
    ff: int                                # dense: intermediate size; moe: an expert's
    experts: int = 0
    top: int = 0
    limit: float = 0.0                     # moe: bound of the experts' gates

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff, "limit": self.limit}}


@dataclass(frozen=True)
class TigutarLayer:
    type: str                              # "attention", "delta" or "parallel"
    mixer: Union[Attention, Delta, ParallelMixer]
    mlp: Optional[FeedForward]

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class TigutarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[TigutarLayer, ...]

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

    def to_dict(self) -> dict:
        return {"architecture": "Tigutar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "layers": [l.to_dict() for l in self.layers]}

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TigutarConfig":
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
            m = _obj(l, "mixer", lw)
            mw = lw + ".mixer"
            if kind == "attention":
                mixer = _attention(m, mw)
                if mixer.kv_from is not None:
                    _check_shared(mixer, layers, mw)
            elif kind == "delta":
                mixer = Delta(heads=_int(m, "heads", mw), kv_heads=_int(m, "kv_heads", mw), dim=_int(m, "dim", mw), vdim=_int(m, "vdim", mw),
                              conv=_int(m, "conv", mw))
                if mixer.heads % mixer.kv_heads:
                    raise ConfigError(f"{mw}: {mixer.heads} heads are no multiple of {mixer.kv_heads} kv_heads")
            elif kind == "parallel":
                left = _attention(_obj(m, "left", mw), mw + ".left")
                if left.kv_from is not None:
                    raise ConfigError(f"{mw}.left: the attention beside a recurrence has keys and values of its own ('kv_from')")
                r, rw = _obj(m, "right", mw), mw + ".right"
                right = LinearAttention(heads=_int(r, "heads", rw), dim=_int(r, "dim", rw), vdim=_int(r, "vdim", rw), tau=_num(r, "tau", rw),
                                        decay_rank=None if r.get("decay_rank") is None else _int(r, "decay_rank", rw))
                if not right.tau > 0:
                    raise ConfigError(f"{rw}: 'tau' must be above 0, got {right.tau}")
                mixer = ParallelMixer(left=left, right=right)
            else:
                raise ConfigError(f"{lw}: mixer type {kind!r} is not known; known: 'attention', 'delta', 'parallel'")
            layers.append(TigutarLayer(kind, mixer, _feed_forward(l.get("mlp"), lw + ".mlp")))
        return cls(vocab=_int(d, "vocab", where), width=_int(d, "width", where),
                   norm_eps=_num(_obj(d, "norm", where), "eps", where + ": norm"), residual_mult=_num(d, "residual_mult", where),
                   layers=tuple(layers))

    def with_checkpoint_sizes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "TigutarConfig":
        """The sizes that only the checkpoint's tensor shapes give: the inner width of every right mixer's decay
        projection (rows of '<layer>.mix.right.a1')."""
        layers = []
        for i, l in enumerate(self.layers):
            if l.type == "parallel" and l.mixer.right.decay_rank is None:
                shape = shapes.get(f"l{i}.mix.right.a1")
                if shape is not None and len(shape) == 2:
                    l = replace(l, mixer=replace(l.mixer, right=replace(l.mixer.right, decay_rank=int(shape[0]))))
            layers.append(l)
        return replace(self, layers=tuple(layers))


def _attention(m: Mapping[str, Any], w: str) -> Attention:
    rot_in, mask = _opt_obj(m, "rot", w), _opt_obj(m, "mask", w)
    rot = None
    if rot_in is not None:
        rot = Rotary(base=_num(rot_in, "base", w + ".rot"), dims=_int(rot_in, "dims", w + ".rot", 0))
        if rot.dims % 2 or rot.base <= 0.0:
            raise ConfigError(f"{w}.rot: 'dims' must be even and 'base' above 0")
        if rot.dims == 0:
            rot = None
    a = Attention(heads=_int(m, "heads", w), kv_heads=_int(m, "kv_heads", w), dim=_int(m, "dim", w), vdim=_int(m, "vdim", w),
                  scale=_num(m, "scale", w), rot=rot, window=None if mask is None else _int(mask, "size", w + ".mask"),
                  kv_from=None if m.get("kv_from") is None else _int(m, "kv_from", w, 0))
    if a.heads % a.kv_heads:
        raise ConfigError(f"{w}: {a.heads} heads are no multiple of {a.kv_heads} kv_heads")
    if rot is not None and rot.dims > a.dim:
        raise ConfigError(f"{w}.rot: {rot.dims} rotated dimensions exceed the head's {a.dim}")
    return a


def _check_shared(a: Attention, before: list, w: str) -> None:
    """A layer on an earlier layer's keys and values: that one must have them, of the same heads and rotation, and keep what
    this one sees."""
    j = a.kv_from
    if j >= len(before) or before[j].type != "attention" or before[j].mixer.kv_from is not None:
        raise ConfigError(f"{w}: 'kv_from' {j} is not an earlier attention layer with keys and values of its own")
    o = before[j].mixer
    if (a.kv_heads, a.dim, a.vdim, a.rot) != (o.kv_heads, o.dim, o.vdim, o.rot):
        raise ConfigError(f"{w}: layer {j}, named by 'kv_from', has other key/value heads or another rotation")
    if o.window is not None and (a.window is None or a.window > o.window):
        raise ConfigError(f"{w}: layer {j}, named by 'kv_from', keeps a window of {o.window} positions only")


def _feed_forward(mlp_in: Any, w: str) -> Optional[FeedForward]:
    if mlp_in is None:
        return None
    if not isinstance(mlp_in, Mapping):
        raise ConfigError(f"{w} must be an object or null")
    kind = mlp_in.get("kind")
    if kind == "dense":
        return FeedForward("dense", ff=_int(mlp_in, "ff", w))
    if kind != "moe":
        raise ConfigError(f"{w}: kind {kind!r} is not known; known: 'dense', 'moe'")
    r, x = _obj(mlp_in, "router", w), _obj(mlp_in, "expert", w)
    e = FeedForward("moe", ff=_int(x, "ff", w + ".expert"), experts=_int(r, "experts", w + ".router"), top=_int(r, "top", w + ".router"),
                    limit=_num(x, "limit", w + ".expert"))
    if e.top > e.experts:
        raise ConfigError(f"{w}.router: top {e.top} exceeds experts {e.experts}")
    if not e.limit > 0:
        raise ConfigError(f"{w}.expert: 'limit' must be above 0, got {e.limit}")
    return e
