"""Configuration of the Duzinex design, read from its own config.json keys.

The file names the design as ``"architecture": "Duzinex"`` and lists the layers one by one:

    vocab, width                       sizes of the vocabulary and of the residual stream
    embedding.scale                    factor on the embedding's rows
    norm.eps                           eps of the root-mean-square divisions in the mixers and the feed-forward
    loop {start, stop, times}          layers start .. stop-1 run ``times`` times in a row (absent: every layer once)
    layers[i].type                     "attention" | "retention" | "mingru"
    layers[i].mixer                    the mixer's sizes and constants (below)
    layers[i].mlp                      {"kind": "dense", "ff"} or null

    attention: heads, kv_heads, dim, vdim, diff, scale, softcap, mask {size, keep_first}, rot {base, dims}
    retention: heads, dim, vdim, decay (a number per head)
    mingru:    width

Everything that can differ between two models of the design is read here; an absent ``mask``, ``rot`` or ``softcap``
switches its mechanism off.  A key the design does not have is a warning on stderr.
"""
from __future__ import annotations

import sys
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .base import ConfigError, KeyReader, ModelConfig

ARCHITECTURE = "Duzinex"


def _unknown(raw: Mapping[str, Any], allowed: set[str], where: str) -> None:
    extra = sorted(set(raw) - allowed)
    if extra:
        print(f"{where}: warning: keys this design does not have are ignored: {', '.join(extra)}", file=sys.stderr)


def _object(raw: Any, where: str) -> Mapping[str, Any]:
    if not isinstance(raw, Mapping):
        raise ConfigError(f"{where} must be an object")
    return raw


@dataclass(frozen=True)
class DuzinexAttention:
    heads: int
    kv_heads: int
    dim: int                              # of one map of a head; queries and keys have two
    vdim: int
    diff: float
    scale: float
    softcap: Optional[float]
    window: Optional[int]                 # None: every earlier key is seen
    keep_first: int
    rot_dims: int                         # 0: no rotation
    rot_base: float

    def to_json(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "diff": self.diff,
                               "scale": self.scale}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.window is not None:
            out["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return out


@dataclass(frozen=True)
class DuzinexRetention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    def to_json(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class DuzinexMinGru:
    width: int

    def to_json(self) -> dict[str, Any]:
        return {"width": self.width}


@dataclass(frozen=True)
class DuzinexLayer:
    type: str
    mixer: Any                            # DuzinexAttention | DuzinexRetention | DuzinexMinGru
    ff: Optional[int]                     # None: no feed-forward

    def to_json(self) -> dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}


@dataclass(frozen=True)
class DuzinexLoop:
    start: int
    stop: int
    times: int

    def to_json(self) -> dict[str, Any]:
        return {"start": self.start, "stop": self.stop, "times": self.times}


def _attention(raw: Mapping[str, Any], where: str) -> DuzinexAttention:
    _unknown(raw, {"heads", "kv_heads", "dim", "vdim", "diff", "scale", "softcap", "mask", "rot"}, where)
    r = KeyReader(raw, where)
    heads = r.integer("heads", minimum=1)
    kv_heads = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    dim = r.integer("dim", minimum=1)
    window, keep_first = None, 0
    if raw.get("mask") is not None:
        _unknown(_object(raw["mask"], where + ".mask"), {"size", "keep_first"}, where + ".mask")
        window = r.integer("mask.size", minimum=1)
        keep_first = r.integer("mask.keep_first", default=0, minimum=0)
    rot_dims, rot_base = 0, 10000.0
    if raw.get("rot") is not None:
        _unknown(_object(raw["rot"], where + ".rot"), {"base", "dims"}, where + ".rot")
        rot_dims = r.integer("rot.dims", default=dim, minimum=0)
        rot_base = r.real("rot.base", positive=True)
        if rot_dims % 2 or rot_dims > dim:
            raise ConfigError(f"{where}: rot.dims is {rot_dims}: it must be even and at most dim = {dim}")
    return DuzinexAttention(
        heads, kv_heads, dim, r.integer("vdim", default=dim, minimum=1), r.real("diff"),
        r.real("scale", default=float(dim) ** -0.5, positive=True),
        r.real("softcap", positive=True) if raw.get("softcap") is not None else None, window, keep_first, rot_dims, rot_base)


def _retention(raw: Mapping[str, Any], where: str) -> DuzinexRetention:
    _unknown(raw, {"heads", "dim", "vdim", "decay"}, where)
    r = KeyReader(raw, where)
    heads, dim = r.integer("heads", minimum=1), r.integer("dim", minimum=1)
    listed = raw.get("decay")
    if not isinstance(listed, (list, tuple)) or not all(isinstance(v, (int, float)) and not isinstance(v, bool) for v in listed):
        raise ConfigError(f"{where}: key 'decay' must be a list of numbers, found {listed!r}")
    if len(listed) != heads:
        raise ConfigError(f"{where}: key 'decay' has {len(listed)} numbers for {heads} heads")
    if not all(0.0 <= float(v) <= 1.0 for v in listed):
        raise ConfigError(f"{where}: key 'decay' must hold numbers between 0 and 1, found {listed!r}")
    return DuzinexRetention(heads, dim, r.integer("vdim", default=dim, minimum=1), tuple(float(v) for v in listed))


def _mingru(raw: Mapping[str, Any], where: str) -> DuzinexMinGru:
    _unknown(raw, {"width"}, where)
    return DuzinexMinGru(KeyReader(raw, where).integer("width", minimum=1))


_MIXERS = {"attention": _attention, "retention": _retention, "mingru": _mingru}


@dataclass(frozen=True)
class DuzinexConfig(ModelConfig):
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    layers: tuple[DuzinexLayer, ...] = ()
    loop: Optional[DuzinexLoop] = None

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str = "config.json") -> "DuzinexConfig":
        _unknown(raw, {"architecture", "architectures", "model_type", "vocab", "width", "embedding", "norm", "layers", "loop",
                       "eos_token_id"}, where)
        r = KeyReader(raw, where)
        for name, allowed in (("norm", {"eps"}), ("embedding", {"scale"})):
            if isinstance(raw.get(name), Mapping):
                _unknown(raw[name], allowed, f"{where}: {name}")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError(f"{where}: key 'layers' must be a list of at least one layer")
        layers: list[DuzinexLayer] = []
        for index, entry in enumerate(listed):
            at = f"{where}: layers[{index}]"
            entry = _object(entry, at)
            _unknown(entry, {"type", "mixer", "mlp"}, at)
            kind = entry.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{at}.type is {kind!r}: this design has {', '.join(sorted(_MIXERS))}")
            mixer = _MIXERS[kind](_object(entry.get("mixer"), at + ".mixer"), at + ".mixer")
            ff = None
            if entry.get("mlp") is not None:
                m = _object(entry["mlp"], at + ".mlp")
                _unknown(m, {"kind", "ff"}, at + ".mlp")
                if m.get("kind", "dense") != "dense":
                    raise ConfigError(f"{at}.mlp.kind is {m.get('kind')!r}: this design has 'dense'")
                ff = KeyReader(m, at + ".mlp").integer("ff", minimum=1)
            layers.append(DuzinexLayer(kind, mixer, ff))
        loop = None
        if raw.get("loop") is not None:
            lp = _object(raw["loop"], f"{where}: loop")
            _unknown(lp, {"start", "stop", "times"}, f"{where}: loop")
            k = KeyReader(lp, f"{where}: loop")
            loop = DuzinexLoop(k.integer("start", default=0, minimum=0), k.integer("stop", default=len(layers), minimum=0),
                               k.integer("times", default=1, minimum=1))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"{where}: loop runs layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        return cls(
            architecture=ARCHITECTURE,
            vocab_size=r.integer("vocab", minimum=1),
            hidden_size=r.integer("width", minimum=1),
            num_hidden_layers=len(layers),
            eos_token_id=tuple(t for t in r.integer_list("eos_token_id", default=()) if t >= 0),
            norm_eps=r.real("norm.eps", positive=True),
            embedding_scale=r.real("embedding.scale", default=1.0),
            layers=tuple(layers),
            loop=loop,
        )

    def to_json_dict(self) -> dict[str, Any]:
        """The config.json that reads back to this configuration."""
        out: dict[str, Any] = {
            "architecture": ARCHITECTURE,
            "vocab": self.vocab_size,
            "width": self.hidden_size,
            "embedding": {"scale": self.embedding_scale},
            "norm": {"eps": self.norm_eps},
            "layers": [layer.to_json() for layer in self.layers],
        }
        if self.loop is not None:
            out["loop"] = self.loop.to_json()
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
