"""Configuration of the Kifunex design, read from its own config.json keys.

The file names the design as ``"architecture": "Kifunex"`` and lists the layers one by one:

    vocab, width                       sizes of the vocabulary and of a row of the residual stream
    streams                            copies of the residual stream (hyper-connections)
    norm.eps                           belongs to the file; this design's norms have no eps
    logit_scale, logit_softcap         factor on the logits, then their cap
    layers[i].type                     "attention"
    layers[i].mixer                    heads, kv_heads, dim, vdim, scale, mask {size},
                                       rot {base, dims, scaling {factor, low, high, original}}
    layers[i].mlp                      null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale"}, "shared": {"ff"}}
    layers[i].weights_of               j: the layer has no tensors of its own and runs layer j's again

Everything that can differ between two models of the design is read here; an absent ``mask``, ``rot``, ``scaling``, ``shared``
or ``logit_softcap`` switches its mechanism off.  The values are the keys as projected, so ``vdim`` is ``dim``.  A key the
design does not have is a warning on stderr.
"""
from __future__ import annotations

import sys
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .base import ConfigError, KeyReader, ModelConfig

ARCHITECTURE = "Kifunex"


def _unknown(raw: Mapping[str, Any], allowed: set[str], where: str) -> None:
    extra = sorted(set(raw) - allowed)
    if extra:
        print(f"{where}: warning: keys this design does not have are ignored: {', '.join(extra)}", file=sys.stderr)


def _object(raw: Any, where: str) -> Mapping[str, Any]:
    if not isinstance(raw, Mapping):
        raise ConfigError(f"{where} must be an object")
    return raw


@dataclass(frozen=True)
class FrequencyBlend:
    factor: float
    low: float
    high: float
    original: float

    def to_json(self) -> dict[str, Any]:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class KifunexAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: Optional[int]                 # None: every earlier key
    rot_dims: int                         # 0: no rotation
    rot_base: float
    blend: Optional[FrequencyBlend]

    def to_json(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.blend is not None:
                out["rot"]["scaling"] = self.blend.to_json()
        return out


@dataclass(frozen=True)
class KifunexExperts:
    experts: int
    top: int
    ff: int
    scale: float = 1.0
    shared_ff: int = 0                    # 0: no shared expert

    def to_json(self) -> dict[str, Any]:
        out: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff},
                               "router": {"experts": self.experts, "top": self.top, "scale": self.scale}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class KifunexLayer:
    mixer: KifunexAttention
    mlp: Optional[KifunexExperts]
    owner: int                            # the layer whose tensors this one runs (its own index unless it runs another's)

    def to_json(self, index: int) -> dict[str, Any]:
        out: dict[str, Any] = {"type": "attention", "mixer": self.mixer.to_json(), "mlp": self.mlp.to_json() if self.mlp else None}
        if self.owner != index:
            out["weights_of"] = self.owner
        return out


def _attention(raw: Mapping[str, Any], where: str) -> KifunexAttention:
    _unknown(raw, {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"}, where)
    r = KeyReader(raw, where)
    heads = r.integer("heads", minimum=1)
    kv_heads = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    dim = r.integer("dim", minimum=1)
    vdim = r.integer("vdim", default=dim, minimum=1)
    if vdim != dim:
        raise ConfigError(f"{where}.vdim is {vdim}: the values are the keys as projected, so it is dim = {dim}")
    window = None
    if raw.get("mask") is not None:
        _unknown(_object(raw["mask"], where + ".mask"), {"size"}, where + ".mask")
        window = r.integer("mask.size", minimum=1)
    rot_dims, rot_base, blend = 0, 10000.0, None
    if raw.get("rot") is not None:
        rot = _object(raw["rot"], where + ".rot")
        _unknown(rot, {"base", "dims", "scaling"}, where + ".rot")
        rot_dims = r.integer("rot.dims", default=dim, minimum=0)
        rot_base = r.real("rot.base", positive=True)
        if rot_dims % 2 or rot_dims > dim:
            raise ConfigError(f"{where}.rot.dims is {rot_dims}: an even number up to dim = {dim}")
        if rot.get("scaling") is not None:
            at = where + ".rot.scaling"
            _unknown(_object(rot["scaling"], at), {"factor", "low", "high", "original"}, at)
            blend = FrequencyBlend(*(r.real(f"rot.scaling.{name}", positive=True) for name in ("factor", "low", "high", "original")))
            if blend.low > blend.high:
                raise ConfigError(f"{at}: low = {blend.low} is above high = {blend.high}")
    return KifunexAttention(heads, kv_heads, dim, r.real("scale", default=float(dim) ** -0.5), window, rot_dims, rot_base, blend)


def _mlp(raw: Any, where: str) -> Optional[KifunexExperts]:
    if raw is None:
        return None
    m = _object(raw, where)
    if m.get("kind", "moe") != "moe":
        raise ConfigError(f"{where}.kind is {m.get('kind')!r}: this design has 'moe'")
    _unknown(m, {"kind", "expert", "router", "shared"}, where)
    for name, allowed in (("expert", {"ff"}), ("router", {"experts", "top", "scale"}), ("shared", {"ff"})):
        if isinstance(m.get(name), Mapping):
            _unknown(m[name], allowed, f"{where}.{name}")
    k = KeyReader(m, where)
    experts, top = k.integer("router.experts", minimum=1), k.integer("router.top", minimum=1)
    if top > experts:
        raise ConfigError(f"{where}.router: top {top} of {experts} experts")
    return KifunexExperts(experts, top, k.integer("expert.ff", minimum=1), k.real("router.scale", default=1.0),
                          k.integer("shared.ff", minimum=1) if m.get("shared") is not None else 0)


def _owner(listed: list, index: int, where: str) -> int:
    """The layer whose tensors layer ``index`` runs, through any number of ``weights_of``."""
    seen = {index}
    while listed[index].get("weights_of") is not None:
        other = KeyReader(listed[index], f"{where}: layers[{index}]").integer("weights_of", minimum=0)
        if other >= len(listed) or other in seen:
            raise ConfigError(f"{where}: layers[{index}].weights_of is {other}: another layer of the {len(listed)} that has tensors")
        seen.add(other)
        index = other
    return index


@dataclass(frozen=True)
class KifunexConfig(ModelConfig):
    streams: int = 1
    norm_eps: Optional[float] = None
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    layers: tuple[KifunexLayer, ...] = ()

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str = "config.json") -> "KifunexConfig":
        _unknown(raw, {"architecture", "architectures", "model_type", "vocab", "width", "streams", "norm", "logit_scale", "logit_softcap",
                       "layers", "eos_token_id"}, where)
        r = KeyReader(raw, where)
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError(f"{where}: key 'layers' must be a list of at least one layer")
        read: list[tuple[KifunexAttention, Optional[KifunexExperts]]] = []
        for index, entry in enumerate(listed):
            at = f"{where}: layers[{index}]"
            entry = _object(entry, at)
            _unknown(entry, {"type", "mixer", "mlp", "weights_of"}, at)
            if entry.get("type") != "attention":
                raise ConfigError(f"{at}.type is {entry.get('type')!r}: this design has 'attention'")
            read.append((_attention(_object(entry.get("mixer"), at + ".mixer"), at + ".mixer"), _mlp(entry.get("mlp"), at + ".mlp")))
        layers = []
        for index, (mixer, mlp) in enumerate(read):
            owner = _owner(listed, index, where)
            if (mixer, mlp) != read[owner]:
                raise ConfigError(f"{where}: layers[{index}] runs the tensors of layers[{owner}] but its entry differs from that layer's")
            layers.append(KifunexLayer(mixer, mlp, owner))
        return cls(
            architecture=ARCHITECTURE,
            vocab_size=r.integer("vocab", minimum=1),
            hidden_size=r.integer("width", minimum=1),
            num_hidden_layers=len(layers),
            eos_token_id=tuple(t for t in r.integer_list("eos_token_id", default=()) if t >= 0),
            streams=r.integer("streams", default=1, minimum=1),
            norm_eps=r.real("norm.eps") if r.present("norm.eps") else None,
            logit_scale=r.real("logit_scale", default=1.0),
            logit_softcap=r.real("logit_softcap", positive=True) if raw.get("logit_softcap") is not None else None,
            layers=tuple(layers),
        )

    def to_json_dict(self) -> dict[str, Any]:
        """The config.json that reads back to this configuration."""
        out: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                               "streams": self.streams, "logit_scale": self.logit_scale,
                               "layers": [layer.to_json(index) for index, layer in enumerate(self.layers)]}
        if self.norm_eps is not None:
            out["norm"] = {"eps": self.norm_eps}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
