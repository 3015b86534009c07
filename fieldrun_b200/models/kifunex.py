"""Kifunex as a plan of parts.

A decoder whose layers are listed one by one in the configuration, on a residual stream kept as several copies.  Every layer
has two sublayers behind dynamic-tanh norms (``dynamic_tanh``: tanh(alpha v) * w + b) in block ``hyper_connections``: a
sublayer reads a weighted sum of the copies, and its output is spread over all of them while they are mixed
(``hyper_connections``).  The model's last norm reads the sum of the copies.

The mixer is grouped-query attention over a window (``gqa_attention`` with ``values_from_keys``: the values are the keys as
projected, before their rotation); the rotation is in halves on the first ``rot.dims`` entries of a head, its frequencies
blended by wavelength (``rotary`` with ``frequency_blend``).  The feed-forward is routed experts: sigmoid scores, a correction
that enters the choice only, weights not renormalized but scaled, and a shared expert that every token uses
(``routed_experts``).  The logits are scaled, then capped (``vocab_head``).

``weights_of``: a layer without tensors of its own is one more run of another layer, with a cache line of its own.

Tensor names: ``embed``, ``head``, ``final.norm[.b|.alpha]``, and per layer i that owns tensors ``l<i>.norm1|norm2[.b|.alpha]``,
``l<i>.hc1|hc2.in|out|mix``, ``l<i>.mix.q|k|o``, ``l<i>.mlp.router|correction``, ``.e<e>.gate|up|down``,
``.shared.gate|up|down``.
"""
from __future__ import annotations

from ..config.kifunex import ARCHITECTURE, KifunexAttention, KifunexConfig, KifunexExperts
from ..config.plan import LayerSpec, ModelPlan, PartSpec, RunSpec
from ..config.registry import Architecture, register_architecture


def _dyt(width: int, name: str) -> PartSpec:
    return PartSpec("dynamic_tanh", {"width": width}, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})


def _attention(cfg: KifunexConfig, m: KifunexAttention, p: str) -> PartSpec:
    position = None
    if m.rot_dims:
        position = {"kind": "rotary", "rotary_dim": m.rot_dims, "theta": m.rot_base, "pairing": "half"}
        if m.blend is not None:
            position["frequency_blend"] = m.blend.to_json()
    return PartSpec(
        "gqa_attention",
        {"hidden_size": cfg.hidden_size, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
         "values_from_keys": True, "qk_norm": "none", "position": position, "softmax_scale": m.scale, "window": m.window},
        {"q_proj": p + "q", "k_proj": p + "k", "o_proj": p + "o"})


def _experts(cfg: KifunexConfig, m: KifunexExperts, p: str) -> PartSpec:
    args = {"hidden_size": cfg.hidden_size, "num_experts": m.experts, "top_k": m.top, "expert_width": m.ff, "score": "sigmoid",
            "choice_bias": True, "renormalize": False, "routed_scale": m.scale}
    tensors = {"router": p + "router", "choice_bias": p + "correction", "w_gate": p + "e{e}.gate", "w_up": p + "e{e}.up",
               "w_down": p + "e{e}.down"}
    if m.shared_ff:
        args["shared_expert"] = {"width": m.shared_ff, "gate": False}
        tensors.update({"shared_gate": p + "shared.gate", "shared_up": p + "shared.up", "shared_down": p + "shared.down"})
    return PartSpec("routed_experts", args, tensors)


def _connections(cfg: KifunexConfig, index: int, feed_forward: bool) -> PartSpec:
    tensors = {f"{local}{q}": f"l{index}.hc{q}.{local}" for q in ((1, 2) if feed_forward else (1,)) for local in ("in", "out", "mix")}
    return PartSpec("hyper_connections", {"streams": cfg.streams, "feed_forward": feed_forward}, tensors)


def kifunex_plan(cfg: KifunexConfig) -> ModelPlan:
    d = cfg.hidden_size
    layers: list[LayerSpec] = []
    place: dict[int, int] = {}                     # layer that owns tensors -> its place among the plan's layers
    for index, layer in enumerate(cfg.layers):
        if layer.owner != index:
            continue
        p = f"l{index}."
        has_ff = layer.mlp is not None
        place[index] = len(layers)
        layers.append(LayerSpec(
            block="hyper_connections", mixer=_attention(cfg, layer.mixer, p + "mix."),
            feed_forward=_experts(cfg, layer.mlp, p + "mlp.") if has_ff else None, mixer_norm=_dyt(d, p + "norm1"),
            feed_forward_norm=_dyt(d, p + "norm2") if has_ff else None, connections=_connections(cfg, index, has_ff)))
    plan = ModelPlan(
        architecture=ARCHITECTURE,
        hidden_size=d,
        vocab_size=cfg.vocab_size,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "width": d}, {"weight": "embed"}),
        layers=tuple(layers),
        run_order=tuple(RunSpec(layer=place[layer.owner], cache_line=index) for index, layer in enumerate(cfg.layers)),
        final_norm=_dyt(d, "final.norm"),
        head=PartSpec("vocab_head", {"vocab_size": cfg.vocab_size, "width": d, "scale": cfg.logit_scale, "softcap": cfg.logit_softcap},
                      {"weight": "head"}),
        eos_token_id=cfg.eos_token_id,
        streams=cfg.streams,
    )
    plan.check()
    return plan


register_architecture(Architecture(
    name=ARCHITECTURE,
    config_from_dict=KifunexConfig.from_dict,
    plan=kifunex_plan,
    model_type_prefixes=("kifunex",),
), replace=True)
