"""Duzinex as a plan of parts.

A decoder whose layers are listed one by one in the configuration.  Every layer is pre-norm (block ``pre_norm``): x <- x +
mixer(shift(norm1(x))), then, if it has a feed-forward, x <- x + ff(norm2(x)).  The norms, and the model's last one, are
dynamic tanh (``dynamic_tanh``: tanh(alpha v) * w + b, no statistics); what a mixer reads goes through a token shift
(``token_shift``: each row mixed with the row before it, the last row being state of the sequence).  Three mixers:

* ``attention``: differential attention (``gqa_attention`` with ``differential``): queries and keys of two maps per head
  over one set of values, rotation of neighbouring pairs, a window beside the first ``keep_first`` tokens, capped scores,
  biases on all four projections;
* ``retention``: linear attention with a fixed decay per head (``retention``);
* ``mingru``: a gated recurrence whose gates read the current token only (``min_gru``).

The feed-forward is one product in, the normed powers of its row (``dense_unit`` with ``activation: poly_norm``), one
product out.  The head is the embedding's table, without the embedding's scale.

``loop``: a stretch of layers runs several times with the same weights; every pass has cache lines of its own, and every
pass but the first begins with a connector (``stream_sum``): x <- x + x0, x0 being the embedding's rows.

Tensor names: ``embed``, ``final.norm[.b|.alpha]``, and per layer i ``l<i>.norm1|norm2[.b|.alpha]``, ``l<i>.shift``,
``l<i>.mix.q|k|v|o[.b]``, ``.lq1|lk1|lq2|lk2`` (attention), ``l<i>.mix.q|k|v|g|o`` (retention), ``l<i>.mix.z|x[.b]``,
``.g``, ``.o`` (mingru), ``l<i>.mlp.up|down|act``.
"""
from __future__ import annotations

from ..config.duzinex import ARCHITECTURE, DuzinexConfig
from ..config.plan import LayerSpec, ModelPlan, PartSpec, RunSpec
from ..config.registry import Architecture, register_architecture


def _dyt(width: int, name: str) -> PartSpec:
    return PartSpec("dynamic_tanh", {"width": width}, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})


def _mixer(cfg: DuzinexConfig, index: int) -> PartSpec:
    d = cfg.hidden_size
    layer = cfg.layers[index]
    m = layer.mixer
    p = f"l{index}.mix."
    if layer.type == "attention":
        position = None
        if m.rot_dims:
            position = {"kind": "rotary", "rotary_dim": m.rot_dims, "theta": m.rot_base, "pairing": "interleaved"}
        return PartSpec(
            "gqa_attention",
            {"hidden_size": d, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
             "bias": True, "output_bias": True, "qk_norm": "none", "position": position, "softmax_scale": m.scale,
             "window": m.window, "keep_first": m.keep_first, "softcap": m.softcap,
             "differential": {"diff": m.diff, "eps": cfg.norm_eps}},
            {"q_proj": p + "q", "k_proj": p + "k", "v_proj": p + "v", "o_proj": p + "o", "q_bias": p + "q.b", "k_bias": p + "k.b",
             "v_bias": p + "v.b", "o_bias": p + "o.b", "lambda_q1": p + "lq1", "lambda_k1": p + "lk1", "lambda_q2": p + "lq2",
             "lambda_k2": p + "lk2"})
    if layer.type == "retention":
        return PartSpec(
            "retention",
            {"hidden_size": d, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "decay": m.decay,
             "norm_eps": cfg.norm_eps},
            {"q_proj": p + "q", "k_proj": p + "k", "v_proj": p + "v", "gate_proj": p + "g", "o_proj": p + "o"})
    return PartSpec(
        "min_gru", {"hidden_size": d, "width": m.width},
        {"z_proj": p + "z", "z_bias": p + "z.b", "x_proj": p + "x", "x_bias": p + "x.b", "gate_proj": p + "g", "o_proj": p + "o"})


def duzinex_plan(cfg: DuzinexConfig) -> ModelPlan:
    d = cfg.hidden_size
    layers = []
    for index, layer in enumerate(cfg.layers):
        p = f"l{index}."
        feed_forward = feed_forward_norm = None
        if layer.ff is not None:
            feed_forward = PartSpec(
                "dense_unit", {"hidden_size": d, "width": layer.ff, "activation": "poly_norm", "norm_eps": cfg.norm_eps},
                {"w_up": p + "mlp.up", "w_down": p + "mlp.down", "coefficients": p + "mlp.act"})
            feed_forward_norm = _dyt(d, p + "norm2")
        layers.append(LayerSpec(block="pre_norm", mixer=_mixer(cfg, index), feed_forward=feed_forward,
                                mixer_norm=_dyt(d, p + "norm1"), feed_forward_norm=feed_forward_norm,
                                mixer_input=PartSpec("token_shift", {"width": d}, {"share": p + "shift"})))
    # the run order: layers before the loop once, the loop's layers ``times`` times (a cache line per run: every pass has
    # keys, values and states of its own), the rest once; the embedding's rows come back in front of every pass but the first
    count = len(cfg.layers)
    loop = cfg.loop
    order: list[tuple[int, int | None]] = []
    if loop is None:
        order = [(i, None) for i in range(count)]
    else:
        order += [(i, None) for i in range(loop.start)]
        for t in range(loop.times):
            order += [(i, t if t and i == loop.start else None) for i in range(loop.start, loop.stop)]
        order += [(i, None) for i in range(loop.stop, count)]
    runs = tuple(RunSpec(layer=i, cache_line=line, writes_cache=True, connector=(0, opens) if opens is not None else None)
                 for line, (i, opens) in enumerate(order))
    connectors = (PartSpec("stream_sum", {"width": d}, {}),) if loop is not None and loop.times > 1 else ()
    plan = ModelPlan(
        architecture=ARCHITECTURE,
        hidden_size=d,
        vocab_size=cfg.vocab_size,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "width": d, "scale": cfg.embedding_scale},
                           {"weight": "embed"}),
        layers=tuple(layers),
        run_order=runs,
        final_norm=_dyt(d, "final.norm"),
        head=PartSpec("vocab_head", {"vocab_size": cfg.vocab_size, "width": d}, {"weight": "embed"}),
        eos_token_id=cfg.eos_token_id,
        connectors=connectors,
    )
    plan.check()
    return plan


register_architecture(Architecture(
    name=ARCHITECTURE,
    config_from_dict=DuzinexConfig.from_dict,
    plan=duzinex_plan,
    model_type_prefixes=("duzinex",),
), replace=True)
