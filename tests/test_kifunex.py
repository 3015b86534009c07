"""The Kifunex design without a GPU: configuration, plan, tensor names, cache needs, rotation frequencies, and the plain
implementation against restatements written out element by element."""
import copy

import numpy as np
import pytest
import torch

import plain_kifunex as pk
from fieldrun_b200.config import ConfigError, ModelPlan
from fieldrun_b200.config.kifunex import KifunexConfig
from fieldrun_b200.config.registry import architecture_for
from fieldrun_b200.engine.model import DecoderModel
from fieldrun_b200.models.kifunex import kifunex_plan
from fieldrun_b200.parts.position import Rotary
from kifunex_configs import ALL, CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, plain_weights, request_tokens


@pytest.mark.parametrize("name", sorted(ALL))
def test_configuration_reads_back(name):
    raw = ALL[name][0]
    cfg = KifunexConfig.from_dict(raw)
    assert KifunexConfig.from_dict(cfg.to_json_dict()) == cfg
    assert cfg.vocab_size == raw["vocab"] and cfg.hidden_size == raw["width"] and len(cfg.layers) == len(raw["layers"])
    assert cfg.streams == raw["streams"] and architecture_for(raw).name == "Kifunex"


def test_absent_keys_switch_their_mechanism_off():
    cfg = KifunexConfig.from_dict(CONFIG_B)
    assert cfg.logit_softcap is None and cfg.logit_scale == 1.7
    assert cfg.layers[0].mixer.rot_dims == 0 and cfg.layers[3].mixer.window is None and cfg.layers[3].mlp is None
    assert cfg.layers[2].mlp.shared_ff == 0 and cfg.layers[2].mlp.scale == 1.0
    plan = kifunex_plan(cfg)
    assert plan.layers[0].mixer.args["position"] is None and plan.layers[2].mixer.args["window"] is None
    assert plan.layers[2].feed_forward is None and plan.head.args["softcap"] is None
    assert "shared_expert" not in plan.layers[1].feed_forward.args
    assert KifunexConfig.from_dict(CONFIG_A).layers[2].mixer.blend is None
    bare = {k: v for k, v in CONFIG_D.items() if k not in ("logit_softcap", "norm", "streams")}
    cfg = KifunexConfig.from_dict(bare)
    assert cfg.logit_scale == 1.0 and cfg.logit_softcap is None and cfg.streams == 1
    assert KifunexConfig.from_dict(cfg.to_json_dict()) == cfg


@pytest.mark.parametrize("path,value,text", [
    (("layers", 0, "type"), "mamba", "type"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "vdim"), 25, "vdim"),
    (("layers", 0, "mixer", "rot", "dims"), 15, "rot.dims"),
    (("layers", 0, "mixer", "rot", "scaling", "low"), 5.0, "low"),
    (("layers", 0, "mixer", "rot", "scaling", "original"), 0, "original"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mlp", "router", "top"), 8, "top"),
    (("layers", 0, "mlp", "kind"), "dense", "kind"),
    (("layers", 3, "weights_of"), 6, "weights_of"),
    (("layers", 3, "weights_of"), 3, "weights_of"),
    (("layers", 3, "weights_of"), 2, "differs"),
    (("streams",), 0, "streams"),
    (("logit_softcap",), 0.0, "logit_softcap"),
])
def test_impossible_values_are_refused_by_key(path, value, text):
    raw = copy.deepcopy(CONFIG_A)
    node = raw
    for piece in path[:-1]:
        node = node[piece]
    node[path[-1]] = value
    with pytest.raises(ConfigError) as err:
        KifunexConfig.from_dict(raw)
    assert text in str(err.value)


def test_layers_that_run_each_others_tensors_in_a_circle_are_refused():
    raw = copy.deepcopy(CONFIG_A)
    raw["layers"][1]["weights_of"] = 3
    with pytest.raises(ConfigError, match="weights_of"):
        KifunexConfig.from_dict(raw)


def test_plan_names_the_owners_tensors_and_gives_every_run_a_cache_line():
    model = DecoderModel(kifunex_plan(KifunexConfig.from_dict(CONFIG_A)), torch.float32)
    names = [need.name for need in model.tensor_needs()]
    assert len(names) == len(set(names))
    for expected in ("embed", "head", "final.norm", "final.norm.b", "final.norm.alpha", "l0.norm1", "l0.norm2.alpha", "l0.hc1.in",
                     "l0.hc2.mix", "l1.hc1.out", "l0.mix.q", "l0.mix.k", "l0.mix.o", "l0.mlp.router", "l0.mlp.correction",
                     "l0.mlp.e6.down", "l0.mlp.shared.gate", "l2.mlp.e4.up"):
        assert expected in names, expected
    assert not any(n.startswith(("l3.", "l4.", "l5.")) or n.endswith("mix.v") for n in names)
    assert "l1.hc2.in" not in names and "l1.norm2" not in names and "l2.mlp.shared.gate" not in names
    shapes = {need.name: tuple(need.shape) for need in model.tensor_needs()}
    assert shapes["l0.hc1.mix"] == (3, 3) and shapes["l0.hc2.out"] == (3,) and shapes["l0.norm1.alpha"] == ()
    assert [(run.layer, run.cache_line) for run in model.plan.run_order] == [(0, 0), (1, 1), (2, 2), (1, 3), (0, 4), (2, 5)]
    needs = model.cache_needs()
    assert [need.window for need in needs] == [33, 70, None, 70, 33, None] and all(not need.state_shape for need in needs)
    assert set(model.kernel_groups()) >= {"common", "experts", "copies"} and model.replayable
    # an owner that comes later, and owners through another layer that has no tensors either
    late = copy.deepcopy(CONFIG_B)
    late["layers"][4]["weights_of"] = 2
    late["layers"].append(dict(late["layers"][4], weights_of=4))
    plan = kifunex_plan(KifunexConfig.from_dict(late))
    assert [run.layer for run in plan.run_order] == [0, 2, 1, 2, 1, 1]


def test_tensor_core_sizes_ask_for_their_kernels():
    model = DecoderModel(kifunex_plan(KifunexConfig.from_dict(CONFIG_C)), torch.bfloat16)
    assert set(model.kernel_groups()) == {"common", "copies", "streams", "attention", "experts", "products"}


def test_a_plan_with_copies_needs_connections_everywhere():
    plan = kifunex_plan(KifunexConfig.from_dict(CONFIG_D))
    fields = {f: getattr(plan, f) for f in plan.__dataclass_fields__}
    with pytest.raises(ValueError, match="connections"):
        ModelPlan(**dict(fields, streams=0)).check()
    with pytest.raises(ValueError, match="single stream"):
        ModelPlan(**dict(fields, connectors=(plan.embedding,))).check()


@pytest.mark.parametrize("dims,base,blend", [
    (16, 1000.0, (8.0, 1.0, 4.0, 200.0)),            # all three ranges
    (32, 10000.0, (4.0, 1.0, 4.0, 1500.0)),
    (12, 20.0, (4.0, 1.0, 4.0, 1e6)),                # every wavelength stays
    (8, 300.0, (5.0, 1.0, 2.0, 3.0)),                # every wavelength is divided
    (2, 300.0, (5.0, 1.0, 1.0, 30.0)),               # nothing in between
    (20, 700.0, (3.0, 2.5, 2.5, 90.0)),
    (10, 50.0, None),
])
def test_rotation_frequencies(dims, base, blend):
    names = ("factor", "low", "high", "original")
    scaling = dict(zip(names, blend)) if blend else None
    want = pk.rotation_frequencies(dims, base, scaling)
    args = {"rotary_dim": dims, "theta": base, "pairing": "half"}
    got = Rotary(dict(args, frequency_blend=scaling) if blend else args)
    np.testing.assert_allclose(got.frequencies().numpy(), want, rtol=1e-12)
    cos, sin = got.tables(300, "cpu")
    np.testing.assert_allclose(cos.numpy(), np.cos(np.arange(300)[:, None] * want[None, :]), atol=1e-6)
    np.testing.assert_allclose(sin.numpy(), np.sin(np.arange(300)[:, None] * want[None, :]), atol=1e-6)
    if blend and blend == (8.0, 1.0, 4.0, 200.0):
        plain = pk.rotation_frequencies(dims, base)
        ratio = want / plain
        assert (ratio == 1.0).any() and np.isclose(ratio, 1 / 8.0).any() and ((ratio > 0.13) & (ratio < 0.99)).any()
    with pytest.raises(ValueError, match="blend"):
        Rotary(dict(args, frequency_blend={"factor": 2.0, "low": 4.0, "high": 1.0, "original": 10.0}))


# ------------------------------------------------------------------------------------------- the plain implementation

def test_mix_is_indexed_from_and_to():
    x = np.zeros((1, 2, 1))
    x[0, :, 0] = [1.0, 10.0]
    new = pk.spread_update(x, np.array([[100.0]]), np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([0.5, 0.25]))
    assert new[0, :, 0].tolist() == [1.0 + 30.0 + 50.0, 2.0 + 40.0 + 25.0]
    assert pk.gather_streams(x, np.array([2.0, 3.0]))[0, 0] == 32.0


def test_two_sublayers_in_one_step_are_the_two_steps_one_after_the_other():
    rng = np.random.default_rng(0)
    x, y1, y2 = rng.normal(size=(4, 3, 5)), rng.normal(size=(4, 5)), rng.normal(size=(4, 5))
    m1, m2, o1, o2 = rng.normal(size=(3, 3)), rng.normal(size=(3, 3)), rng.normal(size=3), rng.normal(size=3)
    after = pk.spread_update(pk.spread_update(x, y1, m1, o1), y2, m2, o2)
    both = pk.spread_update(x, y1, m1 @ m2, o1 @ m2) + np.einsum("td,s->tsd", y2, o2)
    assert np.allclose(after, both)


def test_window_counts_the_token_itself():
    rng = np.random.default_rng(1)
    q, k, v = rng.normal(size=(9, 4, 6)), rng.normal(size=(9, 2, 6)), rng.normal(size=(9, 2, 6))
    out = pk.windowed_attention(q, k, v, scale=0.7, window=4)
    for i in range(9):
        for h in range(4):
            seen = [j for j in range(9) if 0 <= i - j < 4]
            e = np.array([np.exp(0.7 * (q[i, h] @ k[j, h // 2])) for j in seen])
            assert np.allclose(out[i, h], sum(w * v[j, h // 2] for w, j in zip(e / e.sum(), seen)))
    assert np.allclose(pk.windowed_attention(q, k, v, scale=0.7, window=1)[5, 3], v[5, 1])


def test_values_are_the_keys_before_their_rotation():
    rng = np.random.default_rng(2)
    h, width = rng.normal(size=(6, 8)), 8
    t = {"q": rng.normal(size=(4, width)), "k": rng.normal(size=(4, width)), "o": rng.normal(size=(width, 4))}
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 0.5, "mask": {"size": 1}, "rot": {"dims": 4, "base": 3.0}}
    assert np.allclose(pk.attention_mixer(h, t, "", m), h @ t["k"].T @ t["o"].T)       # one key seen: its value, not its rotation


def test_the_correction_chooses_but_does_not_weigh():
    scores = np.array([0.9, 0.2, 0.5, 0.4])
    ids, weights = pk.choose_experts(scores, np.array([-1.0, 0.0, 0.0, 0.3]), 2, 1.5)
    assert ids.tolist() == [3, 2] and np.allclose(weights, [0.6, 0.75])


def test_whole_model_runs_and_a_repeated_layer_is_a_layer_with_the_same_tensors():
    config, weights = plain_weights("A")
    ids = request_tokens("A", 12, 1)
    streams = []
    logits = pk.forward(config, weights, ids, streams=streams)
    assert logits.shape == (12, config["vocab"]) and len(streams) == 6 and np.isfinite(logits).all()
    assert np.abs(logits).max() < config["logit_softcap"]
    unrolled = copy.deepcopy(config)
    copied = dict(weights)
    for index, layer in enumerate(unrolled["layers"]):
        owner = layer.pop("weights_of", None)
        if owner is not None:
            copied.update({f"l{index}." + n.split(".", 1)[1]: v for n, v in weights.items() if n.startswith(f"l{owner}.")})
    assert np.allclose(pk.forward(unrolled, copied, ids), logits)
    # a token's logits do not depend on later tokens
    assert np.allclose(pk.forward(config, weights, ids[:7]), logits[:7])
