"""The Duzinex design without a GPU: configuration, plan, tensor names, cache needs and pages, and the plain implementation
against restatements written out element by element."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_duzinex as pd
from duzinex_configs import ALL, CONFIG_A, CONFIG_B, CONFIG_E
from fieldrun_b200.cache import CacheNeed, SequenceCache
from fieldrun_b200.config import ConfigError, DuzinexConfig
from fieldrun_b200.config.registry import architecture_for
from fieldrun_b200.engine.model import DecoderModel
from fieldrun_b200.models.duzinex import duzinex_plan


@pytest.mark.parametrize("name", sorted(ALL))
def test_configuration_reads_back(name):
    raw = ALL[name][0]
    cfg = DuzinexConfig.from_dict(raw)
    assert DuzinexConfig.from_dict(cfg.to_json_dict()) == cfg
    assert cfg.vocab_size == raw["vocab"] and cfg.hidden_size == raw["width"] and len(cfg.layers) == len(raw["layers"])
    assert architecture_for(raw).name == "Duzinex"


def test_absent_keys_switch_their_mechanism_off():
    cfg = DuzinexConfig.from_dict(CONFIG_B)
    plain = cfg.layers[1].mixer
    assert plain.window is None and plain.keep_first == 0 and plain.rot_dims == 0 and plain.softcap == 4.0
    plan = duzinex_plan(cfg)
    assert plan.layers[1].mixer.args["position"] is None and plan.layers[1].mixer.args["window"] is None
    assert plan.layers[2].feed_forward is None and plan.layers[2].feed_forward_norm is None
    assert plan.layers[3].mixer.args["softcap"] is None and not plan.connectors


@pytest.mark.parametrize("path,value,text", [
    (("layers", 0, "type"), "rwkv", "type"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "rot", "dims"), 15, "rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), 26, "rot.dims"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 0, "mixer", "diff"), "x", "diff"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"),
    (("layers", 3, "mixer", "decay"), [0.9, 0.9], "decay"),
    (("layers", 3, "mixer", "decay"), [0.9, 0.9, 1.5], "decay"),
    (("layers", 1, "mixer", "width"), 0, "width"),
    (("loop", "stop"), 5, "loop"),
    (("norm", "eps"), 0.0, "eps"),
])
def test_impossible_values_are_refused_by_key(path, value, text):
    raw = copy.deepcopy(CONFIG_A)
    node = raw
    for piece in path[:-1]:
        node = node[piece]
    node[path[-1]] = value
    with pytest.raises(ConfigError) as err:
        DuzinexConfig.from_dict(raw)
    assert text in str(err.value)


def test_run_order_gives_every_pass_lines_of_its_own_and_adds_the_embedding_before_all_but_the_first():
    plan = duzinex_plan(DuzinexConfig.from_dict(CONFIG_A))
    runs = [(r.layer, r.cache_line, r.connector is not None) for r in plan.run_order]
    assert runs == [(0, 0, False), (1, 1, False), (2, 2, False), (1, 3, True), (2, 4, False), (1, 5, True), (2, 6, False),
                    (3, 7, False)]
    once = duzinex_plan(DuzinexConfig.from_dict(CONFIG_E))
    assert [r.layer for r in once.run_order] == [0, 1, 2] and not once.connectors
    assert [(layer, again) for layer, again in pd.run_order(CONFIG_A)] == [(layer, again) for layer, _, again in runs]


def test_plan_names_every_tensor_and_the_cache_needs_hold_both_states():
    cfg = DuzinexConfig.from_dict(CONFIG_A)
    model = DecoderModel(duzinex_plan(cfg), torch.float32)
    assert model.head_is_tied and model.replayable
    shapes = {need.name: tuple(need.shape) for need in model.tensor_needs()}
    assert shapes["l0.mix.q"] == (4 * 2 * 24, 96) and shapes["l0.mix.k"] == (2 * 2 * 24, 96) and shapes["l0.mix.v"] == (2 * 40, 96)
    assert shapes["l0.mix.q.b"] == (192,) and shapes["l0.mix.o"] == (96, 160) and shapes["l0.mix.o.b"] == (96,)
    assert shapes["l0.mix.lq1"] == shapes["l0.mix.lk2"] == (24,) and shapes["l0.shift"] == (96,) and shapes["l0.norm1.alpha"] == ()
    assert shapes["l1.mix.z"] == (72, 96) and shapes["l1.mix.x.b"] == (72,) and "l1.mix.g.b" not in shapes
    assert shapes["l3.mix.k"] == (60, 96) and shapes["l3.mix.g"] == (108, 96) and shapes["l0.mlp.act"] == (4,)
    assert "l2.norm2" not in shapes and "l2.mlp.up" not in shapes and "head" not in shapes and shapes["embed"] == (131, 96)
    needs = model.cache_needs()
    first = needs[0]
    assert (first.kv_heads, first.head_dim, first.value_heads, first.value_dim, first.window, first.keep_first) == (4, 24, 2, 40, 33, 3)
    assert first.state_shape == (2, 96)                                       # the token shift alone
    assert needs[1].state_shape == (2, 72 + 96) and needs[1].kv_heads == 0    # the recurrence, then the shift
    assert needs[7].state_shape == (2, 3 * 20 * 36 + 96)
    assert needs[2] == needs[4] == needs[6] and needs[2].keep_first == 75


def test_a_line_keeps_the_pages_of_the_first_tokens_and_gives_back_those_in_between():
    need = CacheNeed(kv_heads=2, head_dim=8, window=70, value_dim=4, value_heads=1, keep_first=65)
    plain = CacheNeed(kv_heads=2, head_dim=8, window=70, value_dim=4, value_heads=1)
    cache = SequenceCache([need, plain], max_tokens=1024, num_slots=3, dtype=torch.float32, device="cpu")
    line = cache.line(0)
    assert line.keys.shape == (16, 2, 64, 8) and line.values.shape == (16, 1, 4, 64)
    kept, others = cache.groups
    slot = cache.alloc()
    for n in (100, 60, 1, 1, 300, 1):
        cache.begin_step([slot], [n])
        cache.end_step([slot], [n])
        cache.check()
        length = cache.length(slot)
        first = max(0, length - 70 + 1) // 64
        held = [i for i in range(16) if kept.table[slot, i] >= 0]
        assert held == sorted({i for i in range((length + 63) // 64) if i >= first or i < 2})
        assert [i for i in range(16) if others.table[slot, i] >= 0] == [i for i in range((length + 63) // 64) if i >= first]
    other = cache.alloc()                          # a short sequence that ends before its first tokens fill their pages
    cache.begin_step([other], [10])
    cache.end_step([other], [10])
    cache.free(other)
    cache.check()
    cache.free(slot)
    cache.check()
    assert kept.pool.num_held == others.pool.num_held == 0


# ------------------------------------------------------------------------------------------- the plain implementation

def test_rotation_pairs_neighbours():
    rng = np.random.default_rng(0)
    v = rng.normal(size=(3, 2, 7))
    out = pd.rotate_neighbours(v, [0, 5, 90], 6, 40.0)
    for t, p in enumerate([0, 5, 90]):
        for h in range(2):
            for i in range(3):
                a = p * 40.0 ** (-2 * i / 6)
                x, y = v[t, h, 2 * i], v[t, h, 2 * i + 1]
                assert out[t, h, 2 * i] == pytest.approx(x * math.cos(a) - y * math.sin(a))
                assert out[t, h, 2 * i + 1] == pytest.approx(y * math.cos(a) + x * math.sin(a))
            assert out[t, h, 6] == v[t, h, 6]


def test_window_with_first_tokens_kept():
    assert pd.visible(9, 3, 2).tolist() == [0, 1, 7, 8, 9]
    assert pd.visible(3, 3, 2).tolist() == [0, 1, 2, 3] and pd.visible(1, 3, 5).tolist() == [0, 1]
    assert pd.visible(4, 2, 0).tolist() == [3, 4] and pd.visible(4, None, 0).tolist() == [0, 1, 2, 3, 4]
    rng = np.random.default_rng(1)
    q, k, v = rng.normal(size=(8, 4, 5)), rng.normal(size=(8, 2, 5)), rng.normal(size=(8, 2, 3))
    out = pd.map_attention(q, k, v, scale=0.7, window=3, keep_first=1, softcap=2.0)
    for i in range(8):
        for h in range(4):
            seen = [j for j in range(i + 1) if i - j < 3 or j < 1]
            s = [2.0 * math.tanh(0.7 * float(q[i, h] @ k[j, h // 2]) / 2.0) for j in seen]
            p = np.exp(s) / np.exp(s).sum()
            assert np.allclose(out[i, h], sum(w * v[j, h // 2] for w, j in zip(p, seen)))


def test_retention_and_the_gated_recurrence_written_out():
    rng = np.random.default_rng(2)
    q, k, v = rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 4))
    decay = [0.9, 0.4]
    out = pd.retention(q, k, v, decay)
    for t in range(6):
        for h in range(2):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert np.allclose(out[t, h], want)
    z, u = rng.uniform(size=(5, 3)), rng.normal(size=(5, 3))
    got = pd.min_gru(z, u)
    for c in range(3):
        s = 0.0
        for t in range(5):
            cand = u[t, c] + 0.5 if u[t, c] >= 0 else 1 / (1 + math.exp(-u[t, c]))
            s = (1 - z[t, c]) * s + z[t, c] * cand
            assert got[t, c] == pytest.approx(s)


def test_normed_powers_difference_of_maps_and_shift():
    z = np.array([[1.0, -2.0, 3.0]])
    n = [z / math.sqrt(14 / 3 + 1e-3), z ** 2 / math.sqrt(98 / 3 + 1e-3), z ** 3 / math.sqrt(794 / 3 + 1e-3)]
    assert np.allclose(pd.poly_norm(z, [2.0, -1.0, 0.5, 0.25], 1e-3), 2 * n[0] - n[1] + 0.5 * n[2] + 0.25)
    assert pd.lambda_of(np.array([1.0, 2.0]), np.array([0.5, 0.1]), np.array([0.3]), np.array([2.0]), 0.4) == \
        pytest.approx(math.exp(0.7) - math.exp(0.6) + 0.4)
    o = np.array([3.0, -4.0]) - 0.5 * np.array([1.0, 2.0])
    assert np.allclose(pd.difference_of_maps(np.array([3.0, -4.0]), np.array([1.0, 2.0]), 0.5, 0.2, 1e-4),
                       o / math.sqrt((o @ o) / 2 + 1e-4) * 0.8)
    h = np.array([[2.0, 4.0], [6.0, 8.0]])
    assert pd.token_shift(h, np.array([0.25, 1.0])).tolist() == [[1.5, 0.0], [5.0, 4.0]]


def test_whole_model_is_causal_and_the_embedding_comes_back():
    from duzinex_configs import plain_weights, request_tokens
    config, weights = plain_weights("D")
    ids = request_tokens("D", 12, 1)
    streams = []
    logits = pd.forward(config, weights, ids, streams)
    assert logits.shape == (12, 64) and len(streams) == 4 and np.isfinite(logits).all()
    assert np.allclose(pd.forward(config, weights, ids[:7]), logits[:7])
    once = dict(config, loop=None)
    assert not np.allclose(pd.forward(once, weights, ids), logits)
