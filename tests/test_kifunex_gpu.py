"""The Kifunex design as whole models in the engine against the plain implementation of ``plain_kifunex``: through the step
function, the cache, recorded decode steps, the generation loop, the trace runner and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import fieldrun_b200 as fr
import plain_kifunex as pk
from kifunex_configs import ALL, model_folder, plain_weights, request_tokens

pytestmark = pytest.mark.gpu

# per row, against the spread of the plain logits; bfloat16 runs compare with the plain model made to use the experts the engine
# used (the choice is not continuous)
MODEL_TOL = {"float32": 3e-5, "bfloat16": 4e-2}
# the engine may pick other experts than the plain model only where the choice is this close
ROUTE_MARGIN = 2e-2
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])

_LOADED = {}


def loaded(name, dtype, record_steps=True):
    key = (name, dtype, record_steps)
    if key not in _LOADED:
        lm = fr.load(model_folder(name), dtype=dtype, max_tokens=4096, num_slots=8)
        lm.engine.record_steps = record_steps and lm.model.replayable
        _LOADED[key] = lm
    return _LOADED[key]


_PLAIN = {}


def plain_run(name, length, seed):
    """(logits, the experts of every layer that has some) of the plain model."""
    key = (name, length, seed)
    if key not in _PLAIN:
        config, weights = plain_weights(name)
        routes = []
        _PLAIN[key] = (pk.forward(config, weights, request_tokens(name, length, seed), routes=routes), routes)
    return _PLAIN[key]


def first_margins(name, length, seed):
    """How close the first layer's choice of experts is to another one, per token."""
    config, weights = plain_weights(name)
    layer = config["layers"][0]
    p = f"l{pk.owner(config, 0)}."
    x = np.repeat(weights["embed"][np.asarray(request_tokens(name, length, seed))][:, None, :], config["streams"], axis=1)
    h = pk.dynamic_tanh(pk.gather_streams(x, weights[p + "hc1.in"]), weights, p + "norm1")
    y = pk.attention_mixer(h, weights, p + "mix.", layer["mixer"])
    x = pk.spread_update(x, y, weights[p + "hc1.mix"], weights[p + "hc1.out"])
    h = pk.dynamic_tanh(pk.gather_streams(x, weights[p + "hc2.in"]), weights, p + "norm2")
    return pk.choice_margin(h, weights, p + "mlp.", layer["mlp"])


def model_close(got, ref, dtype, what):
    """Row by row: the root mean square of the difference over the vocabulary (its mean taken off) against the root mean square
    of the plain logits."""
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    assert np.isfinite(got).all(), what
    diff = got - ref
    diff = diff - diff.mean(axis=-1, keepdims=True)
    per_row = np.sqrt((diff ** 2).mean(axis=-1)) / np.sqrt(((ref - ref.mean()) ** 2).mean())
    assert per_row.max() <= MODEL_TOL[dtype], (
        f"{what}: relative error {per_row.max():.3e} > {MODEL_TOL[dtype]:.1e} ({dtype}); first wrong row "
        f"{int(np.argmax(per_row > MODEL_TOL[dtype]))} of {len(per_row)}, the worst {int(np.argmax(per_row))}")


class Routes:
    """Collects the experts the engine uses, layer by layer, while steps run directly (``on_route`` is called by every
    routed feed-forward with the ids of the step's rows)."""

    def __init__(self, lm):
        self.parts = [block.feed_forward for block in lm.model.blocks if hasattr(block.feed_forward, "route_log")]
        self.step = []

    def __enter__(self):
        for part in self.parts:
            part.on_route = lambda ids: self.step.append(ids.cpu().numpy().copy())
        return self

    def __exit__(self, *exc):
        for part in self.parts:
            part.on_route = None
        return False


def run_schedule(lm, requests, steps, routes=None):
    """``steps``: lists of (request, first position, end position); every place is wanted.  A request gets its slot
    at its first step and gives it back after its last token.  Returns request -> logits [length, vocab] and, with
    ``routes``, request -> the experts used, per layer with experts [length, top]."""
    engine = lm.engine
    slots, rows_of, used = {}, {key: [] for key in requests}, {key: None for key in requests}
    for step in steps:
        for key, lo, hi in step:
            if key not in slots:
                slots[key] = engine.new_sequence()
        if routes is not None:
            routes.step.clear()
        out = engine.step([slots[k] for k, _, _ in step], [requests[k][lo:hi] for k, lo, hi in step],
                          [list(range(hi - lo)) for _, lo, hi in step]).float().cpu().numpy()
        at = 0
        for key, lo, hi in step:
            rows_of[key].append(out[at:at + hi - lo])
            if routes is not None:
                if used[key] is None:
                    used[key] = [[] for _ in routes.step]
                for run, ids in enumerate(routes.step):
                    used[key][run].append(ids[at:at + hi - lo])
            at += hi - lo
            if hi == len(requests[key]):
                engine.release(slots.pop(key))
    engine.check()
    engine.cache.check()
    assert not slots
    logits = {key: np.concatenate(parts) for key, parts in rows_of.items()}
    if routes is None:
        return logits, None
    return logits, {key: [np.concatenate(parts) for parts in runs] for key, runs in used.items()}


def check_request(name, dtype, length, seed, got, used, what):
    """float32: against the plain model as it is.  bfloat16: against the plain model made to use the experts the engine
    used, and the engine's experts against the plain model's own, which may differ only where the choice is close."""
    plain, own = plain_run(name, length, seed)
    if dtype == "float32":
        model_close(got, plain, dtype, what)
        return
    config, weights = plain_weights(name)
    model_close(got, pk.forward(config, weights, request_tokens(name, length, seed), forced_routes=used), dtype, what)
    if own and own[0].shape[1] < config["layers"][0]["mlp"]["router"]["experts"]:
        differs = (np.sort(own[0], axis=-1) != np.sort(used[0], axis=-1)).any(axis=-1)
        margins = first_margins(name, length, seed)
        assert not (differs & (margins > ROUTE_MARGIN)).any(), f"{what}: other experts than the plain model's where the choice is clear"


def through(name, dtype, requests, steps, seeds, what):
    lm = loaded(name, dtype, record_steps=dtype == "float32")
    if dtype == "float32":
        got, used = run_schedule(lm, requests, steps)
    else:
        with Routes(lm) as routes:
            got, used = run_schedule(lm, requests, steps, routes)
    for key, ids in requests.items():
        check_request(name, dtype, len(ids), seeds[key], got[key], used[key] if used else None, f"model {name}, {what}, request {key}")


@BOTH
@pytest.mark.parametrize("name", sorted(ALL))
def test_whole_prompts(name, dtype):
    for length, seed in ((1, 0), (2, 1), (63, 2), (64, 3), (65, 4), (300, 5)):
        through(name, dtype, {"r": request_tokens(name, length, seed)}, [[("r", 0, length)]], {"r": seed}, f"{length} tokens whole")


@BOTH
@pytest.mark.parametrize("name", sorted(ALL))
def test_prompt_then_token_by_token(name, dtype):
    length, tail = 260, 140                 # the decoded tokens cross page borders (64) and pass every window's edge
    steps = [[("r", 0, length - tail)]] + [[("r", p, p + 1)] for p in range(length - tail, length)]
    through(name, dtype, {"r": request_tokens(name, length, 6)}, steps, {"r": 6}, f"last {tail} tokens one by one")


@BOTH
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_a_sequence_decoded_from_its_first_token(name, dtype):
    length = 140
    through(name, dtype, {"r": request_tokens(name, length, 7)}, [[("r", p, p + 1)] for p in range(length)], {"r": 7},
            "one token a step from the start")


@BOTH
@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("portion", [2, 3, 17, 64, 65])
def test_prompts_in_portions(name, dtype, portion):
    length = 135
    steps = [[("r", lo, min(lo + portion, length))] for lo in range(0, length, portion)]
    through(name, dtype, {"r": request_tokens(name, length, 8)}, steps, {"r": 8}, f"portions of {portion}")


@BOTH
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_requests_in_one_batch_then_decoded_together_over_reused_slots(name, dtype):
    for turn in range(2):                 # the second turn takes the slots and pages the first gave back
        lengths = {"a": 1 + 30, "b": 70 + 30, "c": 200 + 30, "d": 64 + 12, "e": 129 + 5} if turn == 0 else \
                  {"a": 90 + 25, "b": 3 + 25, "c": 64 + 25}
        tails = {"a": 30, "b": 30, "c": 30, "d": 12, "e": 5} if turn == 0 else {"a": 25, "b": 25, "c": 25}
        seeds = {k: 20 + turn * 10 + i for i, k in enumerate(lengths)}
        requests = {k: request_tokens(name, n, seeds[k]) for k, n in lengths.items()}
        steps = [[(k, 0, lengths[k] - tails[k]) for k in lengths]]
        for t in range(max(tails.values())):
            steps.append([(k, lengths[k] - tails[k] + t, lengths[k] - tails[k] + t + 1) for k in lengths if t < tails[k]])
        through(name, dtype, requests, steps, seeds, f"batch, turn {turn}")


def test_a_long_sequence_decoded_for_hundreds_of_tokens():
    name, length, tail = "B", 700, 400
    steps = [[("r", 0, length - tail)]] + [[("r", p, p + 1)] for p in range(length - tail, length)]
    through(name, "float32", {"r": request_tokens(name, length, 9)}, steps, {"r": 9}, "four hundred tokens one by one")


@pytest.mark.parametrize("name", ["A", "C"])
def test_recorded_decode_steps_equal_direct_ones(name):
    """Five sequences decode in a recorded step of six rows, the last sequence twice: the cache must come
    out as if it were there once."""
    results = []
    for record in (False, True):
        lm = loaded(name, "bfloat16", record_steps=record)
        engine = lm.engine
        prompts = [request_tokens(name, n, 40 + i) for i, n in enumerate((5, 64, 1, 30, 100))]
        slots = [engine.new_sequence() for _ in prompts]
        rows = [engine.step(slots, prompts).float().cpu().numpy()]
        for step in range(12):
            tokens = [[(7 * step + 3 * i) % ALL[name][0]["vocab"]] for i in range(len(slots))]
            rows.append(engine.step(slots, tokens).float().cpu().numpy())
        for slot in slots:
            engine.release(slot)
        if record:
            assert engine.steps_replayed > 0
        results.append(np.stack(rows))
    assert np.array_equal(results[0], results[1])


def test_pages_outside_the_window_go_back_to_the_pool():
    lm = loaded("C", "float32")                       # windows of 100, 64 and 130 keys, and none
    engine = lm.engine
    slot = engine.new_sequence()
    engine.step([slot], [request_tokens("C", 700, 50)])
    held = {group.window: group.pool.num_held for group in engine.cache.groups}
    assert held == {w: 700 // 64 + 1 - ((700 - w + 1) // 64 if w else 0) for w in (100, 64, 130, None)}
    engine.release(slot)
    engine.cache.check()
    assert all(group.pool.num_held == 0 for group in engine.cache.groups)


def test_company_and_wanted_places_do_not_change_a_requests_logits():
    name = "C"
    lm = loaded(name, "float32")
    engine = lm.engine
    ids = request_tokens(name, 130, 70)
    alone, _ = run_schedule(lm, {"r": ids}, [[("r", 0, 130)]])
    slots = [engine.new_sequence() for _ in range(3)]
    others = [request_tokens(name, n, 71 + n) for n in (200, 7)]
    out = engine.step(slots, [others[0], ids, others[1]], [[], [0, 64, 129], [6]]).float().cpu().numpy()
    for slot in slots:
        engine.release(slot)
    model_close(out[:3], alone["r"][[0, 64, 129]], "float32", "in company")


def test_a_norm_of_another_kind_runs_on_copies_in_a_whole_model():
    """The same plan with RMS norms: the sum of the copies goes through a buffer to a norm that knows nothing of them."""
    import dataclasses
    import torch
    from fieldrun_b200.config import PartSpec
    from fieldrun_b200.config.kifunex import KifunexConfig
    from fieldrun_b200.engine.engine import Engine
    from fieldrun_b200.engine.model import DecoderModel
    from fieldrun_b200.models.kifunex import kifunex_plan
    from fieldrun_b200.weights import FolderSource
    name = "A"
    plan = kifunex_plan(KifunexConfig.from_dict(ALL[name][0]))

    def rms(spec):
        return PartSpec("rmsnorm", {"width": spec.args["width"], "eps": 1e-5}, {"weight": spec.tensors["weight"]}) if spec else None

    layers = tuple(dataclasses.replace(layer, mixer_norm=rms(layer.mixer_norm), feed_forward_norm=rms(layer.feed_forward_norm))
                   for layer in plan.layers)
    model = DecoderModel(dataclasses.replace(plan, layers=layers, final_norm=rms(plan.final_norm)), torch.float32)
    source = FolderSource(model_folder(name), model.tensor_needs(), torch.float32, "cuda")
    model.load(source)
    source.close()
    engine = Engine(model, max_tokens=512)
    ids = request_tokens(name, 90, 80)
    slot = engine.new_sequence()
    got = [engine.step([slot], [ids[:80]], [list(range(80))])] + [engine.step([slot], [[t]]) for t in ids[80:]]
    config, weights = plain_weights(name)
    kept = pk.dynamic_tanh
    pk.dynamic_tanh = lambda v, t, n: v / np.sqrt((v * v).mean(axis=-1, keepdims=True) + 1e-5) * t[n]
    try:
        want = pk.forward(config, weights, ids)
    finally:
        pk.dynamic_tanh = kept
    model_close(np.concatenate([g.float().cpu().numpy() for g in got]), want, "float32", "RMS norms")


def test_greedy_generation_through_the_entry_point():
    name = "A"
    config, weights = plain_weights(name)
    lm = loaded(name, "float32")
    prompts = [request_tokens(name, n, 60 + i) for i, n in enumerate((9, 1, 70))]
    got = lm.generate_batch(prompts, max_tokens=14, ignore_eos=True)
    for prompt, tokens in zip(prompts, got):
        ids = list(prompt)
        for _ in range(14):
            row = pk.forward(config, weights, ids)[-1]
            top2 = np.sort(row)[-2:]
            assert top2[1] - top2[0] > 1e-4, "a near tie: the case does not pin the greedy choice"
            ids.append(int(np.argmax(row)))
        assert tokens == ids[len(prompt):]
    assert lm.generate(prompts[0], 5) == got[0][:5]


@BOTH
def test_a_trace_replayed_through_the_runner(tmp_path, dtype):
    """bin/trace_run as a user drives it: a batch of three prompts of unequal lengths (one of a single token, one of
    which nothing is wanted), decoded together while the shorter requests end, then another batch in the freed slots."""
    name = "D"                            # no close call among its routers: both of its two experts are always used
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    vocab = ALL[name][0]["vocab"]
    lengths = {"p": 1 + 6, "q": 80 + 20, "r": 130 + 9, "s": 65 + 12}
    heads = {"p": 1, "q": 80, "r": 130, "s": 65}
    ids = {k: request_tokens(name, n, 70 + i) for i, (k, n) in enumerate(lengths.items())}
    steps, rows, step = [], {k: [] for k in ids}, 0
    for batch in (["p", "q", "r"], ["s"]):
        entries = []
        at = 0
        for k in batch:
            want = [] if k == "q" else ([0] if heads[k] == 1 else [0, heads[k] // 2, heads[k] - 1])
            entries.append({"id": k, "tokens": ids[k][:heads[k]], "want": want})
            for w in want:
                rows[k].append((step, at, w))
                at += 1
        steps.append({"step": step, "entries": entries, "end": []})
        step += 1
        for t in range(max(lengths[k] - heads[k] for k in batch)):
            live = [k for k in batch if heads[k] + t < lengths[k]]
            steps.append({"step": step, "entries": [{"id": k, "tokens": [ids[k][heads[k] + t]], "want": [0]} for k in live],
                          "end": [k for k in live if heads[k] + t == lengths[k] - 1]})
            for row, k in enumerate(live):
                rows[k].append((step, row, heads[k] + t))
            step += 1
    text = "".join(json.dumps(x) + "\n" for x in steps)
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model_folder(name), "--dtype", dtype,
                           "--out", str(tmp_path), "--max-tokens", "384"], input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [line for line in proc.stdout.splitlines() if line.startswith("done ")] == [f"done {x['step']}" for x in steps]
    out = {}
    for x in steps:
        wanted = sum(len(e["want"]) for e in x["entries"])
        if wanted:
            out[x["step"]] = np.fromfile(os.path.join(tmp_path, f"{x['step']}.f32"), dtype="<f4").reshape(wanted, vocab)
    for i, (k, n) in enumerate(lengths.items()):
        plain = plain_run(name, n, 70 + i)[0]
        got = np.stack([out[s][row] for s, row, _ in rows[k]])
        model_close(got, plain[[pos for _, _, pos in rows[k]]], dtype, f"request {k}")


def test_command_line_generates_with_the_design(tmp_path):
    """`python -m fieldrun_b200 random` writes a model of the design from a config.json, and the command line
    generates from it what the plain model's greedy loop gives."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(ALL["D"][0]))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, "-m", "fieldrun_b200", "random", "--config", str(config_path), "--seed", "9", "--std", "0.2",
                           "--bias-std", "0.3", "-o", str(folder)], capture_output=True, text=True, cwd=root, timeout=300)
    assert made.returncode == 0, made.stderr
    with open(folder / "config.json") as handle:
        config = json.load(handle)
    from fieldrun_b200.weights.safetensors_io import ModelFolder
    files = ModelFolder(str(folder))
    weights = {n: files.tensor(n).double().numpy() for n in files.entries}
    files.close()
    ids = request_tokens("D", 20, 90)
    (tmp_path / "ids.json").write_text(json.dumps(ids))
    run = subprocess.run([sys.executable, "-m", "fieldrun_b200", "--model", str(folder), "--ids", str(tmp_path / "ids.json"), "--ctx", "12",
                          "--generate", "6", "--dtype", "float32", "--eos", "none"], capture_output=True, text=True, cwd=root, timeout=600)
    assert run.returncode == 0, run.stderr
    want = ids[:12]
    for _ in range(6):
        want.append(int(np.argmax(pk.forward(config, weights, want)[-1])))
    assert " ".join(str(t) for t in want[12:]) in run.stdout, run.stdout
