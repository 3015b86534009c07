"""Small configurations of the Duzinex design for the tests, with random weights of a spread that makes every mechanism
matter.  They differ from one another in every size, in the order of the layers and in every constant: a loop over the middle
layers, over the first ones, over the last one, one that runs once, and none; windows of 5 to 200 over pages of 64 and none;
no first tokens kept, a few, more than a page of them, more than the window has; rotations over all of a map, a part of it and
none; capped and plain scores; one to four query heads a key head; value sizes below, at and above twice the key size;
decays of nothing, a third, close to one and one; widths that are no multiple of four; a layer without feed-forward.
``C`` has sizes that the tensor-core kernels take, among them value heads of the keys' size and of twice that."""
import functools
import json
import os
import tempfile

import numpy as np

import fieldrun_b200 as fr
from fieldrun_b200 import RandomInit
from fieldrun_b200.weights.safetensors_io import ModelFolder


def dense(ff):
    return {"kind": "dense", "ff": ff}


def attention(heads, kv_heads, dim, vdim, scale, diff, mlp, *, mask=None, rot=None, softcap=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if mask is not None:
        mixer["mask"] = {"size": mask[0], "keep_first": mask[1]}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
    if softcap is not None:
        mixer["softcap"] = softcap
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def retention(heads, dim, vdim, decay, mlp):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def mingru(width, mlp):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


CONFIG_A = {
    "architecture": "Duzinex", "vocab": 131, "width": 96, "embedding": {"scale": 5.0}, "norm": {"eps": 1e-5},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        attention(4, 2, 24, 40, 0.3, 0.35, dense(112), mask=(33, 3), rot=(16, 1000.0), softcap=9.0),
        mingru(72, dense(50)),
        attention(3, 3, 16, 16, 0.4, 0.7, None, mask=(70, 75), rot=(16, 50.0)),
        retention(3, 20, 36, [0.9921, 0.9, 0.31], dense(80)),
    ],
}
INIT_A = RandomInit(seed=21, matrix_std=0.09, norm_std=0.2, bias_std=0.4)

CONFIG_B = {
    "architecture": "Duzinex", "vocab": 77, "width": 42, "embedding": {"scale": 9.0}, "norm": {"eps": 1e-6},
    "layers": [
        retention(2, 9, 33, [0.0, 1.0], dense(30)),
        attention(4, 1, 10, 20, 0.5, 0.2, dense(44), softcap=4.0),
        mingru(33, None),
        attention(2, 2, 8, 30, 0.6, 0.9, dense(20), mask=(200, 0), rot=(2, 300.0)),
    ],
}
INIT_B = RandomInit(seed=22, matrix_std=0.14, norm_std=0.15, bias_std=0.6)

CONFIG_C = {
    "architecture": "Duzinex", "vocab": 200, "width": 128, "embedding": {"scale": 7.0}, "norm": {"eps": 1e-6},
    "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": [
        attention(4, 2, 64, 128, 0.12, 0.45, dense(256), mask=(100, 70), rot=(64, 10000.0), softcap=20.0),
        retention(2, 64, 64, [0.98, 0.9995], dense(128)),
        attention(6, 1, 32, 64, 0.2, 0.6, dense(192), mask=(64, 5), rot=(32, 500.0), softcap=6.0),
        attention(2, 2, 128, 128, 0.09, 0.3, dense(128), mask=(130, 1), rot=(32, 1000.0)),
        retention(3, 32, 128, [0.7, 0.97, 0.999], None),
        mingru(160, dense(256)),
    ],
}
INIT_C = RandomInit(seed=23, matrix_std=0.07, norm_std=0.1, bias_std=0.3)

CONFIG_D = {
    "architecture": "Duzinex", "vocab": 64, "width": 31, "embedding": {"scale": 6.0}, "norm": {"eps": 1e-5},
    "loop": {"start": 2, "stop": 3, "times": 2},
    "layers": [
        mingru(17, dense(23)),
        retention(1, 5, 7, [0.95], dense(40)),
        attention(2, 1, 6, 5, 0.7, 0.5, None, mask=(5, 2), rot=(4, 20.0)),
    ],
}
INIT_D = RandomInit(seed=24, matrix_std=0.17, norm_std=0.1, bias_std=0.5)

# a loop that runs once: the embedding is never added again
CONFIG_E = dict(CONFIG_D, loop={"start": 0, "stop": 2, "times": 1})
INIT_E = RandomInit(seed=25, matrix_std=0.17, norm_std=0.1, bias_std=0.5)

ALL = {"A": (CONFIG_A, INIT_A), "B": (CONFIG_B, INIT_B), "C": (CONFIG_C, INIT_C), "D": (CONFIG_D, INIT_D), "E": (CONFIG_E, INIT_E)}

_ROOT = tempfile.mkdtemp(prefix="fieldrun_b200_duzinex_")


@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    config, init = ALL[name]
    folder = os.path.join(_ROOT, name)
    fr.write_random_model(folder, config, init)
    return folder


@functools.lru_cache(maxsize=None)
def plain_weights(name: str):
    """(config.json as a dictionary, tensors as float64 arrays by name) of the written folder."""
    folder = model_folder(name)
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as handle:
        config = json.load(handle)
    files = ModelFolder(folder)
    try:
        weights = {n: files.tensor(n).double().numpy() for n in files.entries}
    finally:
        files.close()
    return config, weights


def request_tokens(name: str, length: int, seed: int) -> list[int]:
    vocab = ALL[name][0]["vocab"]
    return np.random.default_rng(7919 * seed + length).integers(0, vocab, size=length).tolist()
