"""Small configurations of the Kifunex design for the tests, with random weights of a spread that makes every mechanism
matter.  They differ from one another in every size, in the order of the layers and in every constant: one to nine copies of
the stream; windows of 1 to 200 over pages of 64 and none; rotations over all of a head, a part of it and none, with frequencies
that all stay, are all divided and are blended; one to eight query heads a key head; expert scales below and above one, all
experts used, with and without shared expert; layers that run an earlier layer's tensors, a later one's, and one whose owner is
itself such a layer's; layers without feed-forward; scaled and capped logits and plain ones; widths that are no multiple of
four.  ``C`` has sizes that the tensor-core kernels take."""
import functools
import json
import os
import tempfile

import numpy as np

import fieldrun_b200 as fr
from fieldrun_b200 import RandomInit
from fieldrun_b200.weights.safetensors_io import ModelFolder


def moe(ff, experts, top, scale=None, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if scale is not None:
        mlp["router"]["scale"] = scale
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def attention(heads, kv_heads, dim, scale, mlp, *, window=None, rot=None, blend=None):
    """``rot`` (dims, base); ``blend`` (factor, low, high, original)."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window is not None:
        mixer["mask"] = {"size": window}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
        if blend is not None:
            mixer["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), blend))
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def again(layers, owner):
    return dict(layers[owner], weights_of=owner)


_A = [attention(4, 2, 24, 0.3, moe(40, 7, 3, 2.5, 56), window=33, rot=(16, 1000.0), blend=(8.0, 1.0, 4.0, 200.0)),
      attention(3, 3, 16, 0.35, None, window=70, rot=(16, 50.0), blend=(3.0, 2.0, 3.0, 40.0)),
      attention(6, 1, 20, 0.25, moe(24, 5, 2, 0.7), rot=(8, 300.0))]
CONFIG_A = {"architecture": "Kifunex", "vocab": 131, "width": 96, "streams": 3, "norm": {"eps": 1e-5}, "logit_scale": 0.6,
            "logit_softcap": 9.0, "layers": _A + [again(_A, 1), again(_A, 0), again(_A, 2)]}
INIT_A = RandomInit(seed=31, matrix_std=0.09, norm_std=0.2, bias_std=0.3)

_B = [attention(4, 1, 10, 0.5, moe(30, 4, 4, 1.3, 22), window=1),
      attention(2, 2, 9, 0.5, moe(18, 6, 1), window=200, rot=(2, 300.0), blend=(5.0, 1.0, 1.0, 30.0)),
      attention(5, 5, 12, 0.4, None, rot=(12, 20.0), blend=(4.0, 1.0, 4.0, 1e6))]
CONFIG_B = {"architecture": "Kifunex", "vocab": 77, "width": 42, "streams": 2, "norm": {"eps": 1e-6}, "logit_scale": 1.7,
            "layers": [_B[0], dict(_B[2], weights_of=3), _B[1], _B[2], dict(_B[1], weights_of=2)]}
INIT_B = RandomInit(seed=32, matrix_std=0.14, norm_std=0.15, bias_std=0.3)

_C = [attention(8, 2, 64, 0.12, moe(128, 8, 2, 1.4, 256), window=100, rot=(64, 10000.0), blend=(8.0, 1.0, 4.0, 128.0)),
      attention(6, 1, 32, 0.2, moe(64, 3, 2, 0.8, 32), window=64, rot=(16, 500.0)),
      attention(2, 2, 128, 0.09, moe(256, 5, 3, 1.0, 128), window=130, rot=(32, 1000.0), blend=(2.0, 1.0, 8.0, 500.0)),
      attention(4, 1, 96, 0.1, None)]
CONFIG_C = {"architecture": "Kifunex", "vocab": 200, "width": 128, "streams": 4, "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "logit_softcap": 20.0, "layers": _C + [again(_C, 0), again(_C, 2)]}
INIT_C = RandomInit(seed=33, matrix_std=0.07, norm_std=0.1, bias_std=0.2)

_D = [attention(2, 1, 6, 0.7, moe(20, 2, 2, 1.5, 14), window=5, rot=(4, 20.0), blend=(4.0, 1.0, 2.0, 16.0))]
CONFIG_D = {"architecture": "Kifunex", "vocab": 64, "width": 31, "streams": 1, "norm": {"eps": 1e-5}, "logit_softcap": 5.0,
            "layers": _D + [again(_D, 0)]}
INIT_D = RandomInit(seed=34, matrix_std=0.17, norm_std=0.1, bias_std=0.4)

_E = [attention(3, 1, 8, 0.6, moe(12, 3, 3, 0.5, 9), window=20, rot=(8, 100.0)), attention(2, 2, 14, 0.4, moe(16, 4, 4, 0.9), window=90)]
CONFIG_E = {"architecture": "Kifunex", "vocab": 50, "width": 40, "streams": 9, "norm": {"eps": 1e-5}, "layers": _E + [again(_E, 1)]}
INIT_E = RandomInit(seed=35, matrix_std=0.12, norm_std=0.12, bias_std=0.4)

ALL = {"A": (CONFIG_A, INIT_A), "B": (CONFIG_B, INIT_B), "C": (CONFIG_C, INIT_C), "D": (CONFIG_D, INIT_D), "E": (CONFIG_E, INIT_E)}

_ROOT = tempfile.mkdtemp(prefix="fieldrun_b200_kifunex_")


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
