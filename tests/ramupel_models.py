"""Small Ramupel configurations for the tests, and model folders with random weights made from them.

They differ in every size, in the order and number of the layers and in every constant; among them they have what a single model can
hide: value heads narrower and wider than key heads in both mixers, one head and many, a latent narrower and wider than a head,
rotated parts of other widths than the unrotated ones, an odd width and an odd number of heads (rows that no vector load fits),
key channels that are no multiple of four, tau above one, one and below, a hidden layer of the decays of other sizes, an embedding
scale above one, one and below, a score scale that is not the heads' size to the power -1/2, a first layer of either kind, a layer
without a feed-forward (also the last one), a model of one layer.
"""
import copy

from forge_b200.config import config_from_dict
from forge_b200.weights import random_tensors
from forge_b200.weights.safetensors_io import write_safetensors


def _lat(heads, dim, rot_dim, vdim, kv_rank, scale, base, ff):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"dims": rot_dim, "base": base}}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _gla(heads, dim, vdim, tau, ff):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _model(vocab, width, eps, scale, layers):
    return {"architecture": "Ramupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


RAM = {
    # sizes that only the kernels of fp32 arithmetic take, everything odd
    "P": _model(203, 77, 1e-3, 0.7, [_gla(3, 10, 17, 4.0, 50), _lat(5, 6, 10, 9, 13, 0.6, 70.0, 41), _gla(1, 33, 5, 0.5, None),
                                     _lat(1, 20, 2, 30, 40, 0.31, 9e4, 96)]),
    "Q": _model(118, 48, 1e-5, 1.0, [_lat(2, 8, 4, 12, 20, 0.3, 1000.0, None), _lat(3, 16, 8, 4, 10, 0.45, 50.0, 72), _gla(6, 8, 8, 1.0, 24), _gla(2, 24, 40, 16.0, 64),
                                     _lat(2, 4, 12, 8, 24, 0.5, 300.0, None)]),
    # widths at which the bfloat16 path takes the tensor-core products and the tensor-core attention kernel
    "R": _model(530, 192, 1e-6, 9.0, [_lat(6, 32, 16, 48, 96, 0.17, 250000.0, 320), _gla(3, 64, 96, 7.0, 256), _lat(4, 48, 32, 32, 160, 0.12, 1e4, 448),
                                      _gla(5, 32, 16, 20.0, 128)]),
    "S": _model(89, 64, 1e-4, 3.0, [_gla(2, 16, 32, 2.5, 40)]),
}
SEEDS = {"P": 61, "Q": 52, "R": 53, "S": 54}
RANKS = {"P": {0: 3, 2: 37}, "Q": {2: 8, 3: 16}, "R": {1: 24, 3: 5}, "S": {0: 1}}          # the decays' hidden layers, by layer
STDS = {"P": dict(std=0.15, embed_std=0.8, norm_std=0.2, bias_std=0.5), "Q": dict(std=0.17, embed_std=0.7, norm_std=0.2, bias_std=0.5),
        "R": dict(std=0.08, embed_std=0.5, norm_std=0.2, bias_std=0.5), "S": dict(std=0.15, embed_std=0.6, norm_std=0.2, bias_std=0.5)}
# the last product of every sublayer is drawn this much larger: beside a tied head a stream that is mostly the embedding of the last
# token would name that token again and again
GAINS = {"P": 12.0, "Q": 3.0, "R": 30.0, "S": 8.0}
LENGTHS = {"P": [70, 129, 33, 150, 64, 97], "Q": [90, 47, 16, 140, 81], "R": [160, 36, 131, 45], "S": [60, 33, 90, 41]}


def ram_config(name):
    return config_from_dict(copy.deepcopy(RAM[name]))


def ram_tensors(name, seed=None):
    """Random tensors as a file would hold them, the decays' hidden layers of the sizes above."""
    import torch
    t = random_tensors(ram_config(name), seed=SEEDS[name] if seed is None else seed, **STDS[name])
    for n in t:
        if n.endswith("mix.o") or n.endswith("mlp.down"):
            t[n] = (t[n].float() * GAINS[name]).to(t[n].dtype)
    for i, r in RANKS[name].items():
        for suffix, axis in (("a1", 0), ("a2", 1)):
            old = t[f"l{i}.mix.{suffix}"]
            shape = list(old.shape)
            shape[axis] = r
            g = torch.Generator().manual_seed(100 * SEEDS[name] + 2 * i + axis)
            t[f"l{i}.mix.{suffix}"] = (torch.randn(shape, generator=g) * 0.4).to(old.dtype)
    return t


def make_ram_dir(tmp_path_factory, name):
    import json
    import os
    d = str(tmp_path_factory.mktemp(f"ram{name}"))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(ram_config(name).to_dict(), f)
    write_safetensors(os.path.join(d, "model.safetensors"), ram_tensors(name))
    return d
