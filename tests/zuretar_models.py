"""Small Zuretar configurations for the tests, and model folders with random weights made from them.

They differ in every size, in the order and number of the layers and in every constant; among them they have what a single model can
hide: value heads narrower and wider than key heads in every mixer, one head and many, query/key heads that are shared by one, two and
three heads, convolutions over one, two, three, four and five tokens, an odd width, key channels that are no multiple of four, a rotation of
all and of some channels of a head, with and without stretched frequencies, chunks shorter than a page, of a page and a half, and longer than
any sequence, a score scale that is not the heads' size to the power -1/2, decays next to one and far from it, a dense and a routed
feed-forward and none beside either mixer, experts in one group, in groups of one, in groups that are all kept and of which some are
dropped, one expert a token and several, layers that use another layer's weights (once, twice, in a row, far apart), a model of one layer.
"""
import copy

from forge_b200.config import config_from_dict
from forge_b200.weights import random_tensors, write_random_model  # noqa: F401  (re-exported)
from forge_b200.weights.safetensors_io import write_safetensors


def _delta(heads, kv, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def _pair(heads, kv, dim, vdim, size, scale, rot, base, rheads, rdim, rvdim, decay, scaling=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale, "rot": {"dims": rot, "base": base}}
    if scaling is not None:
        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay}}}


def _moe(layer, ff, experts, top, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "router": router})


def _dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def _bare(layer):
    return dict(layer, mlp=None)


def _model(vocab, width, eps, layers):
    # a layer given as a number is that layer's entry again, with its weights
    return {"architecture": "Zuretar", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(copy.deepcopy(layers[e]), weights_of=e) if isinstance(e, int) else e for e in layers]}


ZUR = {
    # sizes that only the kernels of fp32 arithmetic take, everything odd
    "E": _model(197, 75, 1e-3, [_dense(_pair(6, 2, 10, 13, 7, 0.5, 6, 40.0, 3, 9, 5, [0.3, 0.9, 0.998], (3.0, 40, 8.0, 0.5)), 41),
                                _moe(_delta(6, 3, 11, 7, 3), 24, 6, 2, (3, 2)), 1, _bare(_delta(2, 2, 6, 15, 1)), 0]),
    "F": _model(130, 48, 1e-5, [_moe(_delta(3, 1, 16, 24, 2), 20, 5, 2, (5, 3)), _bare(_pair(4, 1, 12, 20, 96, 0.4, 12, 1e4, 2, 16, 8, [0.95, 0.5])),
                                _dense(_delta(4, 4, 8, 8, 5), 72), 1, _moe(_pair(2, 2, 14, 6, 1000, 0.3, 8, 300.0, 5, 4, 4, [0.1, 0.7, 0.9, 0.99, 0.9999]), 12, 9, 3,
                                                                           (3, 1))]),
    # widths at which the bfloat16 path takes the tensor-core products and the tensor-core attention kernel
    "G": _model(520, 192, 1e-6, [_dense(_delta(4, 2, 32, 48, 4), 320), _moe(_pair(8, 2, 64, 32, 72, 0.15, 48, 250000.0, 4, 32, 16, [0.6, 0.9, 0.97, 0.999],
                                                                                (8.0, 64, 16.0, 1.0)), 64, 8, 2, (4, 2)),
                                 0, _moe(_delta(3, 1, 64, 32, 4), 96, 4, 1)]),
    "H": _model(89, 64, 1e-4, [_dense(_delta(2, 1, 16, 32, 4), 40)]),
    "J": _model(101, 56, 1e-2, [_moe(_pair(3, 3, 16, 8, 20, 0.7, 16, 100.0, 2, 8, 24, [0.8, 0.97]), 16, 4, 4, (2, 2)), 0, 0]),
}
SEEDS = {"E": 61, "F": 62, "G": 63, "H": 64, "J": 65}
STDS = {"E": dict(std=0.15, embed_std=0.8, norm_std=0.2, bias_std=0.5), "F": dict(std=0.17, embed_std=0.7, norm_std=0.2, bias_std=0.5),
        "G": dict(std=0.08, embed_std=0.6, norm_std=0.2, bias_std=0.5), "H": dict(std=0.15, embed_std=0.6, norm_std=0.2, bias_std=0.5),
        "J": dict(std=0.15, embed_std=0.6, norm_std=0.2, bias_std=0.5)}
LENGTHS = {"E": [70, 129, 33, 150, 64, 97], "F": [90, 47, 16, 140, 81], "G": [160, 36, 131, 45], "H": [60, 33, 90, 41], "J": [50, 61, 22, 35]}


def zur_config(name):
    return config_from_dict(copy.deepcopy(ZUR[name]))


def zur_tensors(name, seed=None):
    """Random tensors as a file would hold them; half of every delta mixer's heads forget slowly."""
    t = random_tensors(zur_config(name), seed=SEEDS[name] if seed is None else seed, **STDS[name])
    for n in t:
        if n.endswith(".A_log"):
            t[n][::2] -= 5.0
    return t


def make_zur_dir(tmp_path_factory, name):
    import json
    import os
    d = str(tmp_path_factory.mktemp(f"zur{name}"))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(zur_config(name).to_dict(), f)
    write_safetensors(os.path.join(d, "model.safetensors"), zur_tensors(name))
    return d
