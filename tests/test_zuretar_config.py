"""Zuretar on the CPU: configuration, plan, tensor names, refusals, cache needs, and the plain implementation against itself."""
import copy
import math

import pytest
import torch

from forge_b200.cache.storage import plan_groups
from forge_b200.config import ConfigError, PartSpec, config_from_dict
from forge_b200.engine.model import Model
from forge_b200.parts import CompositeCacheSpec, KVCacheSpec, Runtime, StateSpec, build_part
from plain import zuretar as PZ
from zatupel_models import rand
from zuretar_models import ZUR, zur_config

CPU = Runtime(torch.device("cpu"), torch.float32)


def _model(name):
    return Model(zur_config(name).plan(), CPU)


def test_registered_by_its_architecture_name():
    from forge_b200.config.zuretar import ZuretarConfig
    assert isinstance(zur_config("E"), ZuretarConfig)
    p = zur_config("E").plan()
    assert p.schedule == [0, 1, 1, 2, 0] and [l.weight_prefix for l in p.layers] == ["l0.", "l1.", "l3."]
    assert [l.mixer.kind for l in p.layers] == ["side_by_side", "gated_delta", "gated_delta"]
    assert [l.feed_forward.kind for l in p.layers] == ["swiglu", "routed_experts", "none"]
    assert zur_config("E").num_hidden_layers == 5 and zur_config("J").plan().schedule == [0, 0, 0]
    assert zur_config("F").plan().schedule == [0, 1, 2, 1, 3] and zur_config("F").plan().layers[3].weight_prefix == "l4."


def test_tensor_names_and_shapes():
    specs = _model("E").tensor_specs()
    for name, shape in {"embed": (197, 75), "final.norm": (75,), "head": (197, 75), "l0.norm1": (75,), "l0.mix.left.q": (60, 75),
                        "l0.mix.left.k": (20, 75), "l0.mix.left.v": (26, 75), "l0.mix.left.sink": (6,), "l0.mix.left.o": (75, 78),
                        "l0.mix.right.q": (27, 75), "l0.mix.right.k": (27, 75), "l0.mix.right.v": (15, 75), "l0.mix.right.g": (15, 75),
                        "l0.mix.right.o": (75, 15), "l0.mix.right.norm": (15,), "l0.mix.left.out": (75,), "l0.mix.right.out": (75,),
                        "l0.mlp.gate": (41, 75), "l0.mlp.gate.b": (41,), "l0.mlp.up.b": (41,), "l0.mlp.down": (75, 41), "l0.mlp.down.b": (75,),
                        "l1.mix.q": (33, 75), "l1.mix.q.conv": (33, 3), "l1.mix.k.conv": (33, 3), "l1.mix.v": (42, 75), "l1.mix.v.conv": (42, 3),
                        "l1.mix.b": (6, 75), "l1.mix.a": (6, 75), "l1.mix.A_log": (6,), "l1.mix.dt_bias": (6,), "l1.mix.norm": (7,),
                        "l1.mix.g": (42, 75), "l1.mix.o": (75, 42), "l1.mlp.router": (6, 75), "l1.mlp.correction": (6,), "l1.mlp.e5.gate": (24, 75),
                        "l1.mlp.e0.down": (75, 24), "l3.mix.q.conv": (12, 1)}.items():
        assert tuple(specs[name].shape) == shape, name
    assert not any(n.startswith(("l2.", "l4.")) for n in specs)                       # layers with another layer's weights have no tensors
    assert "l3.mlp.gate" not in specs and "l1.mlp.e0.gate.b" not in specs and "l0.mix.left.q.b" not in specs and "l0.norm2" not in specs
    assert all(s.required for s in specs.values())


def test_cache_needs():
    m = _model("E")
    specs = m.cache_specs()
    assert len(specs) == 5 and m.cache_from() == [None] * 5                            # every run keeps a cache of its own
    assert specs[0] == specs[4] == CompositeCacheSpec((KVCacheSpec(2, 10, None, v_head_dim=13, chunk=7), StateSpec((136,))))     # 3*9*5 = 135, filled up
    # six 11 x 7 matrices and three rows of 2*3*11 + 6*7 inputs of the convolutions
    assert specs[1] == specs[2] == StateSpec((6 * 77 + 3 * 108 + 2,))
    groups, _ = plan_groups(specs, m.cache_from())
    assert len(groups) == 1
    assert m.graph_safe()


@pytest.mark.parametrize("change, message", [
    (lambda d: d["layers"][1].update(type="attention"), "type"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda d: d["layers"][0]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("mask"), "mask"),
    (lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "rot"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=12), "rot"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda d: d["layers"][0]["mixer"]["right"].pop("decay"), "decay"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda d: d["layers"][1]["mlp"].update(kind="gelu"), "mlp.kind"),
    (lambda d: d["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda d: d["layers"][2].update(weights_of=5), "weights_of"),
    (lambda d: d["layers"][2].update(weights_of=2), "weights_of"),
    (lambda d: (d["layers"][2].update(weights_of=4), d["layers"][4].update(weights_of=2)), "weights_of"),
    (lambda d: d["layers"][2].update(weights_of=0), "differs"),
    (lambda d: d["layers"][2]["mixer"].update(vdim=8), "differs"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_refusals(change, message):
    d = copy.deepcopy(ZUR["E"])
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_what_the_parts_refuse():
    base = {"hidden_size": 16, "num_heads": 4, "head_dim": 8, "eps": 1e-5}
    for kind, more in (("gated_delta", {"taps": 0}), ("gated_delta", {"taps": 2, "num_qk_heads": 3}), ("gated_delta", {"taps": 2, "head_dim": 257}),
                       ("lightning", {"decay": [0.5]}), ("lightning", {"decay": [0.5] * 4, "head_dim": 300})):
        with pytest.raises(ConfigError):
            build_part("mixer", PartSpec(kind, {**base, **more}), CPU)
    att = {"hidden_size": 16, "num_heads": 4, "num_kv_heads": 2, "head_dim": 8}
    with pytest.raises(ConfigError, match="inv_freq"):                       # pairs of neighbours are another rotation
        build_part("mixer", PartSpec("masked_attention", dict(att, position=PartSpec("rope_pairs", {"head_dim": 8}))), CPU)
    with pytest.raises(ConfigError, match="output norms"):
        build_part("mixer", PartSpec("side_by_side", {"mixers": [PartSpec("masked_attention", att)], "hidden_size": 16, "out_norms": ["a", "b"], "eps": 1e-5}), CPU)
    with pytest.raises(ConfigError, match="two largest"):
        build_part("feed_forward", PartSpec("routed_experts", {"hidden_size": 16, "intermediate_size": 8, "experts": 4, "top": 1, "group_top": 3}), CPU)


def test_to_dict_round_trip_and_keys_that_are_absent():
    for name in ZUR:
        cfg = zur_config(name)
        assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == ZUR[name]
    d = copy.deepcopy(ZUR["G"])
    del d["layers"][0]["mixer"]["kv_heads"], d["layers"][2]["mixer"]["kv_heads"]      # as many query/key heads as heads
    del d["layers"][1]["mixer"]["left"]["rot"]["scaling"]
    d["layers"][3]["weights_of"] = None
    p = config_from_dict(d).plan()
    assert p.layers[0].mixer.params["num_qk_heads"] == 4 and p.schedule == [0, 1, 0, 2]
    assert build_part("mixer", p.layers[1].mixer.params["mixers"][0], CPU).position.amplitude == 1.0
    d["layers"][1]["weights_of"] = 1
    with pytest.raises(ConfigError):
        config_from_dict(d)


def test_weights_of_a_layer_that_uses_another_layers():
    d = copy.deepcopy(ZUR["J"])
    d["layers"][2]["weights_of"] = 1                                          # through a layer that has none of its own
    assert config_from_dict(d).plan().schedule == [0, 0, 0] and PZ.weights_layer(d["layers"], 2) == 0
    # the layer with the weights may come later
    d["layers"][0]["weights_of"], d["layers"][2] = 2, {k: v for k, v in d["layers"][2].items() if k != "weights_of"}
    d["layers"][1]["weights_of"] = 2
    p = config_from_dict(d).plan()
    assert p.schedule == [0, 0, 0] and p.layers[0].weight_prefix == "l2."


# ------------------------------------------------------------------------------------ the plain implementation against itself

def test_the_convolution_looks_back_and_no_further():
    x, w = rand(12, 3, seed=1).double(), rand(3, 4, seed=2).double()
    y = PZ.short_convolution(x, w)
    assert torch.allclose(y[0], x[0] * w[:, 3]) and torch.allclose(y[7], x[4] * w[:, 0] + x[5] * w[:, 1] + x[6] * w[:, 2] + x[7] * w[:, 3])
    assert torch.allclose(PZ.short_convolution(x, w[:, 3:]), x * w[:, 3])
    assert torch.allclose(PZ.short_convolution(x[:5], w), y[:5])


def test_the_delta_rule_replaces_what_a_key_held():
    k = torch.eye(3, dtype=torch.float64)[[0, 1, 0, 2]][:, None, :]
    v = torch.tensor([[1.0, 2.0], [3.0, 4.0], [5.0, 6.0], [0.0, 0.0]], dtype=torch.float64)[:, None, :]
    one = torch.ones(4, 1, dtype=torch.float64)
    o, S = PZ.delta_rule(k, k, v, one, one)
    assert torch.allclose(o[:, 0], v[:, 0])                                  # the read-out sees the write
    assert torch.allclose(S[0], torch.tensor([[5.0, 6.0], [3.0, 4.0], [0.0, 0.0]], dtype=torch.float64))
    _, half = PZ.delta_rule(k, k, v, one, one / 2)
    assert torch.allclose(half[0, 0], torch.tensor([2.75, 3.5], dtype=torch.float64))        # 1/2 -> 1/2 + (5 - 1/2) / 2
    _, S2 = PZ.delta_rule(k, k, v, one / 2, one)
    assert torch.allclose(S2[0, 1], torch.tensor([0.75, 1.0], dtype=torch.float64))          # two tokens' decay
    # carried over a cut
    q, kk, vv = rand(9, 2, 4, seed=1).double(), PZ.unit(rand(9, 2, 4, seed=2).double()), rand(9, 2, 5, seed=3).double()
    g, b = torch.sigmoid(rand(9, 2, seed=4).double()), torch.sigmoid(rand(9, 2, seed=5).double())
    o, S = PZ.delta_rule(q, kk, vv, g, b)
    o1, S1 = PZ.delta_rule(q[:4], kk[:4], vv[:4], g[:4], b[:4])
    o2, S2 = PZ.delta_rule(q[4:], kk[4:], vv[4:], g[4:], b[4:], state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)


def test_stretched_frequencies():
    f0, amp0 = PZ.rotation_frequencies(32, 1e4)
    f, amp = PZ.rotation_frequencies(32, 1e4, {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0})
    assert amp0 == 1.0 and abs(amp - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    assert torch.allclose(f[:2], f0[:2]) and torch.allclose(f[-2:], f0[-2:] / 8.0) and bool((f <= f0 + 1e-15).all() and (f >= f0 / 8.0 - 1e-15).all())
    x = rand(6, 2, 10, seed=2).double()
    y = PZ.rotate(x, {"dims": 6, "base": 100.0})
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    a = 5 * 100.0 ** (-2 / 6)
    assert torch.allclose(y[5, 1, 1], x[5, 1, 1] * math.cos(a) - x[5, 1, 4] * math.sin(a))
    assert torch.allclose(y[5, 1, 4], x[5, 1, 4] * math.cos(a) + x[5, 1, 1] * math.sin(a))


def test_chunks_and_the_sink():
    ok = PZ.chunk_mask(12, 5)
    assert ok[7].tolist() == [False] * 5 + [True] * 3 + [False] * 4 and ok[5].tolist() == [False] * 5 + [True] + [False] * 6
    s = rand(5, 5, seed=1).double()
    seen = PZ.chunk_mask(5, 9)
    p = PZ.softmax_with_sink(s, seen, torch.tensor(0.3, dtype=torch.float64))
    share = math.exp(0.3) / (torch.exp(s.masked_fill(~seen, -math.inf)).sum(-1) + math.exp(0.3))
    assert torch.allclose(p.sum(-1), 1.0 - share)
    assert float(PZ.softmax_with_sink(s, seen, torch.tensor(900.0, dtype=torch.float64)).max()) == 0.0


def test_lightning_in_closed_form():
    q, k, v = rand(7, 2, 3, seed=1).double(), rand(7, 2, 3, seed=2).double(), rand(7, 2, 4, seed=3).double()
    d = torch.tensor([0.5, 0.9], dtype=torch.float64)
    o, _ = PZ.linear_recurrence(q, k, v, d)
    for n in range(2):
        want = sum(d[n] ** (6 - j) * (q[6, n] @ k[j, n]) * v[j, n] for j in range(7))
        assert torch.allclose(o[6, n], want)


def test_groups_are_ranked_by_their_two_largest():
    w = {"router": torch.zeros(6, 4, dtype=torch.float64), "correction": torch.tensor([0.5, -0.9, 0.3, 0.25, -0.4, -0.45], dtype=torch.float64)}
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    idx, wts, _ = PZ.route(torch.ones(1, 4, dtype=torch.float64), w, r)
    assert idx.tolist() == [[2, 3]] and torch.allclose(wts, torch.full((1, 2), 0.5, dtype=torch.float64))    # 0.55 beats -0.4; weights without the correction
    idx, _, _ = PZ.route(torch.ones(1, 4, dtype=torch.float64), w, dict(r, groups={"count": 6, "keep": 3}))     # groups of one: their only number
    assert idx.tolist() == [[0, 2]]


def test_no_look_ahead():
    from zuretar_models import zur_tensors
    for name in ("E", "F"):
        t = zur_tensors(name)
        toks = torch.randint(0, ZUR[name]["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
        whole = PZ.forward(ZUR[name], t, toks)
        assert torch.allclose(PZ.forward(ZUR[name], t, toks[:23]), whole[:23])
