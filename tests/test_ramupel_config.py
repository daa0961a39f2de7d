"""Ramupel on the CPU: configuration, plan, tensor names, refusals, cache needs, and the plain implementation against itself."""
import copy
import math

import pytest
import torch

from forge_b200.cache.storage import plan_groups
from forge_b200.config import ConfigError, config_from_dict
from forge_b200.engine.model import Model
from forge_b200.parts import KVCacheSpec, Runtime, StateSpec
from plain import ramupel as PR
from ramupel_models import RAM, RANKS, ram_config, ram_tensors
from zatupel_models import rand


def _model(name):
    return Model(ram_config(name).plan(), Runtime(torch.device("cpu"), torch.bfloat16))


def test_registered_by_its_architecture_name():
    from forge_b200.config.ramupel import RamupelConfig
    assert isinstance(ram_config("P"), RamupelConfig)
    p = ram_config("P").plan()
    assert p.depth_average and p.schedule == [0, 1, 2, 3] and [l.block for l in p.layers] == ["parallel_depth"] * 4
    assert [l.mixer.kind for l in p.layers] == ["gated_linear", "latent_attention", "gated_linear", "latent_attention"]
    assert [l.feed_forward.kind for l in p.layers] == ["dense", "dense", "none", "dense"]
    assert [l.block_params["depth"] for l in p.layers] == [2, 3, 4, 5]
    assert ram_config("Q").num_hidden_layers == 5 and ram_config("Q").vocab_size == 118 and ram_config("Q").hidden_size == 48


def test_tensor_names_and_shapes():
    specs = _model("P").tensor_specs()
    for name, shape in {"embed": (203, 77), "final.norm": (77,), "l0.norm1": (77,), "l0.rg1": (77, 77), "l0.rg1.b": (77,), "l0.rg2": (77, 77),
                        "l0.rg2.b": (77,), "l0.dwa": (2,), "l3.dwa": (5,), "l0.mix.q": (30, 77), "l0.mix.k": (30, 77), "l0.mix.v": (51, 77),
                        "l0.mix.g": (51, 77), "l0.mix.o": (77, 51), "l0.mix.norm": (17,), "l0.mix.a1": (-1, 77), "l0.mix.a2": (30, -1),
                        "l0.mix.a2.b": (30,), "l0.mlp.up": (50, 77), "l0.mlp.down": (77, 50), "l0.mlp.act": (2,), "l1.mix.q": (80, 77),
                        "l1.mix.dkv": (23, 77), "l1.mix.dkv.norm": (13,), "l1.mix.uk": (30, 13), "l1.mix.uv": (45, 13), "l1.mix.g": (5, 77),
                        "l1.mix.o": (77, 45)}.items():
        assert tuple(specs[name].shape) == shape, name
    assert not any(n.endswith("norm2") or n.endswith("norm1.b") or ".dq" in n or ".uq" in n or "sink" in n for n in specs)
    # a layer without a feed-forward: a file need not hold (but may hold) a second gate
    assert "l2.mlp.up" not in specs and not specs["l2.rg2"].required and not specs["l2.rg2.b"].required and specs["l2.rg1"].required
    assert specs["l0.rg2"].required and not specs["head"].required


def test_cache_needs():
    m = _model("Q")
    specs = m.cache_specs()
    # rows of latent + rotated part, all positions kept; a matrix per head in 32-bit
    assert specs[0] == KVCacheSpec(1, 24, None, v_head_dim=0) and specs[1] == KVCacheSpec(1, 18, None, v_head_dim=0)
    assert specs[2] == StateSpec((6 * 8 * 8,), torch.float32) and specs[3] == StateSpec((2 * 24 * 40,), torch.float32)
    groups, per_run = plan_groups(specs, m.cache_from())
    assert len(groups) == 3 and per_run[2] is None and per_run[3] is None
    assert m.graph_safe()


@pytest.mark.parametrize("change, message", [
    (lambda d: d["layers"][1].update(type="attention"), "type"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=2), "rot"),
    (lambda d: d["layers"][1]["mixer"].update(rot_dim=3), "rot"),
    (lambda d: d["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][0]["mixer"].update(tau=0.0), "tau"),
    (lambda d: d["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda d: d["layers"][0]["mixer"].update(heads=0), "heads"),
    (lambda d: d["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "mlp.kind"),
    (lambda d: d["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.update(embedding=3), "embedding"),
    (lambda d: d.update(layers=[]), "layers"),
    (lambda d: d.update(width=0), "width"),
])
def test_refusals(change, message):
    d = copy.deepcopy(RAM["P"])
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_what_the_parts_refuse():
    from forge_b200.config import LayerSpec, ModelPlan, PartSpec
    rt = Runtime(torch.device("cpu"), torch.float32)
    from forge_b200.parts import build_block, build_part
    with pytest.raises(ConfigError, match="tau"):
        build_part("mixer", PartSpec("gated_linear", {"hidden_size": 8, "num_heads": 1, "head_dim": 4, "tau": -1.0, "eps": 1e-5}), rt)
    with pytest.raises(ConfigError, match="256"):
        build_part("mixer", PartSpec("gated_linear", {"hidden_size": 8, "num_heads": 1, "head_dim": 257, "tau": 1.0, "eps": 1e-5}), rt)
    plan = ram_config("P").plan()
    first = plan.layers[0]
    with pytest.raises(ConfigError, match="depth"):
        build_block(LayerSpec(block="parallel_depth", mixer=first.mixer, feed_forward=first.feed_forward, norms=first.norms, weight_prefix="",
                              block_params={"depth": 1}), rt)
    fields = dict(plan.__dict__, schedule=[0, 1, 1, 2, 3])
    with pytest.raises(ConfigError, match="depth"):
        Model(ModelPlan(**fields), rt)
    lat = dict(plan.layers[1].mixer.params, out_gate="row")
    with pytest.raises(ConfigError, match="gate"):
        build_part("mixer", PartSpec("latent_attention", lat), rt)


def test_to_dict_round_trip_and_keys_that_are_absent():
    for name in RAM:
        cfg = ram_config(name)
        assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict()["layers"] == RAM[name]["layers"]
    d = copy.deepcopy(RAM["P"])
    d.pop("embedding")
    assert config_from_dict(d).embedding_scale == 1.0
    d["layers"][0].pop("mlp")
    assert config_from_dict(d).plan().layers[0].feed_forward.kind == "none"
    d["max_positions"], d["eos_token_id"] = 500, 7
    assert config_from_dict(config_from_dict(d).to_dict()).max_positions == 500 and config_from_dict(d).eos_token_id == 7


def test_random_weights_fit_the_model():
    for name in RAM:
        t = ram_tensors(name)
        specs = _model(name).tensor_specs()
        assert set(t) == {n for n, s in specs.items() if s.required}
        for i, r in RANKS[name].items():
            assert t[f"l{i}.mix.a1"].shape[0] == t[f"l{i}.mix.a2"].shape[1] == r


# ----------------------------------------------------------------------------------------------- the plain implementation itself

def test_plain_looks_at_nothing_ahead():
    cfg, t = RAM["Q"], ram_tensors("Q")
    toks = torch.randint(0, 118, (40,), generator=torch.Generator().manual_seed(1)).tolist()
    a = PR.forward(cfg, t, toks)
    b = PR.forward(cfg, t, toks[:25])
    assert torch.allclose(a[:25], b, atol=1e-12)
    changed = list(toks)
    changed[30] = (changed[30] + 1) % 118
    c = PR.forward(cfg, t, changed)
    assert torch.allclose(a[:30], c[:30], atol=1e-12) and float((a[30:] - c[30:]).abs().max()) > 1e-3


def test_plain_activation():
    z = torch.linspace(-6, 6, 1201, dtype=torch.float64)
    p, q = torch.tensor(0.3, dtype=torch.float64), torch.tensor(-1.1, dtype=torch.float64)
    y = PR.xielu(z, p, q)
    sp = lambda v: math.log1p(math.exp(v))
    for i in (0, 350, 599, 600, 601, 900, 1200):
        v = float(z[i])
        want = sp(0.3) * v * v + v / 2 if v > 0 else (0.5 + sp(-1.1)) * (math.exp(v) - 1 - v) + v / 2
        assert abs(float(y[i]) - want) < 1e-12
    assert float(PR.xielu(torch.zeros(1, dtype=torch.float64), p, q)) == 0.0


def test_plain_recurrence_in_closed_form_and_carried_over():
    T, N, K, V = 9, 2, 3, 4
    q, k, v = rand(T, N, K, seed=1).double(), rand(T, N, K, seed=2).double(), rand(T, N, V, seed=3).double()
    a = torch.sigmoid(rand(T, N, K, seed=4)).double()
    o, S = PR.gated_recurrence(q, k, v, a)
    for t in range(T):
        want = torch.zeros(N, V, dtype=torch.float64)
        for s in range(t + 1):
            reach = a[s + 1:t + 1].prod(dim=0)                                # what the decays leave of token s, per key channel
            want += (q[t] * k[s] * reach).sum(-1, keepdim=True) * v[s]
        assert torch.allclose(o[t], want, atol=1e-12)
    o1, S1 = PR.gated_recurrence(q[:4], k[:4], v[:4], a[:4])
    o2, S2 = PR.gated_recurrence(q[4:], k[4:], v[4:], a[4:], state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o, atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_plain_decay():
    w = {"a1": rand(3, 5, seed=1).double(), "a2": rand(4, 3, seed=2).double(), "a2.b": rand(4, seed=3).double()}
    h = rand(6, 5, seed=4).double()
    one, many = PR.channel_decay(h, w, 1.0), PR.channel_decay(h, w, 16.0)
    assert torch.allclose(many ** 16, one, atol=1e-12) and bool((many > one).all())
    assert torch.allclose(one, torch.sigmoid(h @ w["a1"].T @ w["a2"].T + w["a2.b"]), atol=1e-12)


def test_plain_rotation():
    x = rand(5, 2, 10, seed=1).double()
    pos = torch.arange(5)
    y = PR.rotate_halves(x, pos, 50.0, 6)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    a = 3 * 50.0 ** (-2.0 / 6)                                              # position 3, pair 1: channels 1 and 4
    assert abs(float(y[3, 1, 1]) - float(x[3, 1, 1] * math.cos(a) - x[3, 1, 4] * math.sin(a))) < 1e-12
    assert abs(float(y[3, 1, 4]) - float(x[3, 1, 4] * math.cos(a) + x[3, 1, 1] * math.sin(a))) < 1e-12
    # scores depend on the distance alone
    same = x[0].expand(5, 2, 10)
    r = PR.rotate_halves(same, pos, 50.0, 10)
    assert abs(float((r[4] * r[2]).sum() - (r[3] * r[1]).sum())) < 1e-10


def test_plain_layer_parts():
    x = rand(7, 12, seed=1, scale=3.0).double() + 5.0
    w = rand(12, seed=2).double()
    n = PR.layer_norm(x, w, 0.0) / w
    assert torch.allclose(n.mean(-1), torch.zeros(7, dtype=torch.float64), atol=1e-12) and torch.allclose((n * n).mean(-1), torch.ones(7, dtype=torch.float64))
    big = PR.layer_norm(x, w, 100.0)
    assert float(big.abs().max()) < float((n * w).abs().max())
    hist = [rand(3, 4, seed=i).double() for i in range(4)]
    c = torch.tensor([0.0, 0.0, 2.0, 1.0], dtype=torch.float64)
    assert torch.allclose(PR.depth_average(hist, c), 2 * hist[2] + hist[3])
    # a layer whose gates are shut passes the stream through; open, it is the ordinary parallel layer
    cfg, t = RAM["S"], {k: torch.as_tensor(v).double() for k, v in ram_tensors("S").items()}
    x = rand(6, 64, seed=9).double()
    h = PR.layer_norm(x, t["l0.norm1"], 1e-4)
    y = PR.mixer("gla", h, PR._sub(t, "l0.mix."), cfg["layers"][0]["mixer"], 1e-4) + PR.feed_forward(h, PR._sub(t, "l0.mlp."))
    for bias, want in ((-1e4, x), (1e4, x + y)):
        for q in (1, 2):
            t[f"l0.rg{q}.b"][:] = bias
        assert torch.allclose(PR.layer(x, t, "l0.", cfg["layers"][0], 1e-4), want, atol=1e-12)
