"""The Ramupel design in the engine against the plain implementation: each mechanism alone, then whole models under every way of
cutting and batching, long decoding, generation through the scheduler, and the trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import schedules
from helpers import TOL, assert_greedy_follows_plain, max_rel_err, random_tokens
from plain import ramupel as PR
from ramupel_models import LENGTHS, RAM, make_ram_dir
from test_engine_gpu import first_bad, run_schedule
from test_zatupel_gpu import CUTS, DEV, DT, DTYPES, PART_TOL, _bf16_weights, _feed, _rt, make_runner
from zatupel_models import rand

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LONG_CUTS = [(0, 64), (64, 130), (130, 131), (131, 133), (133, 150), (150, 152), (152, 230)]


# ----------------------------------------------------------------------------------------------- norm and activation

@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("W", [7, 48, 1030])
def test_layer_norm_without_a_bias(dtype, W):
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    x, w = rand(9, W, seed=W, scale=2.0) + 3.0, (1.0 + rand(W, seed=W + 1, scale=0.3)).to(torch.bfloat16)
    norm = build_part("norm", PartSpec("layernorm", {"size": W, "eps": 1e-2, "names": {"weight": "n"}, "has_bias": False}), _rt(dtype))
    assert set(norm.tensor_specs()) == {"n"}
    norm.bind({"n": w})
    want = PR.layer_norm(x.double(), w.double(), 1e-2)
    assert max_rel_err(norm.forward(x.to(DEV)), want) <= PART_TOL[dtype]
    rows = torch.tensor([8, 0, 3], dtype=torch.int32, device=DEV)
    assert max_rel_err(norm.forward(x.to(DEV), rows=rows), want[[8, 0, 3]]) <= PART_TOL[dtype]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T, W, F", [(1, 64, 40), (3, 24, 72), (7, 77, 50), (40, 128, 512), (130, 64, 96), (300, 256, 640), (100, 72, 2050)])
def test_xielu_feed_forward(dtype, T, W, F):
    """One token, few, many (the products' kernels for each), widths that only the fp32 arithmetic takes, odd numbers of columns."""
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    ff = build_part("feed_forward", PartSpec("dense", {"hidden_size": W, "intermediate_size": F, "activation": "xielu"}), _rt(dtype))
    for p, q in ((0.4, -0.9), (-3.0, 2.0)):
        t = {"mlp.up": rand(F, W, seed=1, scale=0.3).to(torch.bfloat16), "mlp.down": rand(W, F, seed=2, scale=0.2).to(torch.bfloat16),
             "mlp.act": torch.tensor([p, q], dtype=torch.bfloat16)}
        ff.bind(t)
        x = rand(T, W, seed=3).to(dtype)
        want = PR.feed_forward(x.double(), {k[4:]: v.double() for k, v in t.items()})
        assert max_rel_err(ff.forward(x.to(DEV), None), want) <= PART_TOL[dtype]
        r0 = rand(T, W, seed=4)
        res = r0.to(DEV)
        ff.forward(x.to(DEV), res)
        assert max_rel_err(res, r0.double() + want) <= PART_TOL[dtype]


def test_xielu_point_by_point():
    from forge_b200 import kernels
    z = torch.cat([torch.linspace(-30, 30, 2001), torch.tensor([0.0, -0.0, 1e-6, -1e-6, 1e-3, -1e-3, -80.0, 40.0])]).reshape(1, -1)
    p, q = torch.tensor(-0.5, dtype=torch.float64), torch.tensor(1.5, dtype=torch.float64)
    numbers = (float(PR.softplus(p)), 0.5 + float(PR.softplus(q)))
    want = PR.xielu(z.double(), p, q)
    got = kernels.act_rows(z.to(DEV), torch.float32, "xielu", numbers).cpu().double()
    # (the terms below zero have other signs: errors are measured against their sizes)
    size = lambda v: v * v + v.abs() + 1e-7
    assert float(((got - want).abs() / size(z.double())).max()) <= 1e-6
    # the activation in the product's epilogue: the unit matrix as weights
    zb = z[:, ::8].to(torch.bfloat16)
    n = zb.shape[1] // 8 * 8
    x, eye = zb[:, :n].reshape(-1, 8).contiguous(), torch.eye(8, dtype=torch.bfloat16)
    got = kernels.gemm_sm100(x.to(DEV), eye.to(DEV), epilogue="xielu", numbers=numbers).float().cpu().double()
    want = PR.xielu(x.double(), p, q)
    assert float(((got - want).abs() / size(x.double())).max()) <= 6e-3
    with pytest.raises(kernels.KernelError):
        kernels.act_rows(z.to(DEV), torch.float32, "xielu")
    with pytest.raises(kernels.KernelError):
        kernels.act_rows(z.to(DEV), torch.float32, "gelu", numbers)


# ----------------------------------------------------------------------------------------------- the layer's step over the depth

@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("W", [7, 64, 77, 1028, 2050, 4096])
@pytest.mark.parametrize("T", [1, 9, 300])
def test_depth_step(dtype, W, T):
    """Gates, the sum over the planes, the norm that follows: with and without each, on all rows and on chosen ones; planes that the
    weights do not name are not touched."""
    from forge_b200 import kernels
    g = torch.Generator().manual_seed(W + T)
    for n, kind, ff, gated, pad in ((2, "layer", True, True, 0), (3, "rms", False, True, 3), (6, "layer", True, True, 8), (5, "layer", True, False, 0), (0, "rms", True, True, 1)):
        P = max(n, 1) + 3
        planes = torch.randn(P, T, W, generator=g) + 0.5
        y1, y2 = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g)
        z = torch.randn(T, 2 * W + pad, generator=g) * 2.0
        c, w, b = torch.randn(n, generator=g), 1.0 + 0.3 * torch.randn(W, generator=g), torch.randn(W, generator=g)
        x_plane, new_plane, s_plane = (0 if n == 2 else P - 1), (n - 1 if n else P - 2), P - 1
        d = lambda t: t.to(DEV).contiguous()
        pd = planes.double()
        g1, g2 = (torch.sigmoid(z[:, pad:pad + W].double()), torch.sigmoid(z[:, pad + W:].double())) if gated else (1.0, 1.0)
        new = pd[x_plane] + y1.double() * g1 + (y2.double() * g2 if ff else 0.0)
        s = PR.depth_average(list(pd[:n - 1]) + [new], c.double()) if n else new
        bias = b if n == 6 else None
        want = (PR.layer_norm(s, w.double(), 1e-3) if kind == "layer" else PR.rms_norm(s, w.double(), 1e-3)) + (bias.double() if bias is not None else 0.0)
        args = dict(gates=(d(z), pad, pad + W) if gated else None, weights=d(c) if n else None)
        norm = (kind, d(w), None if bias is None else d(bias), 1e-3)
        on = d(planes)
        got = kernels.depth_step(on, n, x_plane, d(y1), d(y2) if ff else None, new_plane=new_plane, s_plane=s_plane, next_norm=norm, out_dtype=dtype, **args)
        assert max_rel_err(got, want) <= PART_TOL[dtype], (n, kind)
        assert max_rel_err(on[new_plane], new) <= 2e-6 and max_rel_err(on[s_plane], s) <= 5e-6
        for j in range(P):
            if j not in (new_plane, s_plane):
                assert torch.equal(on[j].cpu(), planes[j])
        # without a norm; and the norm alone of chosen rows, nothing stored
        on = d(planes)
        assert kernels.depth_step(on, n, x_plane, d(y1), d(y2) if ff else None, new_plane=new_plane, s_plane=s_plane, **args) is None
        assert max_rel_err(on[s_plane], s) <= 5e-6
        on, rows = d(planes), torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
        got = kernels.depth_step(on, n, x_plane, d(y1), d(y2) if ff else None, next_norm=norm, out_dtype=dtype, rows=rows.to(DEV), **args)
        assert max_rel_err(got, want[rows.long()]) <= PART_TOL[dtype] and torch.equal(on.cpu(), planes)


def test_depth_step_refuses_what_does_not_fit():
    from forge_b200 import kernels
    planes, y = torch.zeros(3, 4, 8, device=DEV), torch.zeros(4, 8, device=DEV)
    c = torch.ones(2, device=DEV)
    for bad in (dict(n=3, weights=c), dict(n=2, weights=c, gates=(torch.zeros(4, 15, device=DEV), 0, 8), y2=y), dict(n=2, weights=c, new_plane=3),
                dict(n=2, weights=c, x_plane=3), dict(n=2, weights=None)):
        k = dict(dict(x_plane=0), **bad)
        with pytest.raises(kernels.KernelError):
            kernels.depth_step(planes, k.pop("n"), k.pop("x_plane"), y, k.pop("y2", None), **k)


# ----------------------------------------------------------------------------------------------- gated linear attention

GLA = {
    "odd_sizes": dict(num_heads=3, head_dim=10, v_head_dim=17, tau=4.0, rank=3),
    "one_channel_values": dict(num_heads=2, head_dim=33, v_head_dim=1, tau=0.5, rank=40),
    "tau_one": dict(num_heads=1, head_dim=64, v_head_dim=96, tau=1.0, rank=16),
    "heads_of_128": dict(num_heads=2, head_dim=128, v_head_dim=64, tau=16.0, rank=8),
    "heads_of_160": dict(num_heads=1, head_dim=160, v_head_dim=24, tau=30.0, rank=16),
    "heads_of_256": dict(num_heads=2, head_dim=256, v_head_dim=20, tau=9.0, rank=1),
    "a_state_too_large_for_one_cta": dict(num_heads=1, head_dim=256, v_head_dim=144, tau=12.0, rank=4),
    "many_heads": dict(num_heads=20, head_dim=4, v_head_dim=8, tau=2.0, rank=200),
}


def _gla(dtype, W, o, eps=1e-3):
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    return build_part("mixer", PartSpec("gated_linear", dict(o, hidden_size=W, eps=eps)), _rt(dtype))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", list(GLA))
def test_gated_linear_mixer_alone(dtype, kind):
    """Two requests side by side, fed in portions down to one token; then a third takes over a slot."""
    from forge_b200.cache import CacheStorage
    o = GLA[kind]
    W, T = 40, 62
    mixer = _gla(dtype, W, o)
    t, w = _bf16_weights(mixer, 0.35, seed=len(kind))
    mixer.bind(t)
    storage = CacheStorage([mixer.cache_spec()], [None], 8, 1, 2, dtype, torch.device(DEV))
    x = rand(T, W, seed=50).to(dtype)
    m = {"heads": o["num_heads"], "dim": o["head_dim"], "vdim": o["v_head_dim"], "tau": o["tau"]}
    want = PR.gla(x.double(), w, m, 1e-3)
    got = _feed(mixer, storage, x, CUTS, requests=("a", "b"))
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype], (kind, r)
    storage.manager.free("a")
    got = _feed(mixer, storage, x, [(0, 2), (2, 3), (3, 60), (60, 62)], requests=("c",))
    assert max_rel_err(got["c"], want) <= PART_TOL[dtype], kind


@pytest.mark.parametrize("K, V, r", [(10, 17, 3), (64, 64, 16), (96, 130, 8), (200, 16, 33)])
def test_the_state_is_carried_in_32_bits(K, V, r):
    """The scan alone: outputs and the state it leaves, for requests of unequal length in one step, from a state that is not zero."""
    from types import SimpleNamespace
    from forge_b200 import kernels
    N, lens = 3, [1, 40, 2, 17]
    T = sum(lens)
    q, k, v, u = rand(T, N * K, seed=1), rand(T, N * K, seed=2), rand(T, N * V, seed=3), rand(T, r, seed=4)
    w2, b, tau = rand(N * K, r, seed=5, scale=0.5), rand(N * K, seed=6) + 1.0, 5.0
    state0 = rand(6, N * K * V, seed=7)
    starts = [0, 1, 41, 43, 60]
    slots = [4, 0, 5, 2]
    i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=DEV)
    batch = SimpleNamespace(q_start=i32(starts), slots=i32(slots), num_requests=4)
    state = state0.to(DEV)
    d = lambda z: z.to(DEV).contiguous()
    got = kernels.gla_scan((d(q), 0), (d(k), 0), (d(v), 0), (d(u), 0), r, d(w2.t()), d(b), tau, batch, state, N, K, V).cpu()
    a = torch.sigmoid(u.double() @ w2.double().T + b.double()) ** (1 / tau)
    for s, (lo, hi) in enumerate(zip(starts, starts[1:])):
        n = hi - lo
        o, S = PR.gated_recurrence(q[lo:hi].double().view(n, N, K) * K ** -0.5, k[lo:hi].double().view(n, N, K), v[lo:hi].double().view(n, N, V),
                                   a[lo:hi].view(n, N, K), state=state0[slots[s]].double().view(N, K, V))
        assert max_rel_err(got[lo:hi], o.reshape(n, N * V)) <= 1e-5
        assert max_rel_err(state[slots[s]], S.reshape(-1)) <= 1e-5
    for s in (1, 3):
        assert torch.equal(state[s].cpu(), state0[s])                       # slots that take no part


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("K, V, r", [(10, 17, 3), (64, 64, 16), (96, 132, 8), (5, 2, 1), (20, 1100, 40), (256, 128, 2)])
def test_one_token_of_every_request_in_one_kernel(dtype, K, V, r):
    """The kernel of single-token steps: what it returns (normed, weighted, gated) and the states it leaves; rows of several
    requests, slots in any order, inputs that are columns of a wider matrix, an output slice; states whose rows no vector load fits."""
    from types import SimpleNamespace
    from forge_b200 import kernels
    N, B, pad = 3, 4, 5 if V % 2 else 8
    w2, b, tau, nw = rand(N * K, r, seed=5, scale=0.5), rand(N * K, seed=6) + 1.0, 5.0, 1.0 + rand(V, seed=8, scale=0.3)
    p = rand(B, pad + 2 * N * (K + V) + r, seed=1)
    cut = [pad, pad + N * K, pad + 2 * N * K, pad + 2 * N * K + N * V, pad + 2 * N * K + 2 * N * V]
    q, k, v, g, u = (p[:, c:c + n].double() for c, n in zip(cut, (N * K, N * K, N * V, N * V, r)))
    state0 = rand(6, N * K * V, seed=7)
    slots, i32 = [4, 0, 5, 2], lambda z: torch.tensor(z, dtype=torch.int32, device=DEV)
    batch = SimpleNamespace(q_start=i32([0, 1, 2, 3, 4]), slots=i32(slots), num_requests=B, num_tokens=B)
    assert kernels.gla_token_supports(batch, N, K, V, r)
    d, state = lambda z: z.to(DEV).contiguous(), state0.to(DEV)
    pd = d(p)
    out = torch.full((B, N * V + 7), 3.0, dtype=dtype, device=DEV)
    kernels.gla_token(*[(pd, c) for c in cut], r, d(w2.t()), d(b), tau, batch, state, N, K, V, d(nw), 1e-3, dtype, out=(out, 2))
    a = (torch.sigmoid(u @ w2.double().T + b.double()) ** (1 / tau)).view(B, N, K)
    for s in range(B):
        o, S = PR.gated_recurrence(q[s:s + 1].view(1, N, K) * K ** -0.5, k[s:s + 1].view(1, N, K), v[s:s + 1].view(1, N, V), a[s:s + 1],
                                   state=state0[slots[s]].double().view(N, K, V))
        want = PR.rms_norm(o, nw.double(), 1e-3).reshape(-1) * g[s] * torch.sigmoid(g[s])
        assert max_rel_err(out[s, 2:2 + N * V], want) <= PART_TOL[dtype]
        assert max_rel_err(state[slots[s]], S.reshape(-1)) <= 1e-5
    for s in (1, 3):
        assert torch.equal(state[s].cpu(), state0[s])
    assert bool((out[:, :2] == 3.0).all()) and bool((out[:, 2 + N * V:] == 3.0).all())
    # portions, and heads too large for one CTA, take the scan
    batch.num_tokens = B + 1
    assert not kernels.gla_token_supports(batch, N, K, V, r)
    batch.num_tokens = B
    assert not kernels.gla_token_supports(batch, N, 256, 512, r)


@pytest.mark.parametrize("dtype", DT)
def test_one_key_is_still_there_hundreds_of_tokens_on(dtype):
    """Decays next to one in one key channel and next to zero in another: what the first token wrote is read hundreds of tokens later
    through the first channel and gone through the second, whatever the cut."""
    from forge_b200.cache import CacheStorage
    W, T = 8, 400
    o = dict(num_heads=1, head_dim=4, v_head_dim=2, tau=2.0, rank=1)
    mixer = _gla(dtype, W, o, eps=1e-12)
    t = {n: torch.zeros([1 if d == -1 else d for d in s.shape], dtype=torch.bfloat16) for n, s in mixer.tensor_specs().items()}
    t["mix.q"][0, 0] = 1.0                  # the last token asks through key channel 0 (input 0) or 1 (input 1)
    t["mix.q"][1, 1] = 1.0
    t["mix.k"][0, 2] = 1.0                  # the first token writes through both (input 2)
    t["mix.k"][1, 2] = 1.0
    t["mix.v"][0, 3] = 1.0                  # values (3, 4): input 3 and 4
    t["mix.v"][1, 4] = 1.0
    t["mix.g"][:, 5] = 1.0
    t["mix.a2.b"][0], t["mix.a2.b"][1] = 30.0, -8.0
    t["mix.norm"][:] = 1.0
    t["mix.o"][0, 0] = t["mix.o"][1, 1] = 1.0
    mixer.bind(t)
    w = {n.split("mix.", 1)[-1]: v.double() for n, v in t.items()}
    for ask in (0, 1):
        x = torch.zeros(T, W)
        x[0, 2], x[0, 3], x[0, 4] = 1.0, 3.0, 4.0
        x[:, 5] = 4.0
        x[1:, ask] = 1.0
        for cuts in ([(0, T)], [(0, 390)] + [(i, i + 1) for i in range(390, T)], [(0, 2), (2, 4), (4, 131), (131, 133), (133, T)]):
            storage = CacheStorage([mixer.cache_spec()], [None], 8, 1, 1, dtype, torch.device(DEV))
            got = _feed(mixer, storage, x.to(dtype), cuts)["r"]
            want = PR.gla(x.to(dtype).double(), w, {"heads": 1, "dim": 4, "vdim": 2, "tau": 2.0}, 1e-12)
            assert max_rel_err(got, want) <= PART_TOL[dtype]
            gate = 4.0 * torch.sigmoid(torch.tensor(4.0))
            far = got[-1, :2] / gate
            if ask == 0:
                assert torch.allclose(far, torch.tensor([0.6, 0.8]) * 2 ** 0.5, atol=2e-2)       # (3, 4) divided by its root mean square
            else:
                assert float(far.abs().max()) < 1e-3


# ----------------------------------------------------------------------------------------------- latent attention

LATENT = {
    "all_sizes_differ": dict(num_heads=3, head_dim=8, rot_dim=4, v_head_dim=12, kv_rank=20, scale=0.4, theta=50.0),
    "one_head": dict(num_heads=1, head_dim=16, rot_dim=8, v_head_dim=8, kv_rank=40, scale=0.25, theta=1e4),
    "rotated_part_wider": dict(num_heads=5, head_dim=6, rot_dim=10, v_head_dim=20, kv_rank=12, scale=0.35, theta=77.0),
    # sizes of the tensor-core kernel (latent and rotated part multiples of 16), in portions that cross its tiles of 64 rows
    "tc": dict(num_heads=4, head_dim=32, rot_dim=16, v_head_dim=48, kv_rank=96, scale=0.15, theta=250000.0, tokens=230, cuts=LONG_CUTS),
    "tc_many_heads": dict(num_heads=12, head_dim=16, rot_dim=16, v_head_dim=24, kv_rank=64, scale=0.2, theta=2e5, tokens=230, cuts=LONG_CUTS),
    "tc_two_value_chunks": dict(num_heads=6, head_dim=20, rot_dim=32, v_head_dim=24, kv_rank=416, scale=0.2, theta=5e3, tokens=230, cuts=LONG_CUTS),
}


def _latent(dtype, W, o, eps=1e-4, **more):
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    o = {k: v for k, v in o.items() if k not in ("tokens", "cuts")}
    theta = o.pop("theta")
    return build_part("mixer", PartSpec("latent_attention", {**o, "hidden_size": W, "q_rank": None, "eps": eps, "out_gate": "head", "position": PartSpec(
        "rope_halves", {"head_dim": o["rot_dim"], "rotary_dims": o["rot_dim"], "theta": theta}), **more}), _rt(dtype))


def _sizes(o):
    return {"heads": o["num_heads"], "dim": o["head_dim"], "rot_dim": o["rot_dim"], "vdim": o["v_head_dim"], "kv_rank": o["kv_rank"],
            "scale": o["scale"], "rot": {"dims": o["rot_dim"], "base": o["theta"]}}


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", list(LATENT))
def test_latent_attention_alone(dtype, kind):
    from forge_b200.cache import CacheStorage
    o = LATENT[kind]
    W, T, cuts = 40, o.get("tokens", 62), o.get("cuts", CUTS)
    mixer = _latent(dtype, W, o)
    t, w = _bf16_weights(mixer, 0.35, seed=len(kind))
    mixer.bind(t)
    storage = CacheStorage([mixer.cache_spec()], [None], 8, 2 * -(-T // 8), 2, dtype, torch.device(DEV))
    x = rand(T, W, seed=50).to(dtype)
    got = _feed(mixer, storage, x, cuts, requests=("a", "b"))
    want = PR.latent_attention(x.double(), w, _sizes(o), 1e-4)
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype], (kind, r)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["all_sizes_differ", "tc"])
def test_the_options_of_the_latent_attention_are_independent(dtype, kind):
    """A gate per head equals the gate per channel whose rows repeat the head's; a shut head falls silent and the others do not;
    without a gate nothing is multiplied; rotating halves equals rotating neighbours of permuted channels; the input product's
    columns may lie anywhere in a wider matrix and the heads' outputs in a slice of one."""
    from forge_b200 import kernels
    from forge_b200.cache import CacheStorage
    from forge_b200.config import PartSpec
    from forge_b200.engine import StepEntry, build_step_batch
    o = LATENT[kind]
    W, T, H, D, R, E = 40, 62, o["num_heads"], o["head_dim"], o["rot_dim"], o["v_head_dim"]
    x = rand(T, W, seed=50)
    x[:, 0] = 1.0
    x = x.to(dtype)
    base = _latent(dtype, W, o)
    t, w = _bf16_weights(base, 0.35, seed=3)

    def run(mixer, tensors, cuts=CUTS):
        mixer.bind(tensors)
        storage = CacheStorage([mixer.cache_spec()], [None], 8, -(-T // 8), 1, dtype, torch.device(DEV))
        return _feed(mixer, storage, x, cuts)["r"]
    ref = run(base, t)
    assert max_rel_err(ref, PR.latent_attention(x.double(), w, _sizes(o), 1e-4)) <= PART_TOL[dtype]
    per_channel = dict(t, **{"mix.g": t["mix.g"].repeat_interleave(E, dim=0)})
    assert max_rel_err(run(_latent(dtype, W, o, out_gate="channel"), per_channel), ref) <= PART_TOL[dtype] / 2
    no_gate = {k: v for k, v in t.items() if k != "mix.g"}
    ungated = run(_latent(dtype, W, o, out_gate=False), no_gate)
    open_gate = {k: v.clone() for k, v in t.items()}
    open_gate["mix.g"].zero_()
    open_gate["mix.g"][:, 0] = 60.0
    assert max_rel_err(run(_latent(dtype, W, o), open_gate), ungated) <= PART_TOL[dtype] / 2
    shut = {k: v.clone() for k, v in open_gate.items()}
    shut["mix.g"][0, 0] = -200.0
    silent = {k: v.clone() for k, v in no_gate.items()}
    silent["mix.o"][:, :E] = 0.0
    assert max_rel_err(run(_latent(dtype, W, o), shut), run(_latent(dtype, W, o, out_gate=False), silent)) <= PART_TOL[dtype] / 2
    # channel i of the halves is channel 2i of the neighbours, i + R/2 is 2i + 1
    perm = torch.arange(R).view(2, R // 2).t().reshape(-1)
    moved = {k: v.clone() for k, v in t.items()}
    q = moved["mix.q"].view(H, D + R, W)
    q[:, D:] = q[:, D:][:, perm].clone()
    moved["mix.dkv"][o["kv_rank"]:] = t["mix.dkv"][o["kv_rank"]:][perm]
    pairs = PartSpec("rope_pairs", {"head_dim": R, "rotary_dims": R, "theta": o["theta"]})
    assert max_rel_err(run(_latent(dtype, W, o, position=pairs), moved), ref) <= PART_TOL[dtype] / 2
    # the same from columns of a wider matrix, into columns of one
    base.bind(t)
    storage = CacheStorage([base.cache_spec()], [None], 8, -(-T // 8), 1, dtype, torch.device(DEV))
    storage.manager.admit("s")
    batch = build_step_batch([StepEntry("s", [0] * T, [])], storage.manager, torch.device(DEV), 64)
    p = base.proj.forward(x.to(DEV))
    wide = torch.full((T, base.in_width() + 13), 7.0, device=DEV)
    wide[:, 5:5 + base.in_width()] = p
    out = torch.full((T, base.out_width() + 9), 3.0, device=DEV, dtype=dtype)
    base.mix(wide, 5, batch, storage.layers[0], out=(out, 4))
    assert torch.equal(out[:, :4].cpu(), torch.full((T, 4), 3.0, dtype=dtype)) and torch.equal(out[:, 4 + base.out_width():].cpu(), torch.full((T, 5), 3.0, dtype=dtype))
    y = base.o.forward(out[:, 4:4 + base.out_width()].contiguous())
    assert max_rel_err(y, PR.latent_attention(x.double(), w, _sizes(o), 1e-4)) <= PART_TOL[dtype]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("page_size", [8, 64])
@pytest.mark.parametrize("D, R, C, H", [(6, 4, 8, 2), (16, 16, 32, 2)])
def test_one_token_that_stands_out(dtype, page_size, D, R, C, H):
    """All tokens look alike except one whose score is huge for head 0; values carry a mark of the token.  Head 0 returns the marked
    token's value wherever it lies: at the start, far back, at a page's border, just before or ahead of the token, the token itself;
    for the tokens of a portion and for tokens that come alone; on pages that the case before gave back.  (16, 16, 32) is a shape
    that the tensor-core kernel takes in bfloat16."""
    from forge_b200.cache import CacheStorage
    from forge_b200.engine import StepEntry, build_step_batch
    W, E, N, P = 16, 4, 290, 27
    dev = torch.device(DEV)
    o = dict(num_heads=H, head_dim=D, rot_dim=R, v_head_dim=E, kv_rank=C, scale=1.0, theta=1e4)
    mixer = _latent(dtype, W, o, eps=1e-6)
    t = {n: torch.zeros(s.shape, dtype=torch.bfloat16) for n, s in mixer.tensor_specs().items()}
    t["mix.dkv.norm"][:] = 1.0
    t["mix.q"][0, 1] = 16.0             # head 0's unrotated channel 0 asks whenever input 1 is set
    t["mix.dkv"][0, 0] = 1.0            # latent channel 0: input 0, set for the star alone
    t["mix.dkv"][1, 2] = 1.0            # latent channel 1: input 2, set for all others
    t["mix.uk"][0, 0] = 4.0             # head 0's key channel 0 = latent channel 0
    for h in range(H):
        t["mix.uv"][h * E, 0] = 1.0     # value channel 0 = latent channel 0
        t["mix.o"][h, h * E] = 1.0
    t["mix.g"][:, 1] = 40.0             # open gates
    mixer.bind(t)
    storage = CacheStorage([mixer.cache_spec()], [None], page_size, -(-(N + P + 2) // page_size), 1, dtype, dev)
    total, star_value = N + P + 2, C ** 0.5                                  # a latent with one channel set, divided by its root mean square
    for case, star in enumerate([0, 1, 63, 64, 150, 255, 256, N - 1, N, N + 5, N + P - 1, N + P, N + P + 1]):
        rid = f"r{case}"
        storage.manager.admit(rid)
        x = torch.zeros(total, W)
        x[:, 1] = 1.0
        x[:, 2] = 1.0
        x[star, 0], x[star, 2] = 1.0, 0.0
        done = 0
        for n in (N, P, 1, 1):
            batch = build_step_batch([StepEntry(rid, [0] * n, [])], storage.manager, dev, 64)
            out = mixer.forward(x[done:done + n].to(DEV).to(dtype).contiguous(), batch, storage.layers[0], None).cpu()
            for i in range(n):
                pos = done + i
                want0 = star_value if star <= pos else 0.0
                mean = star_value / (pos + 1) if star <= pos else 0.0
                assert abs(float(out[i, 0]) - want0) <= 2e-2 * star_value, (star, pos, out[i, :2].tolist())
                assert abs(float(out[i, 1]) - mean) <= 2e-2 * max(mean, 0.05), (star, pos, out[i, :2].tolist(), mean)
            done += n
        storage.manager.free(rid)                                            # the next case takes over these pages
        storage.manager.check()


def test_mixers_of_this_design_side_by_side():
    """Both mixers offer their two products, so they may share one of each with other mixers of a layer."""
    from forge_b200.cache import CacheStorage
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    W, T = 40, 62
    lat = dict(LATENT["all_sizes_differ"])
    theta = lat.pop("theta")
    specs = [PartSpec("latent_attention", {**lat, "hidden_size": W, "q_rank": None, "eps": 1e-4, "out_gate": "head", "prefix": "mix.a.", "position": PartSpec(
                 "rope_halves", {"head_dim": 4, "rotary_dims": 4, "theta": theta})}),
             PartSpec("gated_linear", {"hidden_size": W, "num_heads": 2, "head_dim": 12, "v_head_dim": 16, "tau": 3.0, "eps": 1e-4, "rank": 5, "prefix": "mix.b."})]
    mixer = build_part("mixer", PartSpec("side_by_side", {"mixers": specs}), _rt(torch.float32))
    t, w = _bf16_weights(mixer, 0.35, seed=8)
    mixer.bind(t)
    assert mixer.proj is not None
    storage = CacheStorage([mixer.cache_spec()], [None], 8, -(-T // 8), 1, torch.float32, torch.device(DEV))
    x = rand(T, W, seed=50)
    got = _feed(mixer, storage, x, CUTS)["r"]
    want = PR.latent_attention(x.double(), PR._sub(w, "a."), _sizes(dict(lat, theta=theta)), 1e-4) + \
        PR.gla(x.double(), PR._sub(w, "b."), {"heads": 2, "dim": 12, "vdim": 16, "tau": 3.0}, 1e-4)
    assert max_rel_err(got, want) <= PART_TOL[torch.float32]


# ----------------------------------------------------------------------------------------------- whole models

class _Plain:
    def __init__(self, d):
        self.cfg, self.tensors = PR.load(d)

    def forward(self, toks, layers_out=None):
        return PR.forward(self.cfg, self.tensors, list(toks), layers_out=layers_out)


@pytest.fixture(scope="module", params=list(RAM))
def ram(request, tmp_path_factory):
    name = request.param
    d = make_ram_dir(tmp_path_factory, name)
    plain = _Plain(d)
    reqs = {f"r{i}": random_tokens(n, RAM[name]["vocab"], seed=10 * i + ord(name)) for i, n in enumerate(LENGTHS[name])}
    return name, d, plain, reqs, {rid: plain.forward(toks).float() for rid, toks in reqs.items()}


def test_layer_by_layer(ram):
    """The stream after every layer, in 32-bit, for a prompt in two portions."""
    name, d, plain, reqs, want = ram
    from forge_b200.engine import StepEntry
    runner = make_runner(d, "float32", 256)
    n = len(runner.model.blocks)
    seen = {i: [] for i in range(n)}
    for i, b in enumerate(runner.model.blocks):
        def wrap(orig, i):
            def f(residual, batch, cache):
                # without a norm to hand over to, the last layer leaves its stream too
                batch.shared["last_norm"] = None
                orig(residual, batch, cache)
                seen[i].append(residual[-1].clone())
            return f
        b.forward = wrap(b.forward, i)
    toks = reqs["r2"]
    runner.admit("x")
    got = [runner.step([StepEntry("x", part, list(range(len(part))))]) for part in (toks[:9], toks[9:])]
    ref = []
    logits = plain.forward(toks, layers_out=ref)
    assert len(ref) == n
    for i in range(n):
        assert max_rel_err(torch.cat(seen[i]), ref[i]) <= 2e-5, f"layer {i}"
    assert max_rel_err(torch.cat(got), logits) <= TOL["float32"]


def test_weights_of_a_gate_that_is_not_there_are_let_pass(tmp_path_factory):
    from forge_b200.engine import ModelRunner, StepEntry
    from ramupel_models import ram_config, ram_tensors
    cfg, tensors = ram_config("Q"), ram_tensors("Q")
    assert "l0.rg2" not in tensors
    more = dict(tensors, **{"l0.rg2": torch.ones(48, 48, dtype=torch.bfloat16), "l0.rg2.b": torch.ones(48, dtype=torch.bfloat16)})
    toks = random_tokens(40, 118, seed=5)
    outs = []
    for t in (tensors, more):
        runner = ModelRunner(config=cfg, tensors=t, dtype="float32", page_size=8, cache_tokens=64, max_requests=1)
        runner.admit("x")
        outs.append(runner.step([StepEntry("x", toks, list(range(40)))]).cpu())
    assert torch.equal(outs[0], outs[1])


def test_a_hidden_layer_of_two_sizes_is_refused():
    from forge_b200.engine import ModelRunner
    from forge_b200.weights.loader import WeightError
    from ramupel_models import ram_config, ram_tensors
    t = ram_tensors("S")
    t["l0.mix.a1"] = torch.zeros(3, 64, dtype=torch.bfloat16)
    with pytest.raises(WeightError, match="a1"):
        ModelRunner(config=ram_config("S"), tensors=t, dtype="float32", page_size=8, cache_tokens=64, max_requests=1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("schedule", ["whole", "last_one_by_one", "changing_portions", "mixed"])
def test_schedules_equal_plain(ram, dtype, schedule):
    name, d, plain, reqs, want = ram
    steps = getattr(schedules, schedule)(reqs)
    # exactly as many pages as the schedule's peak needs: freed pages and slots are taken again at once
    runner = make_runner(d, dtype, schedules.peak_tokens(reqs, steps, round_to=8))
    got = run_schedule(runner, reqs, steps)
    msg = first_bad(got, want, TOL[dtype])
    assert msg is None, msg
    assert runner.manager.num_free_pages() == {g: runner.num_pages for g in runner.manager.groups}


@pytest.mark.parametrize("dtype", DTYPES)
def test_rows_that_are_wanted_and_steps_that_want_nothing(ram, dtype):
    """The last layer works on the wanted rows alone, and in a step that wants none only its cache is written."""
    name, d, plain, reqs, want = ram
    from forge_b200.engine import StepEntry
    runner = make_runner(d, dtype, 512)
    a, b = reqs["r0"], reqs["r1"]
    runner.admit("a")
    runner.admit("b")
    assert runner.step([StepEntry("a", a[:20], []), StepEntry("b", b[:7], [])]) is None
    got = runner.step([StepEntry("a", a[20:31], [10, 0]), StepEntry("b", b[7:9], [])]).cpu()
    assert max_rel_err(got, want["r0"][[30, 20]]) <= TOL[dtype]
    got = runner.step([StepEntry("b", b[9:30], [3, 4, 20]), StepEntry("a", a[31:32], [0])]).cpu()
    assert max_rel_err(got, torch.stack([want["r1"][i] for i in (12, 13, 29)] + [want["r0"][31]])) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_page_size_and_graphs_do_not_matter(ram, dtype):
    name, d, plain, reqs, want = ram
    small = {k: reqs[k] for k in list(reqs)[:3]}
    for ps, graphs in ((16, True), (64, True), (8, False)):
        steps = schedules.mixed(small, max_live=2)
        runner = make_runner(d, dtype, schedules.peak_tokens(small, steps, round_to=ps), page_size=ps, cuda_graphs=graphs)
        got = run_schedule(runner, small, steps)
        msg = first_bad(got, {k: want[k] for k in small}, TOL[dtype])
        assert msg is None, f"page size {ps}: {msg}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_first_tokens(ram, dtype):
    """Two tokens, then hundreds one by one (graph replays)."""
    name, d, plain, reqs, want = ram
    n = {"P": 230, "Q": 300, "R": 200, "S": 120}[name]
    toks = random_tokens(n, RAM[name]["vocab"], seed=77)
    ref = plain.forward(toks).float()
    runner = make_runner(d, dtype, -(-n // 8) * 8)
    assert runner.cuda_graphs
    steps = [([("x", 0, 2)], [])] + [([("x", p, 1)], []) for p in range(2, n)]
    got = run_schedule(runner, {"x": toks}, steps)
    msg = first_bad(got, {"x": ref}, TOL[dtype])
    assert msg is None, msg


def test_a_batch_equals_each_request_alone(ram):
    """Unequal requests in one step against each of them alone, in 32-bit, portion by portion."""
    name, d, plain, reqs, want = ram
    from forge_b200.engine import StepEntry
    small = {k: reqs[k] for k in list(reqs)[:4]}
    cuts = {"r0": [5, 1, 20, 2], "r1": [1, 30, 1, 1], "r2": [2, 2, 9, 3], "r3": [17, 1, 1, 11]}

    def run(ids):
        runner = make_runner(d, "float32", 512, cuda_graphs=False)
        got = {r: [] for r in ids}
        at = {r: 0 for r in ids}
        for r in ids:
            runner.admit(r)
        for k in range(4):
            entries = [StepEntry(r, small[r][at[r]:at[r] + cuts[r][k]], list(range(cuts[r][k]))) for r in ids]
            rows = runner.step(entries).cpu()
            for r in ids:
                got[r].append(rows[:cuts[r][k]])
                rows = rows[cuts[r][k]:]
                at[r] += cuts[r][k]
        return {r: torch.cat(v) for r, v in got.items()}
    together = run(list(small))
    for r in small:
        alone = run([r])[r]
        assert float((together[r] - alone).abs().max()) <= 2e-5 * float(alone.abs().max()), r


def test_fp32_logits_do_not_depend_on_the_cut(ram):
    """In 32-bit every sum is taken in an order that the position alone decides: the four schedules agree to rounding."""
    name, d, plain, reqs, want = ram
    small = {k: reqs[k] for k in list(reqs)[:3]}
    outs = []
    for schedule in ("whole", "last_one_by_one", "changing_portions", "mixed"):
        steps = getattr(schedules, schedule)(small)
        runner = make_runner(d, "float32", schedules.peak_tokens(small, steps, round_to=8), cuda_graphs=False)
        outs.append(run_schedule(runner, small, steps))
    for o in outs[1:]:
        for rid in small:
            assert float((o[rid] - outs[0][rid]).abs().max()) <= 2e-5 * float(outs[0][rid].abs().max()), rid


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_through_the_scheduler(ram, dtype):
    """Greedy generation through forge.Model and through RequestScheduler with more requests than slots and few pages."""
    import forge_b200 as forge
    name, d, plain, reqs, want = ram
    model = forge.Model(d, dtype=dtype, block_size=8, max_num_seqs=2, cache_tokens=512, max_tokens_per_step=48)
    prompt = reqs["r1"][:30]
    out = model.generate(prompt, max_new_tokens=12, do_sample=False)
    assert out["num_generated_tokens"] == 12 and out["finish_reason"] == "length"
    logits_fn = lambda ids: plain.forward(ids).float()
    assert len(set(out["token_ids"])) >= 4                                   # a text that repeats one token would show little
    assert_greedy_follows_plain(logits_fn, prompt, out["token_ids"], TOL[dtype], what="generate")
    sched = forge.RequestScheduler(model, max_num_seqs=2, max_tokens_per_step=48)
    prompts = [reqs["r0"][:50], reqs["r2"][:9], reqs["r3"][:31], reqs["r1"][:3]]
    ids = [sched.submit(p, 8, -1, forge.SamplerConfig(do_sample=False)) for p in prompts]
    done = {r.request_id: r for r in sched.run()}
    for rid, p in zip(ids, prompts):
        assert done[rid].num_generated == 8
        assert_greedy_follows_plain(logits_fn, p, list(done[rid].output_tokens), TOL[dtype], what=f"request {rid}")
    model.runner.manager.check()
    model.runner.check_status()


def test_trace_replay_as_a_subprocess(ram, tmp_path):
    name, d, plain, reqs, want = ram
    small = {k: reqs[k] for k in list(reqs)[:3]}
    steps = schedules.mixed(small, max_live=2)
    lines, asked = [], {}
    for n, (entries, end) in enumerate(steps):
        es = []
        for rid, p, cnt in entries:
            w = [cnt - 1] if (p + cnt) % 3 == 0 or p + cnt == len(small[rid]) else []
            es.append({"id": rid, "tokens": small[rid][p:p + cnt], "want": w})
            if w:
                asked.setdefault(n, []).extend((rid, p + i) for i in w)
        lines.append(json.dumps({"step": n, "entries": es, "end": end}))
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", str(schedules.peak_tokens(small, steps, round_to=64))], input="\n".join(lines) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(steps))]
    V = RAM[name]["vocab"]
    for n, rows in asked.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), V))
        ref = torch.stack([want[rid][pos] for rid, pos in rows])
        assert max_rel_err(got, ref) <= TOL["float32"], n
    assert sorted(os.listdir(out)) == sorted(f"{n}.f32" for n in asked)


def test_command_line(ram):
    """bin/forge-cli on a Ramupel folder: greedy tokens in 32-bit follow the plain implementation; sampling runs."""
    name, d, plain, reqs, want = ram
    prompt = reqs["r1"][:6]
    cli = [sys.executable, os.path.join(ROOT, "bin", "forge-cli"), "-m", d, "-p", " ".join(map(str, prompt)), "-n", "5", "--no-stream",
           "--page-size", "8", "--kv-pages", "2"]
    proc = subprocess.run(cli + ["--temp", "0", "--repeat-penalty", "1.0", "--dtype", "float32"], capture_output=True, text=True, timeout=300)
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = [int(t) for t in proc.stdout.strip().splitlines()[0].split()]
    assert len(got) == 5 and "6 prompt" in proc.stdout and "5 generated" in proc.stdout
    assert_greedy_follows_plain(lambda ids: plain.forward(ids).float(), prompt, got, TOL["float32"], what="forge-cli")
    proc = subprocess.run(cli + ["--temp", "0.8", "--top-k", "20", "--seed", "3", "--dtype", "bfloat16"], capture_output=True, text=True, timeout=300)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert len(proc.stdout.strip().splitlines()[0].split()) == 5
