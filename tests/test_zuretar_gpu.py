"""The Zuretar design in the engine against the plain implementation: each mechanism alone, then whole models under every way of
cutting and batching, long decoding, generation through the scheduler, and the trace replay."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import schedules
from helpers import TOL, assert_greedy_follows_plain, max_rel_err, random_tokens
from plain import zuretar as PZ
from test_engine_gpu import run_schedule
from test_natalorn_gpu import LONG_CUTS, _Adds, _engine_choices, _first_bad
from test_zatupel_gpu import CUTS, DEV, DT, DTYPES, PART_TOL, _bf16_weights, _feed, _rt, make_runner
from zatupel_models import rand
from zuretar_models import LENGTHS, ZUR, make_zur_dir, zur_config, zur_tensors

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _part(category, kind, dtype, **params):
    from forge_b200.config import PartSpec
    from forge_b200.parts import build_part
    return build_part(category, PartSpec(kind, params), _rt(dtype))


def _i32(z):
    return torch.tensor(z, dtype=torch.int32, device=DEV)


def _storage(mixer, dtype, pages, requests, page_size=8):
    from forge_b200.cache import CacheStorage
    return CacheStorage([mixer.cache_spec()], [None], page_size, pages, requests, dtype, torch.device(DEV))


# ----------------------------------------------------------------------------------------------- outputs that join the stream

@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("W, T", [(1, 3), (7, 5), (48, 9), (256, 150), (1030, 4), (4096, 3), (9000, 2)])
def test_join(dtype, W, T):
    from forge_b200 import kernels
    ys = [rand(T, W, seed=i, scale=0.5 + i) for i in range(4)]
    ws = [1.0 + rand(W, seed=10 + i, scale=0.3) for i in range(4)]
    x0, wn = rand(T, W, seed=20), 1.0 + rand(W, seed=21, scale=0.3)
    d = lambda z: None if z is None else z.to(DEV)
    for normed, scales in ([True], [0.7]), ([False], [1.0]), ([True, True], [0.5, 0.5]), ([True, True, False], [0.5, 0.25, 1.0]), \
            ([False, True, False, True], [2.0, -1.0, 0.3, 1.0]):
        terms = [(ys[i], ws[i] if n else None, s) for i, (n, s) in enumerate(zip(normed, scales))]
        want = x0.double() + sum(s * (PZ.rms(y.double(), 1e-2) * w.double() if w is not None else y.double()) for y, w, s in terms)
        for follows in (False, True):
            x = x0.to(DEV)
            got = kernels.join(x, [(d(y), d(w), s) for y, w, s in terms], 1e-2, next_norm=(d(wn), 1e-3) if follows else None, out_dtype=dtype)
            assert max_rel_err(x, want) <= 2e-6
            assert (got is None) == (not follows)
            if follows:
                assert max_rel_err(got, PZ.rms(want, 1e-3) * wn.double()) <= PART_TOL[dtype]
    with pytest.raises(kernels.KernelError):
        kernels.join(x0.to(DEV), [], 1e-2)
    with pytest.raises(kernels.KernelError):
        kernels.join(x0.to(DEV), [(torch.zeros(T + 1, W, device=DEV), None, 1.0)], 1e-2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("n, T, col", [(5, 3, 1), (48, 200, 4), (1200, 2, 0), (6000, 1, 8)])
def test_heads_normed_together(dtype, n, T, col):
    from forge_b200 import kernels
    o, w, g = rand(T, n, seed=1, scale=3.0), 1.0 + rand(n, seed=2, scale=0.3), rand(T, n + col + 3, seed=3)
    got = kernels.gated_rows(o.to(DEV), w.to(DEV), (g.to(DEV), col), 1e-2, dtype)
    want = PZ.rms(o.double(), 1e-2) * w.double() * torch.sigmoid(g[:, col:col + n].double())
    assert max_rel_err(got, want) <= PART_TOL[dtype]


# ----------------------------------------------------------------------------------------------- gated delta rule

DELTA = {
    "odd_sizes_three_heads_a_key": dict(num_heads=6, num_qk_heads=2, head_dim=10, v_head_dim=17, taps=3),
    "no_convolution": dict(num_heads=2, num_qk_heads=2, head_dim=33, v_head_dim=1, taps=1),
    "two_taps": dict(num_heads=4, num_qk_heads=1, head_dim=16, v_head_dim=8, taps=2),
    "seven_taps_keys_of_odd_size": dict(num_heads=3, num_qk_heads=3, head_dim=5, v_head_dim=12, taps=7),
    "heads_of_128": dict(num_heads=2, num_qk_heads=1, head_dim=128, v_head_dim=128, taps=4),
    "heads_of_160": dict(num_heads=1, num_qk_heads=1, head_dim=160, v_head_dim=24, taps=4),
    "heads_of_256": dict(num_heads=2, num_qk_heads=2, head_dim=256, v_head_dim=20, taps=2),
    "wide_values": dict(num_heads=1, num_qk_heads=1, head_dim=8, v_head_dim=1200, taps=4),
    "values_too_wide_for_one_cta": dict(num_heads=1, num_qk_heads=1, head_dim=4, v_head_dim=610 * 2 - 1, taps=4),
    "many_heads": dict(num_heads=24, num_qk_heads=8, head_dim=4, v_head_dim=8, taps=4),
}


def _delta_sizes(o):
    return {"heads": o["num_heads"], "kv_heads": o["num_qk_heads"], "dim": o["head_dim"], "vdim": o["v_head_dim"], "conv": o["taps"]}


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", list(DELTA))
def test_gated_delta_mixer_alone(dtype, kind):
    """Two requests side by side, fed in portions down to one token; then a third takes over a slot."""
    o = DELTA[kind]
    W, T = 40, 62
    mixer = _part("mixer", "gated_delta", dtype, hidden_size=W, eps=1e-3, **o)
    t, _ = _bf16_weights(mixer, 0.35, seed=len(kind))
    t["mix.A_log"][::2] -= 4.0                                               # every other head forgets slowly
    w = {n.split("mix.", 1)[-1]: v.double() for n, v in t.items()}
    mixer.bind(t)
    storage = _storage(mixer, dtype, 1, 2)
    x = rand(T, W, seed=50).to(dtype)
    want = PZ.delta_mixer(x.double(), w, _delta_sizes(o), 1e-3)
    got = _feed(mixer, storage, x, CUTS, requests=("a", "b"))
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype], (kind, r)
    storage.manager.free("a")
    for cuts in ([(0, 2), (2, 3), (3, 60), (60, 62)], [(i, i + 1) for i in range(20)] + [(20, 22), (22, 24), (24, 62)]):
        got = _feed(mixer, storage, x, cuts, requests=("c",))
        assert max_rel_err(got["c"], want) <= PART_TOL[dtype], kind
        storage.manager.free("c")
    assert storage.check_canaries() == []


def _delta_case(N, M, K, V, taps, T, pad, seed=1):
    """Inputs of the gated delta rule's kernels as columns of a wider matrix, and the plain recurrence's inputs made from them."""
    C = 2 * M * K + N * V
    p = rand(T, pad + C + N * V + 2 * N + 3, seed=seed)
    conv = rand(C, taps, seed=seed + 1, scale=0.6)
    rate, dt = torch.exp(rand(N, seed=seed + 2) - 2.0), rand(N, seed=seed + 3)
    return C, p, conv, rate, dt, (pad, pad + C, pad + C + N * V, pad + C + N * V + N)


def _plain_delta(p, before, conv, rate, dt, cols, N, M, K, V, state):
    """One request's tokens p [n, ..], its last taps - 1 convolution inputs before them, and its state."""
    n, C, taps = p.shape[0], conv.shape[0], conv.shape[1]
    raw = torch.cat([before, p[:, cols[0]:cols[0] + C].double()])
    x = PZ.silu(PZ.short_convolution(raw, conv.double()))[taps - 1:]
    share = N // M
    q = (PZ.unit(x[:, :M * K].view(n, M, K)) * K ** -0.5).repeat_interleave(share, dim=1)
    k = PZ.unit(x[:, M * K:2 * M * K].view(n, M, K)).repeat_interleave(share, dim=1)
    beta = torch.sigmoid(p[:, cols[2]:cols[2] + N].double())
    g = torch.exp(-rate.double() * PZ.softplus(p[:, cols[3]:cols[3] + N].double() + dt.double()))
    return PZ.delta_rule(q, k, x[:, 2 * M * K:].reshape(n, N, V), g, beta, state=state)


def _ring(state_row, N, K, V, taps, C, pos):
    """The last taps - 1 inputs before position pos, oldest first, from a state row."""
    ring = state_row[N * K * V:N * K * V + taps * C].view(taps, C).double()
    return torch.stack([ring[(pos - j) % taps] if pos - j >= 0 else torch.zeros(C, dtype=torch.float64) for j in range(taps - 1, 0, -1)]) \
        if taps > 1 else torch.zeros(0, C, dtype=torch.float64)


@pytest.mark.parametrize("N, M, K, V, taps", [(3, 1, 10, 17, 3), (4, 2, 64, 64, 4), (2, 2, 96, 130, 5), (2, 1, 200, 16, 1)])
def test_delta_state_is_carried_in_32_bits(N, M, K, V, taps):
    """Preparation and scan alone: outputs, states and rings, for requests of unequal length at unequal positions in one step, from states
    that are not zero."""
    from forge_b200 import kernels
    lens, pos0, slots = [1, 40, 2, 17], [5, 0, 1, 33], [4, 0, 5, 2]
    starts = [0, 1, 41, 43, 60]
    T = sum(lens)
    C, p, conv, rate, dt, cols = _delta_case(N, M, K, V, taps, T, pad=4)
    row = N * K * V + taps * C
    row += -row % 4
    state0 = rand(6, row, seed=7)
    batch = SimpleNamespace(q_start=_i32(starts), slots=_i32(slots), num_requests=4, tok_req=_i32([s for s, n in enumerate(lens) for _ in range(n)]),
                            positions=_i32([a + j for a, n in zip(pos0, lens) for j in range(n)]), num_tokens=T)
    d, state = lambda z: z.to(DEV).contiguous(), state0.to(DEV)
    qkv, g, beta = kernels.gated_delta_prepare(d(p), cols[0], cols[2], cols[3], d(conv.flip(1).t()), d(rate), d(dt), batch, state, N, M, K, V)
    got = kernels.gated_delta_scan(qkv, g, beta, batch, state, N, M, K, V).cpu()
    for s, (lo, hi) in enumerate(zip(starts, starts[1:])):
        old = state0[slots[s]]
        o, S = _plain_delta(p[lo:hi], _ring(old, N, K, V, taps, C, pos0[s]), conv, rate, dt, cols, N, M, K, V, old[:N * K * V].double().view(N, K, V))
        assert max_rel_err(got[lo:hi], o.reshape(hi - lo, N * V)) <= 1e-5
        new = state[slots[s]].cpu()
        assert max_rel_err(new[:N * K * V], S.reshape(-1)) <= 1e-5
        raw = torch.cat([_ring(old, N, K, V, taps, C, pos0[s]), p[lo:hi, cols[0]:cols[0] + C].double()])
        if taps > 1:
            assert torch.equal(_ring(new, N, K, V, taps, C, pos0[s] + hi - lo).float(), raw[-(taps - 1):].float())
    for s in (1, 3):
        assert torch.equal(state[s].cpu(), state0[s])                       # slots that take no part


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("N, M, K, V, taps", [(3, 1, 10, 17, 3), (4, 2, 64, 64, 4), (2, 2, 96, 132, 5), (2, 1, 5, 2, 1), (3, 3, 9, 12, 2), (1, 1, 20, 1100, 4),
                                              (2, 1, 256, 128, 4), (2, 1, 300, 40, 3), (1, 1, 20, 511, 9)])
def test_one_token_of_every_request_in_one_delta_kernel(dtype, N, M, K, V, taps):
    """The kernel of single-token steps: what it returns (normed, weighted, gated) and the states and rings it leaves; slots in any order,
    inputs that are columns of a wider matrix, an output slice; heads whose rows no vector load fits, and heads that registers do not hold."""
    from forge_b200 import kernels
    B, pos, slots = 4, [0, 7, 2, 31], [4, 0, 5, 2]
    C, p, conv, rate, dt, cols = _delta_case(N, M, K, V, taps, B, pad=5 if V % 2 else 8)
    row = N * K * V + taps * C
    row += -row % 4
    state0, nw = rand(6, row, seed=7), 1.0 + rand(V, seed=8, scale=0.3)
    batch = SimpleNamespace(q_start=_i32([0, 1, 2, 3, 4]), slots=_i32(slots), positions=_i32(pos), num_requests=B, num_tokens=B)
    assert kernels.token_state_supports(batch, K, V, True) or V > 512
    d, state = lambda z: z.to(DEV).contiguous(), state0.to(DEV)
    out = torch.full((B, N * V + 7), 3.0, dtype=dtype, device=DEV)
    kernels.gated_delta_token(d(p), cols[0], cols[1], cols[2], cols[3], d(conv.flip(1).t()), d(rate), d(dt), batch, state, N, M, K, V, d(nw), 1e-3, dtype, out=(out, 2))
    for s in range(B):
        old = state0[slots[s]]
        before = _ring(old, N, K, V, taps, C, pos[s])
        o, S = _plain_delta(p[s:s + 1], before, conv, rate, dt, cols, N, M, K, V, old[:N * K * V].double().view(N, K, V))
        want = (PZ.rms(o, 1e-3) * nw.double()).reshape(-1) * PZ.silu(p[s, cols[1]:cols[1] + N * V].double())
        assert max_rel_err(out[s, 2:2 + N * V], want) <= PART_TOL[dtype]
        new = state[slots[s]].cpu()
        assert max_rel_err(new[:N * K * V], S.reshape(-1)) <= 1e-5
        if taps > 1:
            raw = torch.cat([before, p[s:s + 1, cols[0]:cols[0] + C].double()])
            assert torch.equal(_ring(new, N, K, V, taps, C, pos[s] + 1).float(), raw[-(taps - 1):].float())
    for s in (1, 3):
        assert torch.equal(state[s].cpu(), state0[s])
    assert bool((out[:, :2] == 3.0).all()) and bool((out[:, 2 + N * V:] == 3.0).all())
    batch.num_tokens = B + 1                                                # portions take the scan, and so do values of very many channels
    assert not kernels.token_state_supports(batch, K, V, True)
    batch.num_tokens = B
    assert not kernels.token_state_supports(batch, 8, 4096, True)


FAR_CUTS = ([(0, 400)], [(0, 390)] + [(i, i + 1) for i in range(390, 400)], [(0, 2), (2, 4), (4, 131), (131, 133), (133, 400)])


@pytest.mark.parametrize("dtype", DT)
def test_what_the_delta_rule_keeps_and_what_it_replaces(dtype):
    """Head 0 all but never forgets, head 1 forgets at once, both read one key head.  The first token writes a value under key A, token 200
    another under key B, token 300 a third under key A: from then on A gives the third, B the second, and head 1 nothing."""
    W, T = 12, 400
    o = dict(num_heads=2, num_qk_heads=1, head_dim=4, v_head_dim=2, taps=2)
    mixer = _part("mixer", "gated_delta", dtype, hidden_size=W, eps=1e-12, **o)
    t = {n: torch.zeros(s.shape, dtype=torch.bfloat16) for n, s in mixer.tensor_specs().items()}
    for m in ("q", "k", "v"):
        t[f"mix.{m}.conv"][:, 1] = 1.0
    t["mix.q"][0, 0] = t["mix.q"][1, 1] = 8.0      # input 0 asks for key A, input 1 for key B
    t["mix.k"][0, 2] = t["mix.k"][1, 3] = 8.0      # input 2 writes under A, input 3 under B
    for h in range(2):
        t["mix.v"][2 * h, 4] = t["mix.v"][2 * h + 1, 5] = 8.0
        t["mix.g"][2 * h:2 * h + 2, 6] = 4.0
        t["mix.o"][2 * h, 2 * h] = t["mix.o"][2 * h + 1, 2 * h + 1] = 1.0
    t["mix.b"][:, 7] = 20.0                        # only tokens that set input 7 write
    t["mix.b"][:, 6] = -20.0
    t["mix.A_log"][:] = torch.tensor([-20.0, 4.0])
    t["mix.norm"][:] = 1.0
    mixer.bind(t)
    w = {n.split("mix.", 1)[-1]: v.double() for n, v in t.items()}
    for ask in (0, 1):
        x = torch.zeros(T, W)
        x[:, 6] = 1.0
        for at, key, value in ((0, 2, (3.0, 4.0)), (200, 3, (1.0, 0.0)), (300, 2, (0.0, 5.0))):
            x[at, key], x[at, 7], x[at, 4], x[at, 5] = 1.0, 2.0, *value
        x[:, ask] = 1.0
        want = PZ.delta_mixer(x.to(dtype).double(), w, _delta_sizes(o), 1e-12)
        for cuts in FAR_CUTS:
            got = _feed(mixer, _storage(mixer, dtype, 1, 1), x.to(dtype), cuts)["r"]
            shown = torch.tensor([0.0, 1.0] if ask == 0 else [1.0, 0.0]) * 2 ** 0.5 * float(PZ.silu(torch.tensor(4.0)))
            assert torch.allclose(got[-1, :2], shown, atol=5e-2), (ask, cuts, got[-1])
            # (a head that holds nothing has no direction to compare: the norm divides by next to nothing)
            assert max_rel_err(got[:, :2], want[:, :2]) <= PART_TOL[dtype] or ask == 1
            assert max_rel_err(got[200:, :2], want[200:, :2]) <= PART_TOL[dtype]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_the_convolution_reaches_over_every_cut(dtype, taps):
    """One token alone has an input; the filters are one for every token that they reach: what the mixer keeps and gives at the tokens
    after it says how far they reach, wherever the step is cut behind it."""
    W, star, T = 8, 9, 24
    o = dict(num_heads=1, num_qk_heads=1, head_dim=4, v_head_dim=4, taps=taps)
    mixer = _part("mixer", "gated_delta", dtype, hidden_size=W, eps=1e-9, **o)
    t = {n: torch.zeros(s.shape, dtype=torch.bfloat16) for n, s in mixer.tensor_specs().items()}
    for m in ("q", "k", "v"):
        t[f"mix.{m}.conv"][:] = 1.0
    t["mix.q"][0, 0] = t["mix.k"][0, 0] = t["mix.v"][1, 1] = 1.0
    t["mix.g"][:, 2] = 4.0
    t["mix.b"][:, 2] = 8.0
    t["mix.A_log"][:] = 8.0                        # nothing is kept: a token's output is what its own convolution gives
    t["mix.norm"][:] = 1.0
    t["mix.o"][:4, :4] = torch.eye(4)
    mixer.bind(t)
    x = torch.zeros(T, W)
    x[:, 0], x[:, 2], x[star, 1] = 1.0, 1.0, 1.0
    for cut in range(star, min(T - 1, star + taps + 1)):
        for cuts in ([(0, cut), (cut, T)] if cut else [(0, T)], [(0, cut)] + [(i, i + 1) for i in range(cut, T)], [(0, cut), (cut, cut + 2), (cut + 2, T)]):
            got = _feed(mixer, _storage(mixer, dtype, 1, 1), x.to(dtype), cuts)["r"]
            reached = [i for i in range(T) if float(got[i, 1].abs()) > 0.1]
            assert reached == list(range(star, star + taps)), (cuts, reached)


# ----------------------------------------------------------------------------------------------- lightning attention

LIGHTNING = {
    "odd_sizes": dict(num_heads=3, head_dim=10, v_head_dim=17, decay=[0.2, 0.9, 0.999]),
    "one_channel_values": dict(num_heads=2, head_dim=33, v_head_dim=1, decay=[1.0, 0.5]),
    "heads_of_128": dict(num_heads=2, head_dim=128, v_head_dim=64, decay=[0.97, 0.3]),
    "heads_of_256": dict(num_heads=1, head_dim=256, v_head_dim=20, decay=[0.99]),
    "wide_values": dict(num_heads=1, head_dim=6, v_head_dim=1300, decay=[0.9]),
    "values_too_wide_for_one_cta": dict(num_heads=1, head_dim=6, v_head_dim=1301, decay=[0.9]),
    "many_heads": dict(num_heads=20, head_dim=4, v_head_dim=8, decay=[1.0 - 0.5 ** i for i in range(1, 21)]),
}


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", list(LIGHTNING))
def test_lightning_mixer_alone(dtype, kind):
    o = LIGHTNING[kind]
    W, T = 40, 62
    mixer = _part("mixer", "lightning", dtype, hidden_size=W, eps=1e-3, **o)
    t, w = _bf16_weights(mixer, 0.35, seed=len(kind))
    mixer.bind(t)
    storage = _storage(mixer, dtype, 1, 2)
    x = rand(T, W, seed=50).to(dtype)
    want = PZ.lightning(x.double(), w, {"heads": o["num_heads"], "dim": o["head_dim"], "vdim": o["v_head_dim"], "decay": o["decay"]}, 1e-3)
    got = _feed(mixer, storage, x, CUTS, requests=("a", "b"))
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype], (kind, r)
    storage.manager.free("a")
    got = _feed(mixer, storage, x, [(0, 2), (2, 3), (3, 60), (60, 62)], requests=("c",))
    assert max_rel_err(got["c"], want) <= PART_TOL[dtype], kind
    assert storage.check_canaries() == []


@pytest.mark.parametrize("K, V", [(10, 17), (64, 64), (96, 132), (5, 2), (7, 12), (20, 500), (256, 128), (300, 40)])
def test_lightning_state_is_carried_in_32_bits(K, V):
    """The scan (unequal requests) and the kernel of single tokens: outputs and states, from states that are not zero."""
    from forge_b200 import kernels
    N, slots, pad = 3, [4, 0, 5, 2], 4
    decay = torch.tensor([0.3, 0.95, 0.9999])
    state0 = rand(6, N * K * V + 4 - N * K * V % 4, seed=7)
    for lens in ([1, 40, 2, 17], [1, 1, 1, 1]):
        if K > 256 and sum(lens) > 4:
            continue                                                        # the scan takes heads of up to 256 key channels
        starts = [sum(lens[:i]) for i in range(5)]
        T = starts[-1]
        p = rand(T, pad + N * (2 * K + V) + 3, seed=1)
        batch = SimpleNamespace(q_start=_i32(starts), slots=_i32(slots), num_requests=4, num_tokens=T)
        single = kernels.token_state_supports(batch, K, V, False)
        assert single == (T == 4)
        state = state0.to(DEV)
        got = (kernels.lightning_token if single else kernels.lightning_scan)(p.to(DEV), pad, decay.to(DEV), batch, state, N, K, V).cpu()
        x = PZ.silu(p.double())
        for s, (lo, hi) in enumerate(zip(starts, starts[1:])):
            n = hi - lo
            cut = lambda a, m, c: x[lo:hi, pad + a:pad + a + N * m].reshape(n, N, m)
            o, S = PZ.linear_recurrence(cut(0, K, 0), cut(N * K, K, 0), cut(2 * N * K, V, 0), decay.double(),
                                        state=state0[slots[s], :N * K * V].double().view(N, K, V))
            assert max_rel_err(got[lo:hi], o.reshape(n, N * V)) <= 1e-5
            assert max_rel_err(state[slots[s], :N * K * V], S.reshape(-1)) <= 1e-5
        for s in (1, 3):
            assert torch.equal(state[s].cpu(), state0[s])


# ----------------------------------------------------------------------------------------------- chunked attention

ATTENTION = {
    # sizes that only the kernel of fp32 arithmetic takes
    "chunk_shorter_than_a_page": dict(num_heads=6, num_kv_heads=2, head_dim=10, v_head_dim=13, scale=0.8, chunk=5, rot=6, theta=40.0, scaling=(3.0, 40, 8.0, 0.5)),
    "chunk_of_one": dict(num_heads=4, num_kv_heads=1, head_dim=12, v_head_dim=20, scale=0.6, chunk=1, rot=12, theta=1e4),
    "one_chunk_for_all": dict(num_heads=3, num_kv_heads=3, head_dim=6, v_head_dim=4, scale=2.5, chunk=1000, rot=4, theta=70.0, scaling=(0.5, 16, 2.0, 1.0)),
    "no_rotated_channels": dict(num_heads=2, num_kv_heads=2, head_dim=8, v_head_dim=8, scale=1.0, chunk=16, rot=0, theta=10.0),
    "heads_of_200": dict(num_heads=2, num_kv_heads=1, head_dim=200, v_head_dim=12, scale=0.1, chunk=24, rot=120, theta=1e4, scaling=(8.0, 30, 4.0, 1.0)),
    # sizes that the tensor-core kernel takes in bfloat16, with edges inside and across its tiles of 64 keys
    "tc_chunk_72": dict(num_heads=8, num_kv_heads=2, head_dim=64, v_head_dim=24, scale=0.2, chunk=72, rot=48, theta=250000.0, scaling=(8.0, 64, 16.0, 1.0),
                        tokens=230, cuts=LONG_CUTS),
    "tc_chunk_64": dict(num_heads=2, num_kv_heads=2, head_dim=16, v_head_dim=64, scale=0.6, chunk=64, rot=16, theta=100.0, tokens=230, cuts=LONG_CUTS),
    "tc_chunk_130": dict(num_heads=6, num_kv_heads=3, head_dim=48, v_head_dim=80, scale=0.3, chunk=130, rot=32, theta=1e4, tokens=230, cuts=LONG_CUTS),
    "tc_values_of_two_chunks": dict(num_heads=2, num_kv_heads=1, head_dim=32, v_head_dim=264, scale=0.4, chunk=33, rot=32, theta=1e4, tokens=150,
                                    cuts=LONG_CUTS[:5]),
}


def _attention(dtype, W, o, eps=1e-3, **more):
    from forge_b200.config import PartSpec
    o = {k: v for k, v in o.items() if k not in ("tokens", "cuts")}
    rot, theta, scaling = o.pop("rot"), o.pop("theta"), o.pop("scaling", None)
    position = PartSpec("rope_halves", {"head_dim": o["head_dim"], "rotary_dims": rot, "theta": theta,
                                        "scaling": None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))})
    return _part("mixer", "masked_attention", dtype, **{**dict(hidden_size=W, position=position, qk_norm=True, eps=eps, sink=True), **o, **more})


def _plain_sizes(o):
    rot = {"dims": o["rot"], "base": o["theta"]}
    if o.get("scaling"):
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), o["scaling"]))
    return {"heads": o["num_heads"], "kv_heads": o["num_kv_heads"], "dim": o["head_dim"], "vdim": o["v_head_dim"], "scale": o["scale"],
            "mask": {"size": o["chunk"]}, "rot": rot}


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", list(ATTENTION))
def test_chunked_attention_alone(dtype, kind):
    """Two requests side by side, fed in portions down to one token; pages behind the chunk go back on the way."""
    o = ATTENTION[kind]
    W, T, cuts = 40, o.get("tokens", 62), o.get("cuts", CUTS)
    mixer = _attention(dtype, W, o)
    t, w = _bf16_weights(mixer, 0.35, seed=len(kind))
    mixer.bind(t)
    storage = _storage(mixer, dtype, 2 * -(-T // 8), 2)
    x = rand(T, W, seed=50).to(dtype)
    got = _feed(_Adds(mixer), storage, x, cuts, requests=("a", "b"))
    want = PZ.chunked_attention(x.double(), w, _plain_sizes(o), 1e-3)
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype], (kind, r)
    table = storage.manager.block_table("a", next(iter(storage.manager.groups)))
    assert sum(p >= 0 for p in table) <= min(T, o["chunk"]) // 8 + 2, (kind, table)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["chunk_shorter_than_a_page", "tc_chunk_72"])
def test_the_options_of_the_attention_are_independent(dtype, kind):
    """The sink, the division by the root mean square, the stretched frequencies and their amplitude (which shows where some channels pass
    unrotated) each change the output, and each by what the equations say."""
    o = ATTENTION[kind]
    W, T = 40, 62
    x = rand(T, W, seed=50).to(dtype)
    outs = {}
    for what in ("all", "sink_sunk", "no_sink", "no_norm", "no_scaling"):
        oo = {k: v for k, v in o.items() if what != "no_scaling" or k != "scaling"}
        mixer = _attention(dtype, W, oo, qk_norm=what != "no_norm", sink=what != "no_sink")
        t, w = _bf16_weights(mixer, 0.35, seed=3)
        if what == "no_sink":
            w["sink"] = torch.full((o["num_heads"],), -1e9, dtype=torch.float64)
        if what == "sink_sunk":
            t["mix.sink"][0] = 120.0
            w["sink"] = t["mix.sink"].double()
        mixer.bind(t)
        got = _feed(_Adds(mixer), _storage(mixer, dtype, 8, 1), x, CUTS)["r"]
        if what == "no_norm":
            saved = PZ.rms
            PZ.rms = lambda y, eps: y
            try:
                want = PZ.chunked_attention(x.double(), w, _plain_sizes(oo), 1e-3)
            finally:
                PZ.rms = saved
        else:
            want = PZ.chunked_attention(x.double(), w, _plain_sizes(oo), 1e-3)
        assert max_rel_err(got, want) <= PART_TOL[dtype], what
        outs[what] = want
    for what in ("sink_sunk", "no_sink", "no_norm", "no_scaling"):
        assert float((outs[what] - outs["all"]).abs().max()) > 0.02 * float(outs["all"].abs().max()), what


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("page_size", [8, 64])
@pytest.mark.parametrize("size, D, E", [(100, 12, 4), (100, 16, 8), (64, 16, 8), (40, 16, 8)])
def test_one_key_that_stands_out(dtype, page_size, size, D, E):
    """All keys are zero except one that head 0 asks for; values carry their position, and every head's sink is zero.  Head 0 returns the
    key's position where the token sees it, and the mean of the visible positions less the sink's share where it does not; head 1 always
    the latter.  The key lies far back, just inside and just outside the token's chunk, at a page's border, ahead in the same portion, or
    is the token itself; for the tokens of a portion and for tokens that come alone; on pages that the case before gave back."""
    from forge_b200.engine import StepEntry, build_step_batch
    N, P, W, H = 290, 27, 16, 2
    dev = torch.device(DEV)
    mixer = _attention(dtype, W, dict(num_heads=H, num_kv_heads=1, head_dim=D, v_head_dim=E, scale=2.5, chunk=size, rot=4, theta=100.0), eps=1e-6)
    t = {n: torch.zeros(s.shape, dtype=torch.bfloat16) for n, s in mixer.tensor_specs().items()}
    t["mix.q"][D - 1, 1] = 4.0                                               # head 0's last channel, which no rotation touches
    t["mix.k"][D - 1, 0] = 4.0
    t["mix.v"][0, 2] = 1.0
    for h in range(H):
        t["mix.o"][h, h * E] = 1.0
    mixer.bind(t)
    storage = _storage(mixer, dtype, 64 * 8 // page_size, 2, page_size)
    total = N + P + 2
    stars = [0, 150, 255, 256, N - 1, N, N + 5, N + P - 1, N + P, N + P + 1]
    edge = size * ((N + P) // size)                                          # the start of the chunk that the portion's end lies in
    stars += [edge - 1, edge, edge + 1, size * (N // size) - 1, size * (N // size), size * (N // size + 1) - 1, size * (N // size + 1)]
    for case, star in enumerate(sorted({s for s in stars if 0 <= s < total})):
        rid = f"r{case}"
        storage.manager.admit(rid)
        x = torch.zeros(total, W)
        x[star, 0] = 1.0
        x[:, 1] = 1.0
        x[:, 2] = torch.arange(total, dtype=torch.float32) / 4.0
        done = 0
        for n in (N, P, 1, 1):
            batch = build_step_batch([StepEntry(rid, [0] * n, [])], storage.manager, dev, 64)
            out = mixer.forward(x[done:done + n].to(DEV).to(dtype).contiguous(), batch, storage.layers[0], None).cpu()
            storage.manager.release_out_of_window(rid)
            for i in range(n):
                pos = done + i
                lo = pos // size * size
                count, mean = pos + 1 - lo, (lo + pos) / 2.0 / 4.0
                share = mean * count / (count + 1.0)
                tol = (1e-4 if dtype == torch.float32 else 2e-2) * max(1.0, pos / 4.0)
                want0 = star / 4.0 if lo <= star <= pos else share
                assert abs(float(out[i, 0]) - want0) <= tol and abs(float(out[i, 1]) - share) <= tol, (size, star, pos, out[i, :2].tolist(), want0, share)
            done += n
        storage.manager.free(rid)                                            # the next case takes over these pages
        storage.manager.check()


@pytest.mark.parametrize("context", [3, 70, 200, 500])
def test_single_tokens_dealt_out_in_runs_count_the_sink_once(context):
    """A decode step's keys are dealt out to several CTAs, whose sums a second kernel puts together: the sink joins there, once."""
    from forge_b200 import kernels
    H, G, D, E, ps = 4, 2, 32, 24, 16
    pages = -(-(context + 1) // ps)
    cache = rand(pages, G * ps * (D + E), seed=1).to(DEV).to(torch.bfloat16)
    q = rand(1, H * D, seed=2).to(DEV).to(torch.bfloat16)
    sink = torch.tensor([0.5, -3.0, 4.0, 30.0], device=DEV)
    table = torch.arange(pages, dtype=torch.int32, device=DEV).view(1, pages)
    outs = []
    for decode in (True, False):
        batch = SimpleNamespace(num_requests=1, num_tokens=1, host_q_start=[0, 1], attention_plan={}, tok_req=_i32([0]), positions=_i32([context]))
        if decode:
            batch.decode_only, batch.max_context = True, 512
        outs.append(kernels.scored_attention(q, cache, SimpleNamespace(block_table=table), batch, H, G, 1, D, E, ps, 0.3, sink=sink).float().cpu())
    kv = cache.float().cpu().double()
    keys, values = kv[:, :G * ps * D].reshape(pages, G, ps, D), kv[:, G * ps * D:].reshape(pages, G, ps, E)
    for h in range(H):
        g = h // (H // G)
        k, v = keys[:, g].reshape(-1, D)[:context + 1], values[:, g].reshape(-1, E)[:context + 1]
        s = (k @ q[0, h * D:(h + 1) * D].float().cpu().double()) * 0.3
        m = max(float(s.max()), float(sink[h]))
        want = (torch.exp(s - m) @ v) / (torch.exp(s - m).sum() + torch.exp(sink[h].cpu().double() - m))
        for o in outs:
            assert float((o[0, h * E:(h + 1) * E] - want).abs().max()) <= 2e-2 * max(1e-3, float(want.abs().max())), (h, context)


# ----------------------------------------------------------------------------------------------- the two side by side, feed-forwards

@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("right", [dict(num_heads=3, head_dim=9, v_head_dim=5, decay=[0.3, 0.9, 0.998]), dict(num_heads=2, head_dim=16, v_head_dim=8, decay=[0.5, 0.99])])
def test_two_mixers_whose_outputs_are_normed(dtype, right):
    from forge_b200.config import PartSpec
    o = ATTENTION["chunk_shorter_than_a_page"]
    W, T = 40, 62
    att = _attention(torch.float32, W, o)                                    # (for its spec's shape only)
    assert att.chunk == 5
    rot = {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 0.5}
    specs = [PartSpec("masked_attention", dict(hidden_size=W, num_heads=6, num_kv_heads=2, head_dim=10, v_head_dim=13, scale=0.8, chunk=5, qk_norm=True,
                                               eps=1e-3, sink=True, prefix="mix.left.", position=PartSpec("rope_halves", {
                                                   "head_dim": 10, "rotary_dims": 6, "theta": 40.0, "scaling": rot}))),
             PartSpec("lightning", dict(right, hidden_size=W, eps=1e-3, prefix="mix.right."))]
    mixer = _part("mixer", "side_by_side", dtype, mixers=specs, hidden_size=W, out_norms=["mix.left.out", "mix.right.out"], out_scale=0.5, eps=1e-3)
    t, w = _bf16_weights(mixer, 0.35, seed=8)
    mixer.bind(t)
    assert mixer.proj is not None and mixer.o is None                        # one input product, an output product each
    x = rand(T, W, seed=50).to(dtype)
    got = _feed(mixer, _storage(mixer, dtype, 16, 2), x, CUTS, requests=("a", "b"))
    m = {"left": _plain_sizes(o), "right": {"heads": right["num_heads"], "dim": right["head_dim"], "vdim": right["v_head_dim"], "decay": right["decay"]}}
    want = PZ.parallel_mixer(x.double(), w, m, 1e-3)
    for r in ("a", "b"):
        assert max_rel_err(got[r], want) <= PART_TOL[dtype]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T, W, F", [(1, 40, 24), (3, 75, 41), (9, 64, 96), (150, 192, 320), (300, 64, 20)])
def test_dense_feed_forward_with_biases(dtype, T, W, F):
    ff = _part("feed_forward", "swiglu", dtype, hidden_size=W, intermediate_size=F, suffix="", bias=True,
               names={"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"})
    t = {n: rand(*s.shape, seed=i, scale=0.7 if n.endswith(".b") else 0.3).to(torch.bfloat16) for i, (n, s) in enumerate(ff.tensor_specs().items())}
    ff.bind(t)
    x, r0 = rand(T, W, seed=9).to(dtype), rand(T, W, seed=10)
    res = r0.clone().to(DEV)
    ff.forward(x.to(DEV), res)
    want = r0.double() + PZ.dense_ff(x.double(), {k.split("mlp.", 1)[1]: v.double() for k, v in t.items()})
    assert max_rel_err(res, want) <= PART_TOL[dtype]


def test_the_router_ranks_groups_by_their_two_largest():
    from forge_b200 import kernels
    for seed, (E, top, groups, keep) in enumerate([(8, 2, 4, 2), (12, 3, 3, 2), (9, 3, 3, 1), (6, 6, 1, 1), (10, 2, 10, 4), (16, 4, 4, 2), (7, 2, 0, 0), (64, 6, 8, 3)]):
        W, T = 24, 200
        w = {"router": rand(E, W, seed=seed, scale=0.5), "correction": rand(E, seed=seed + 50, scale=0.3)}
        x = rand(T, W, seed=seed + 100)
        r = {"experts": E, "top": top}
        if groups:
            r["groups"] = {"count": groups, "keep": keep}
        want_idx, want_w, margin = PZ.route(x.double(), {k: v.double() for k, v in w.items()}, r)
        idx, wts = kernels.moe_route(x.to(DEV), w["router"].to(DEV), top, correction=w["correction"].to(DEV), groups=groups, keep=keep, group_top=2)
        clear = margin > 1e-5
        assert int(clear.sum()) > T * 0.9
        assert torch.equal(idx.cpu().long()[clear], want_idx[clear]), (E, top, groups, keep)
        assert max_rel_err(wts.cpu()[clear], want_w[clear]) <= 1e-5
    # two good experts beat the best one beside a bad one; negative numbers count as they are, and a dropped block's are out
    router, corr = torch.zeros(6, 8), torch.tensor([0.5, -2.9, -0.6, -0.7, -1.3, -1.4])
    for group_top, want in ((2, [2, 3]), (1, [0, 1])):
        idx, wts = kernels.moe_route(torch.ones(2, 8).to(DEV), router.to(DEV), 2, correction=corr.to(DEV), groups=3, keep=1, group_top=group_top)
        assert idx.cpu().tolist() == [want, want] and torch.allclose(wts.cpu(), torch.full((2, 2), 0.5))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("W, F, E, top, groups, keep, T", [(40, 24, 6, 2, 3, 2, 19), (40, 16, 4, 1, 1, 1, 3), (64, 48, 9, 3, 3, 1, 300), (192, 128, 8, 2, 4, 2, 130),
                                                          (256, 64, 4, 2, 4, 2, 1), (64, 16, 12, 3, 0, 0, 11)])
def test_routed_experts_of_this_kind(dtype, W, F, E, top, groups, keep, T):
    ff = _part("feed_forward", "routed_experts", dtype, hidden_size=W, intermediate_size=F, experts=E, top=top, correction=True, groups=groups, keep=keep,
               group_top=2)
    t = {n: rand(*s.shape, seed=i, scale=0.3).to(torch.bfloat16) for i, (n, s) in enumerate(ff.tensor_specs().items())}
    ff.bind(t)
    x = rand(T, W, seed=9, scale=1.5).to(dtype)
    r = {"experts": E, "top": top, **({"groups": {"count": groups, "keep": keep}} if groups else {})}
    want, _, margin = PZ.routed_ff(x.double(), {k.split("mlp.", 1)[1]: v.double() for k, v in t.items()}, {"router": r})
    clear = margin > 1e-3                                                    # no test rests on a close call
    assert int(clear.sum()) >= max(1, T // 3)
    assert max_rel_err(ff.forward(x.to(DEV), None).cpu()[clear], want[clear]) <= PART_TOL[dtype]


# ----------------------------------------------------------------------------------------------- whole models

class _Plain:
    def __init__(self, d):
        self.dir = d
        self.cfg, self.tensors = PZ.load(d)
        self.close = {}

    def forward(self, toks, layers_out=None, margins=None, choices=None):
        return PZ.forward(self.cfg, self.tensors, list(toks), layers_out=layers_out, margins=margins, choices=choices)

    def forward_as_routed_in_16_bits(self, toks):
        """Where two experts' (or two groups') ranking numbers lie within the rounding of 16-bit activations, either choice is right and
        the outputs differ.  So the 16-bit runtime is compared with the plain implementation taking the experts that the engine took for
        the whole prompt, and every choice that is not the plain router's own must be such a close call."""
        theirs = _engine_choices(self.dir, list(toks))
        if not theirs:
            return self.forward(toks)
        margins = []
        out = self.forward(toks, margins=margins, choices=theirs)
        assert len(margins) == len(theirs)
        for k, (own, m) in enumerate(margins):
            for t in torch.nonzero(m > 0.03).flatten().tolist():
                assert sorted(theirs[k][t].tolist()) == sorted(own[t].tolist()), f"routed run {k}, token {t}: the engine chose other experts on a clear call"
        # tokens with a close call somewhere: cut otherwise (a token alone, a portion) the 16-bit runtime may decide them the other way
        self.close[tuple(toks)] = torch.stack([m for _, m in margins]).min(dim=0).values < 0.01
        return out

    def close_calls(self, toks):
        return self.close.get(tuple(toks), torch.zeros(len(toks), dtype=torch.bool))


@pytest.fixture(scope="module", params=list(ZUR))
def zur(request, tmp_path_factory):
    name = request.param
    d = make_zur_dir(tmp_path_factory, name)
    plain = _Plain(d)
    reqs = {f"r{i}": random_tokens(n, ZUR[name]["vocab"], seed=10 * i + ord(name)) for i, n in enumerate(LENGTHS[name])}
    want = {"float32": {rid: plain.forward(toks).float() for rid, toks in reqs.items()},
            "bfloat16": {rid: plain.forward_as_routed_in_16_bits(toks).float() for rid, toks in reqs.items()}}
    return name, d, plain, reqs, want


def test_layer_by_layer(zur):
    """The stream after every layer, in 32-bit, for a prompt in two portions."""
    name, d, plain, reqs, want = zur
    from forge_b200.engine import StepEntry
    runner = make_runner(d, "float32", 256)
    seen = []
    for b in set(runner.model.blocks):
        def wrap(orig):
            def f(residual, batch, cache):
                orig(residual, batch, cache)
                seen.append(residual.clone())
            return f
        b.forward = wrap(b.forward)
    toks = reqs["r2"]
    runner.admit("x")
    for part in (toks[:9], toks[9:]):
        runner.step([StepEntry("x", part, [])])
    ref = []
    plain.forward(toks, layers_out=ref)
    n = len(ZUR[name]["layers"])
    assert len(ref) == n and len(seen) == 2 * n
    for i in range(n):
        assert max_rel_err(torch.cat([seen[i], seen[n + i]]), ref[i]) <= 2e-5, f"layer {i}"


def test_shared_weights_equal_copies_of_them():
    """A layer that uses another's weights computes what a layer with copies of them would, with a cache and a state of its own."""
    import copy
    from forge_b200.config import config_from_dict
    from forge_b200.engine import ModelRunner, StepEntry
    for name in ("E", "F"):
        tensors, d = zur_tensors(name), copy.deepcopy(ZUR[name])
        copies = dict(tensors)
        for i, layer in enumerate(d["layers"]):
            j = layer.pop("weights_of", None)
            if j is not None:
                copies.update({f"l{i}." + n.split(".", 1)[1]: v for n, v in tensors.items() if n.startswith(f"l{j}.")})
        toks = random_tokens(50, d["vocab"], seed=5)
        outs = []
        for cfg, t in ((zur_config(name), tensors), (config_from_dict(d), copies)):
            runner = ModelRunner(config=cfg, tensors=t, dtype="float32", page_size=8, cache_tokens=64, max_requests=1)
            runner.admit("x")
            outs.append([runner.step([StepEntry("x", part, list(range(len(part))))]).cpu() for part in (toks[:30], toks[30:31], toks[31:])])
        for a, b in zip(*outs):
            assert torch.equal(a, b), name


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("schedule", ["whole", "last_one_by_one", "changing_portions", "mixed"])
def test_schedules_equal_plain(zur, dtype, schedule):
    name, d, plain, reqs, want = zur
    steps = getattr(schedules, schedule)(reqs)
    # exactly as many pages as the schedule's peak needs: freed pages and slots are taken again at once
    runner = make_runner(d, dtype, schedules.peak_tokens(reqs, steps, round_to=8))
    got = run_schedule(runner, reqs, steps)
    msg = _first_bad(plain, reqs, got, want[dtype], dtype)
    assert msg is None, msg
    assert runner.manager.num_free_pages() == {g: runner.num_pages for g in runner.manager.groups}
    runner.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_page_size_and_graphs_do_not_matter(zur, dtype):
    name, d, plain, reqs, want = zur
    small = {k: reqs[k] for k in list(reqs)[:3]}
    for ps, graphs in ((16, True), (64, True), (8, False)):
        steps = schedules.mixed(small, max_live=2)
        runner = make_runner(d, dtype, schedules.peak_tokens(small, steps, round_to=ps), page_size=ps, cuda_graphs=graphs)
        got = run_schedule(runner, small, steps)
        msg = _first_bad(plain, small, got, {k: want[dtype][k] for k in small}, dtype)
        assert msg is None, f"page size {ps}: {msg}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_first_tokens(zur, dtype):
    """Two tokens, then hundreds one by one (graph replays): chunks pass over decoded tokens, the convolutions' inputs go round."""
    name, d, plain, reqs, want = zur
    n = {"E": 210, "F": 260, "G": 170, "H": 140, "J": 110}[name]
    toks = random_tokens(n, ZUR[name]["vocab"], seed=77)
    ref = (plain.forward(toks) if dtype == "float32" else plain.forward_as_routed_in_16_bits(toks)).float()
    runner = make_runner(d, dtype, -(-n // 8) * 8)
    assert runner.cuda_graphs
    steps = [([("x", 0, 2)], [])] + [([("x", p, 1)], []) for p in range(2, n)]
    got = run_schedule(runner, {"x": toks}, steps)
    msg = _first_bad(plain, {"x": toks}, got, {"x": ref}, dtype)
    assert msg is None, msg


def test_a_batch_equals_each_request_alone(zur):
    """Unequal requests in one step against each of them alone, in 32-bit, portion by portion."""
    name, d, plain, reqs, want = zur
    from forge_b200.engine import StepEntry
    small = {k: reqs[k] for k in list(reqs)[:4]}
    cuts = {"r0": [5, 1, 20, 2], "r1": [1, 30, 1, 1], "r2": [2, 2, 9, 3], "r3": [17, 1, 1, 11]}

    def run(ids):
        runner = make_runner(d, "float32", 512, cuda_graphs=False)
        got, at = {r: [] for r in ids}, {r: 0 for r in ids}
        for r in ids:
            runner.admit(r)
        for k in range(4):
            rows = runner.step([StepEntry(r, small[r][at[r]:at[r] + cuts[r][k]], list(range(cuts[r][k]))) for r in ids]).cpu()
            for r in ids:
                got[r].append(rows[:cuts[r][k]])
                rows = rows[cuts[r][k]:]
                at[r] += cuts[r][k]
        return {r: torch.cat(v) for r, v in got.items()}
    together = run(list(small))
    for r in small:
        alone = run([r])[r]
        assert float((together[r] - alone).abs().max()) <= 2e-5 * float(alone.abs().max()), r


def test_fp32_logits_do_not_depend_on_the_cut(zur):
    name, d, plain, reqs, want = zur
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
def test_generation_through_the_scheduler(zur, dtype):
    """Greedy generation through forge.Model and through RequestScheduler with more requests than slots and few pages."""
    import forge_b200 as forge
    name, d, plain, reqs, want = zur
    model = forge.Model(d, dtype=dtype, block_size=8, max_num_seqs=2, cache_tokens=512, max_tokens_per_step=48)
    prompt = reqs["r1"][:30]
    out = model.generate(prompt, max_new_tokens=12, do_sample=False)
    assert out["num_generated_tokens"] == 12 and out["finish_reason"] == "length"
    logits_fn = lambda ids: (plain.forward(ids) if dtype == "float32" else plain.forward_as_routed_in_16_bits(ids)).float()
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


def test_trace_replay_as_a_subprocess(zur, tmp_path):
    name, d, plain, reqs, want = zur
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
    V = ZUR[name]["vocab"]
    for n, rows in asked.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), V))
        ref = torch.stack([want["float32"][rid][pos] for rid, pos in rows])
        assert max_rel_err(got, ref) <= TOL["float32"], n
    assert sorted(os.listdir(out)) == sorted(f"{n}.f32" for n in asked)


def test_command_line(zur):
    """bin/forge-cli on a Zuretar folder: greedy tokens in 32-bit follow the plain implementation; sampling runs."""
    name, d, plain, reqs, want = zur
    if name in ("H", "J"):
        return
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
