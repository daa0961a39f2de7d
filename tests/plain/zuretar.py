"""Whole-sequence Zuretar decoder, written from the design's equations: one request, all of its tokens, every time; no cache, no
batching, no fusing, one token after the other through the recurrences.  float64 on the CPU.  One function per mechanism.

Notation: T tokens, W model width; in the delta mixer N heads of K key and V value channels that share M query/key heads; in the
attention H query heads on G key/value heads of D query/key and E value channels.
"""
import json
import math
import os

import torch

from .safetensors_reader import read_safetensors


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


# ---------------------------------------------------------------------------------------------- the delta mixer

def short_convolution(x, w):
    """x [T, C], w [C, n]: y_t[c] = sum_j w[c, n-1-j] x_{t-j}[c], nothing before the start."""
    T, C = x.shape
    n = w.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=x.dtype), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(n))


def delta_rule(q, k, v, g, beta, state=None):
    """q, k [T, N, K], v [T, N, V], g, beta [T, N] -> (o [T, N, V], the state [N, K, V] after the last token)."""
    T, N, K = q.shape
    S = torch.zeros(N, K, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("nkv,nk->nv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("nkv,nk->nv", S, q[t]))
    return torch.stack(out), S


def delta_mixer(h, w, m, eps):
    T = h.shape[0]
    N, M, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    share = N // M
    q = (unit(q.view(T, M, K)) * K ** -0.5).repeat_interleave(share, dim=1)        # head n reads query/key head n // share
    k = unit(k.view(T, M, K)).repeat_interleave(share, dim=1)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = delta_rule(q, k, v.view(T, N, V), g, beta)
    y = rms(o, eps) * w["norm"] * silu((h @ w["g"].T).view(T, N, V))
    return y.reshape(T, N * V) @ w["o"].T


# ---------------------------------------------------------------------------------------------- the two mixers side by side

def rotation_frequencies(dims, base, scaling=None):
    """(frequency per pair, what cos and sin are multiplied by)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim_of(scaling["fast"])), 0), min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, D] at positions 0 .. T-1: the first rot["dims"] channels turn (channel i with channel i + dims/2), the rest pass."""
    dims = rot["dims"]
    half = dims // 2
    f, amp = rotation_frequencies(dims, rot["base"], rot.get("scaling"))
    a = (torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f)[:, None, :]
    c, s = (torch.cos(a) * amp).to(x.dtype), (torch.sin(a) * amp).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def chunk_mask(T, size):
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def softmax_with_sink(scores, seen, sink):
    """scores [T, T]; the denominator also counts exp(sink)."""
    s = scores.masked_fill(~seen, -math.inf)
    m = torch.maximum(s.max(dim=-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    p = torch.exp(s - m)
    return p / (p.sum(dim=-1, keepdim=True) + torch.exp(sink - m))


def chunked_attention(h, w, m, eps):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(rotate((h @ w["q"].T).view(T, H, D), m["rot"]), eps)
    k = rms(rotate((h @ w["k"].T).view(T, G, D), m["rot"]), eps)
    v = (h @ w["v"].T).view(T, G, E)
    seen = chunk_mask(T, m["mask"]["size"])
    heads = []
    for n in range(H):
        g = n // (H // G)
        heads.append(softmax_with_sink(q[:, n] @ k[:, g].T * m["scale"], seen, w["sink"][n]) @ v[:, g])
    return torch.cat(heads, dim=-1) @ w["o"].T


def linear_recurrence(q, k, v, decay, state=None):
    """q, k [T, N, K], v [T, N, V], decay [N] -> (o [T, N, V], the state after the last token)."""
    T, N, K = q.shape
    S = torch.zeros(N, K, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("nkv,nk->nv", S, q[t]))
    return torch.stack(out), S


def lightning(h, w, m, eps):
    T = h.shape[0]
    N, K, V = m["heads"], m["dim"], m["vdim"]
    q, k, v = silu(h @ w["q"].T).view(T, N, K), silu(h @ w["k"].T).view(T, N, K), silu(h @ w["v"].T).view(T, N, V)
    o, _ = linear_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o.reshape(T, N * V), eps) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def parallel_mixer(h, w, m, eps):
    left = chunked_attention(h, _sub(w, "left."), m["left"], eps)
    right = lightning(h, _sub(w, "right."), m["right"], eps)
    return (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"]) / 2.0


# ---------------------------------------------------------------------------------------------- feed-forwards

def dense_ff(h, w):
    return (silu(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def route(h, w, r):
    """(the chosen experts [T, top], their weights, by how much the choice was made: the smaller of the distance between the last chosen
    and the first left-out expert and the distance between the last kept and the first dropped group)."""
    n, top = r["experts"], r["top"]
    s = torch.sigmoid(h @ w["router"].T)
    choice = s + w["correction"]
    margin = torch.full((h.shape[0],), math.inf, dtype=h.dtype)
    groups = r.get("groups")
    if groups:
        count, keep = groups["count"], groups["keep"]
        per = n // count
        best = choice.view(-1, count, per).sort(dim=-1, descending=True).values[..., :2].sum(dim=-1)        # the two largest of each group
        order = best.sort(dim=-1, descending=True)
        kept = torch.zeros(h.shape[0], count, dtype=torch.bool).scatter_(1, order.indices[:, :keep], True)
        choice = choice.masked_fill(~kept.repeat_interleave(per, dim=1), -math.inf)
        if keep < count:
            margin = torch.minimum(margin, order.values[:, keep - 1] - order.values[:, keep])
    order = choice.sort(dim=-1, descending=True)
    idx = order.indices[:, :top]
    if top < n:
        margin = torch.minimum(margin, order.values[:, top - 1] - order.values[:, top])
    return idx, s.gather(1, idx), margin


def routed_ff(h, w, mlp, chosen=None):
    """(output, the router's own choice, its margin); ``chosen`` [T, top]: take these experts instead."""
    own, _, margin = route(h, w, mlp["router"])
    idx = own if chosen is None else chosen
    wts = torch.sigmoid(h @ w["router"].T).gather(1, idx)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = f"e{int(idx[t, j])}."
            y[t] += wts[t, j] * (w[e + "down"] @ (silu(w[e + "gate"] @ h[t]) * (w[e + "up"] @ h[t])))
    return y, own, margin


# ---------------------------------------------------------------------------------------------- the decoder

def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def weights_layer(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None, margins=None, choices=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that receives the stream after every layer; ``margins``: receives
    (own choice, margin) of every routed layer; ``choices``: the experts that the routed layers take, in order."""
    t = {k: torch.as_tensor(v).to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.tensor(tokens)]
    routed = 0
    for i, spec in enumerate(cfg["layers"]):
        w = _sub(t, f"l{weights_layer(cfg['layers'], i)}.")
        h = rms(x, eps) * w["norm1"]
        add = (delta_mixer if spec["type"] == "delta" else parallel_mixer)(h, _sub(w, "mix."), spec["mixer"], eps)
        mlp = spec.get("mlp")
        if mlp is not None and mlp["kind"] == "dense":
            add = add + dense_ff(h, _sub(w, "mlp."))
        elif mlp is not None:
            y, own, margin = routed_ff(h, _sub(w, "mlp."), mlp, None if choices is None else choices[routed])
            add, routed = add + y, routed + 1
            if margins is not None:
                margins.append((own, margin))
        x = x + add
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * t["final.norm"]) @ t["head"].T


def load(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))
