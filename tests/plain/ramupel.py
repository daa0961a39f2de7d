"""Whole-sequence Ramupel decoder, written from the design's equations: one request, all of its tokens, every time; no
cache, no batching, no fusing, keys and values formed per head, one token after the other through the recurrence.  float64
on the CPU.  One function per mechanism.

Notation: T tokens, W model width, H heads of the latent mixer with D unrotated and R rotated query/key channels and E value
channels, C the latent's width; N heads of the recurrent mixer with K key and V value channels.
"""
import json
import math
import os

import torch

from .safetensors_reader import read_safetensors


def layer_norm(x, w, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def xielu(z, p, q):
    """Quadratic above zero, exponential below, with slope 1/2 at zero from both sides."""
    above = softplus(p) * z * z + 0.5 * z
    neg = z.clamp(max=0.0)
    below = (0.5 + softplus(q)) * (torch.expm1(neg) - neg) + 0.5 * z
    return torch.where(z > 0, above, below)


def rotate_halves(x, positions, base, dims):
    """x [T, ..., >= dims]: channel i turns with channel i + dims/2 by position * base^(-2i/dims); the rest pass."""
    half = dims // 2
    i = torch.arange(half, dtype=x.dtype)
    f = torch.pow(torch.tensor(float(base), dtype=x.dtype), -2.0 * i / dims)
    a = positions.to(x.dtype)[:, None] * f[None, :]
    while a.dim() < x.dim():
        a = a.unsqueeze(1)
    c, s = torch.cos(a), torch.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def causal_softmax(scores):
    T = scores.shape[0]
    ok = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    s = scores.masked_fill(~ok, -math.inf)
    p = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return p / p.sum(dim=-1, keepdim=True)


def latent_attention(h, w, m, eps):
    T = h.shape[0]
    H, D, R, E, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w["q"].T).view(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :C], w["dkv.norm"], eps)
    kr = rotate_halves(down[:, C:], pos, m["rot"]["base"], R)              # [T, R], one for all heads
    qr = rotate_halves(q[..., D:], pos, m["rot"]["base"], R)
    ku = (c @ w["uk"].T).view(T, H, D)
    val = (c @ w["uv"].T).view(T, H, E)
    gate = torch.sigmoid(h @ w["g"].T)                                     # [T, H]
    heads = [causal_softmax((q[:, n, :D] @ ku[:, n].T + qr[:, n] @ kr.T) * m["scale"]) @ val[:, n] * gate[:, n:n + 1] for n in range(H)]
    return torch.cat(heads, dim=-1) @ w["o"].T


def channel_decay(h, w, tau):
    """A decay in (0, 1) per token and key channel, from a projection through a small hidden layer."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_recurrence(q, k, v, decay, state=None):
    """q, k, decay [T, N, K], v [T, N, V] -> (o [T, N, V], the state [N, K, V] after the last token)."""
    T, N, K = q.shape
    S = torch.zeros(N, K, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("nkv,nk->nv", S, q[t]))
    return torch.stack(out), S


def gla(h, w, m, eps):
    T = h.shape[0]
    N, K, V = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, N, K) * K ** -0.5, (h @ w["k"].T).view(T, N, K), (h @ w["v"].T).view(T, N, V)
    o, _ = gated_recurrence(q, k, v, channel_decay(h, w, m["tau"]).view(T, N, K))
    g = h @ w["g"].T
    return (rms_norm(o, w["norm"], eps).reshape(T, N * V) * g * torch.sigmoid(g)) @ w["o"].T


def feed_forward(h, w):
    return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def depth_average(history, weights):
    """The weighted sum of everything the layers have left so far, the embedding output first."""
    return sum(weights[j] * history[j] for j in range(len(history)))


def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, w, m, eps):
    if kind == "latent_attention":
        return latent_attention(h, w, m, eps)
    if kind == "gla":
        return gla(h, w, m, eps)
    raise ValueError(kind)


def layer(x, t, prefix, spec, eps):
    """What a layer leaves before the average over the depth."""
    h = layer_norm(x, t[prefix + "norm1"], eps)

    def gate(n):
        return torch.sigmoid(h @ t[f"{prefix}rg{n}"].T + t[f"{prefix}rg{n}.b"])
    y = x + mixer(spec["type"], h, _sub(t, prefix + "mix."), spec["mixer"], eps) * gate(1)
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, _sub(t, prefix + "mlp.")) * gate(2)
    return y


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that receives the stream after every layer (averaged)."""
    t = {k: torch.as_tensor(v).to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.tensor(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    history = [x]
    for i, spec in enumerate(cfg["layers"]):
        history.append(layer(x, t, f"l{i}.", spec, eps))
        x = depth_average(history, t[f"l{i}.dwa"])
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, t["final.norm"], eps) @ t["embed"].T


def load(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))
