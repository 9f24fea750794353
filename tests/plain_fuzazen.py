"""The Fuzazen decoder written out plainly in float64, one function per mechanism, whole sequences
at a time and with no cache: the oracle of the engine's tests.  It shares nothing with the engine.

Notation: x [n, width] is the residual stream of one sequence whose tokens sit at positions 0..n-1
and at the same time what a sublayer reads, t a dict of the model's tensors by name, m a layer's
`mixer` entry.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scaled_embedding(table, tokens, scale):
    return table[torch.tensor(tokens)] * scale


def turn_pairs(x, positions, base, dims):
    """x [n, heads, size]: entries 2i and 2i + 1 (2i < dims) are the two coordinates that position *
    base^(-2i/dims) turns; entries from `dims` on stay."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def seen(n, chunk: Optional[int]):
    """[n, n], row i true at the positions that a query at i sees: not after i, and in i's own block of
    `chunk` positions, blocks counted from the sequence's start."""
    p = torch.arange(n)
    ok = p[None, :] <= p[:, None]
    if chunk:
        ok = ok & (torch.div(p[None, :], chunk, rounding_mode="floor") == torch.div(p[:, None], chunk, rounding_mode="floor"))
    return ok


def softmax_with_sink(scores, sink):
    """Rows of weights; the sink takes a share of the sum and carries nothing."""
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def one_head(q, k, v, scale, mask, sink):
    s = ((q @ k.T) * scale).masked_fill(~mask, -math.inf)
    return softmax_with_sink(s, sink) @ v


def attention(t: Dict[str, torch.Tensor], p: str, m, h, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(n)
    rot = m["rot"]
    q = turn_pairs((h @ t[p + "q"].T).view(n, H, d), pos, rot["base"], rot["dims"])
    k = turn_pairs((h @ t[p + "k"].T).view(n, G, d), pos, rot["base"], rot["dims"])
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    v = (h @ t[p + "v"].T).view(n, G, dv)
    gate = torch.sigmoid(h @ t[p + "g"].T)
    mask = seen(n, (m.get("mask") or {}).get("size"))
    outs = []
    for head in range(H):
        g = head // (H // G)
        o = one_head(q[:, head], k[:, g], v[:, g], m["scale"], mask, t[p + "sink"][head])
        outs.append(o * gate[:, head: head + 1])
    return torch.cat(outs, -1) @ t[p + "o"].T


def feed_forward(t, p: str, h):
    z = h @ t[p + "gate"].T
    return (z * torch.sigmoid(z) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def add_normed(x, y, w, mult, eps):
    return x + mult * (unit_rms(y, eps) * w)


def capped(z, cap: Optional[float]):
    return cap * torch.tanh(z / cap) if cap else z


def forward(config, tensors: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None):
    """Logits [n, vocab] of one sequence; `collect` receives the stream after every layer run."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = scaled_embedding(t["embed"], tokens, config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        source = layer.get("weights_of")
        name = f"l{i if source is None else source}."
        x = add_normed(x, attention(t, name + "mix.", layer["mixer"], x, eps), t[name + "norm1"], mult, eps)
        if layer.get("mlp") is not None:
            x = add_normed(x, feed_forward(t, name + "mlp.", x), t[name + "norm2"], mult, eps)
        if collect is not None:
            collect.append(x)
    z = (unit_rms(x, eps) * t["final.norm"]) @ t["head"].T
    return capped(z, config.get("logit_softcap"))
