"""The Sizitar decoder written out plainly in float64, one function per mechanism, whole sequences
at a time and with no cache: the oracle of the engine's tests.  It shares nothing with the engine.

Notation: x [n, width] is the residual stream of one sequence whose tokens sit at positions 0..n-1,
h a sublayer's input, t a dict of the model's tensors by name, m a layer's `mixer` entry.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """The weight is stored around zero: the factor is 1 + w."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30.0, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def short_convolution(u, w):
    """u [n, channels]; w [channels, taps] whose last column meets the current token; zeros before
    the start."""
    n, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    out = torch.zeros_like(u)
    for j in range(taps):
        out = out + padded[j: j + n] * w[:, j][None, :]
    return out


# ----------------------------------------------------------------------------- the gated delta rule

def unit_vector(x, tiny=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + tiny)


def decay_per_head(t, p: str, m, h):
    """[n, heads, 1]: one factor for every row of a head's state."""
    z = softplus(h @ t[p + "a"].T + t[p + "dt_bias"])
    return torch.exp(-torch.exp(t[p + "A_log"])[None, :] * z)[:, :, None]


def decay_per_channel(t, p: str, m, h):
    """[n, heads, dim]: a factor for each of the state's key channels."""
    z = softplus((h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "dt_bias"]).view(h.shape[0], m["heads"], m["dim"])
    return torch.exp(-torch.exp(t[p + "A_log"])[None, :, None] * z)


def delta_rule(q, k, v, g, beta, start=None):
    """One head: q, k [n, dim], v [n, vdim], g [n, dim or 1], beta [n].  Returns (outputs, the state
    after the last token [dim, vdim])."""
    n, d, dv = q.shape[0], q.shape[1], v.shape[1]
    S = torch.zeros(d, dv, dtype=q.dtype) if start is None else start.clone()
    out = torch.zeros(n, dv, dtype=q.dtype)
    for i in range(n):
        S = S * g[i][:, None]
        u = beta[i] * (v[i] - S.T @ k[i])
        S = S + torch.outer(k[i], u)
        out[i] = S.T @ q[i]
    return out, S


def delta_mixer(t: Dict[str, torch.Tensor], p: str, m, h, eps, kind: str):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ t[p + x].T, t[p + x + ".conv"])) for x in "qkv")
    q = unit_vector(q.view(n, G, d)) * d ** -0.5
    k = unit_vector(k.view(n, G, d))
    v = v.view(n, H, dv)
    beta = torch.sigmoid(h @ t[p + "b"].T)
    g = decay_per_head(t, p, m, h) if kind == "delta" else decay_per_channel(t, p, m, h)
    outs = []
    for head in range(H):
        at = head // (H // G)
        outs.append(delta_rule(q[:, at], k[:, at], v[:, head], g[:, head], beta[:, head])[0])
    o = unit_rms(torch.stack(outs, 1), eps) * t[p + "norm"]
    if kind == "delta":
        gate = silu(h @ t[p + "g"].T)
    else:
        gate = torch.sigmoid((h @ t[p + "g1"].T) @ t[p + "g2"].T)
    return (o.reshape(n, H * dv) * gate) @ t[p + "o"].T


# ----------------------------------------------------------------------------- attention

def turn_neighbours(x, positions, dims, base):
    """x [n, heads, size]: entry 2i is paired with entry 2i + 1 (2i < dims) and the pair turned by
    position * base^(-2i/dims); entries from `dims` on stay."""
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * freq[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def softmax_and_one(s):
    """exp(s_j) / (1 + sum_j exp(s_j)) along the last axis."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def causal_attention(q, k, v, scale):
    """One head: q [n, d], k [n, d], v [n, dv]; key j is seen by query i when j <= i."""
    s = (q @ k.T) * scale
    p = torch.arange(q.shape[0])
    s = s.masked_fill(p[None, :] > p[:, None], -math.inf)
    return softmax_and_one(s) @ v


def attention(t: Dict[str, torch.Tensor], p: str, m, h, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_convolution(h @ t[p + x].T, t[p + x + ".conv"]) for x in "qkv")
    q = (unit_rms(q, eps) * t[p + "q.norm"]).view(n, H, d)          # one norm over all heads
    k = (unit_rms(k, eps) * t[p + "k.norm"]).view(n, G, d)
    v = v.view(n, G, dv)
    pos, rot = torch.arange(n), m["rot"]
    q, k = turn_neighbours(q, pos, rot["dims"], rot["base"]), turn_neighbours(k, pos, rot["dims"], rot["base"])
    outs = []
    for head in range(H):
        g = head // (H // G)
        outs.append(causal_attention(q[:, head], k[:, g], v[:, g], m["scale"]))
    return torch.cat(outs, -1) @ t[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward

def dense(t, p: str, h):
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def expert(t, p: str, h):
    return torch.relu(h @ t[p + "up"].T) ** 2 @ t[p + "down"].T


def route(t: Dict[str, torch.Tensor], p: str, r, h, margins: Optional[list] = None):
    """Returns (ids [n, top], weights [n, top]).  `margins` receives, per token, how far the last expert
    chosen lies above the first one left out (infinite where none is)."""
    z = h @ t[p + "router"].T + t[p + "router.b"]
    top = z.topk(r["top"], -1)
    if margins is not None:
        order = z.sort(-1, descending=True).values
        margins.append(order[:, r["top"] - 1] - order[:, r["top"]] if r["top"] < r["experts"]
                       else torch.full((h.shape[0],), math.inf, dtype=F64))
    return top.indices, torch.softmax(top.values, -1)


def mixture(t: Dict[str, torch.Tensor], p: str, mlp, h, margins: Optional[list] = None):
    ids, weights = route(t, p, mlp["router"], h, margins)
    out = expert(t, p + "shared.", h)
    for e in range(mlp["router"]["experts"]):
        rows, place = torch.nonzero(ids == e, as_tuple=True)
        if rows.numel():
            out[rows] += weights[rows, place][:, None] * expert(t, f"{p}e{e}.", h[rows])
    return out


# ----------------------------------------------------------------------------- the model

def run_order(config) -> List[int]:
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    inside = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inside * loop["times"] + list(range(loop["stop"], n))


def layer(config, t, i: int, x, margins: Optional[list] = None):
    eps, entry, p = config["norm"]["eps"], config["layers"][i], f"l{i}."
    h = norm_around_zero(x, t[p + "norm1"], eps)
    if entry["type"] == "attention":
        y = attention(t, p + "mix.", entry["mixer"], h, eps)
    else:
        y = delta_mixer(t, p + "mix.", entry["mixer"], h, eps, entry["type"])
    x = x + y * t[p + "ls1"]
    mlp = entry.get("mlp")
    if mlp is not None:
        h = norm_around_zero(x, t[p + "norm2"], eps)
        y = dense(t, p + "mlp.", h) if mlp["kind"] == "dense" else mixture(t, p + "mlp.", mlp, h, margins)
        x = x + y * t[p + "ls2"]
    return x


def forward(config, tensors: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None,
            margins: Optional[list] = None):
    """Logits [n, vocab] of one sequence; `collect` receives the stream after every layer run, `margins` the
    routers' margins (see `route`)."""
    t = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in tensors.items()}
    x = t["embed"][torch.tensor(tokens)]
    for i in run_order(config):
        x = layer(config, t, i, x, margins)
        if collect is not None:
            collect.append(x)
    return norm_around_zero(x, t["final.norm"], config["norm"]["eps"]) @ t["head"].T * config["logit_scale"]
