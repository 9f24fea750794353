"""Small Fuzazen configurations with random weights made here (names and shapes written out from
the configuration, independent of the engine's own list), their model folders, and the comparison
of replayed logits with the plain implementation."""

from __future__ import annotations

import copy
import functools
import json
from typing import Dict, List, Sequence, Tuple

import torch

import helpers as H
import plain_fuzazen as P


def attention(heads, kv_heads, dim, vdim, chunk, rot_dims, base=10000.0, scale=None, ff=None):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                      "rot": {"base": base, "dims": rot_dims}, "scale": dim ** -0.5 if scale is None else scale}}


def again(layer, j):
    """One more run of layer j (whose entry is `layer`) with its tensors."""
    return dict(copy.deepcopy(layer), weights_of=j)


def model(layers, width, vocab, scale=1.3, mult=0.6, cap=25.0, eps=1e-5):
    return {"architecture": "Fuzazen", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "residual_mult": mult, "logit_softcap": cap, "layers": copy.deepcopy(layers)}


def _cfg_f():
    a = attention(4, 2, 16, 24, 20, 8, ff=96)
    b = attention(6, 3, 32, 16, 33, 32, base=500.0, scale=0.4)                   # no feed-forward
    c = attention(2, 1, 64, 64, 50, 32, scale=0.3, ff=40)                       # equal heads of 64
    return model([a, b, again(a, 0), c, again(b, 1), again(a, 0)], width=64, vocab=97, scale=0.7, mult=0.4, cap=3.0)


def _cfg_g():
    # what another model makes equal or 1: a factor of 1 on what is added and on the embedding, every head its
    # own keys, one head, one key head for all, blocks as long as a page, key and value heads of one size
    a = attention(3, 3, 48, 48, 64, 16, base=50.0, ff=120)
    b = attention(8, 1, 64, 64, 100, 64, scale=0.2, ff=56)
    c = attention(1, 1, 112, 32, 7, 2, scale=0.15)
    return model([a, again(b, 2), b, c, again(c, 3)], width=96, vocab=131, scale=1.0, mult=1.0, cap=2.5, eps=1e-6)


CFG_F, CFG_G = _cfg_f(), _cfg_g()
CONFIGS = {"F": (CFG_F, 16), "G": (CFG_G, 32)}


def tensor_shapes(cfg) -> Dict[str, Tuple[int, ...]]:
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}.", layer["mixer"]
        n, g, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "mix.q": (n * d, W), p + "mix.k": (g * d, W), p + "mix.v": (g * e, W),
                    p + "mix.g": (n, W), p + "mix.o": (W, n * e), p + "mix.sink": (n,)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_tensors(cfg, seed: int) -> Dict[str, torch.Tensor]:
    """Values of a size that keeps every activation of order one; bfloat16, as files store them."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        x = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or name == "final.norm":
            x = 1.0 + 0.2 * x
        elif last == "sink":
            x = 1.5 * x
        elif last == "g":
            x = 1.5 * x / shape[1] ** 0.5
        elif len(shape) == 2 and name != "embed":
            x = x / shape[1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out


def write_folder(folder, cfg, tensors) -> None:
    from bare_cuda_4gib_b200.weights.safetensors_io import write_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    write_safetensors(folder / "model.safetensors", tensors)
    (folder / "config.json").write_text(json.dumps(cfg))


_tensors: Dict[str, Dict[str, torch.Tensor]] = {}


def register(folder, cfg, tensors) -> None:
    write_folder(folder, cfg, tensors)
    _tensors[str(folder)] = tensors


@functools.lru_cache(maxsize=None)
def model_folder(name: str, seed: int = 3):
    cfg, _page = CONFIGS[name]
    folder = H.tmp_root() / f"fuzazen{name}-{seed}"
    register(folder, cfg, random_tensors(cfg, seed))
    return folder


# Per logits row: max |got - want| / max |want| against the float64 plain implementation.  A logic
# fault (a key, a sink, a gate, a block's edge lost or shifted) shows at 1e-2 and more.
TOLERANCE = {"float32": 2e-5, "bfloat16": 5e-2}

_plain: Dict[Tuple, torch.Tensor] = {}


def plain_logits(folder, ids: Sequence[int]) -> torch.Tensor:
    key = (str(folder), tuple(ids))
    if key not in _plain:
        cfg = json.loads((folder / "config.json").read_text())
        _plain[key] = P.forward(cfg, _tensors[str(folder)], list(ids))
    return _plain[key]


def check(folder, requests: Dict[str, List[int]], got, dtype: str, expect_all: bool = True) -> float:
    worst = 0.0
    for rid, ids in requests.items():
        want = plain_logits(folder, ids)
        places = sorted(p for (r, p) in got if r == rid)
        if expect_all:
            assert places == list(range(len(ids))), f"request {rid}: places {places}"
        for p in places:
            err = H.row_error(got[(rid, p)], want[p])
            worst = max(worst, err)
            assert err <= TOLERANCE[dtype], f"request {rid} position {p} of {len(ids)}: error {err:.3e}"
    return worst


# ------------------------------------------------------------------------------ planted weights

def planted(layer, seed, name, sink=None):
    """One layer whose scores are decided by two tokens.  Token 1's embedding lies along one direction,
    which only the queries read; token 0's along a second one, which only the keys read; every other
    token's is orthogonal to both.  The query of a token 1 and the key of a token 0 point the same
    way (along entries that no rotation turns), so a token 1 finds the earlier tokens 0 that it may
    see, however far back, far above every other key: their score is dim * scale.  `sink` (None: as
    drawn): the heads' sinks."""
    cfg = model([layer], width=64, vocab=53, scale=2.0, mult=0.7, cap=20.0, eps=1e-6)
    t = {k: v.float() for k, v in random_tensors(cfg, seed).items()}
    t["embed"][:, :2] = 0.0
    t["embed"][:2] = 0.0
    t["embed"][1, 0] = 1.0
    t["embed"][0, 1] = 1.0
    m = layer["mixer"]
    d, rot = m["dim"], m["rot"]["dims"]
    way = torch.zeros(d)
    way[rot:] = 1.0
    q, k = t["l0.mix.q"].view(m["heads"], d, -1), t["l0.mix.k"].view(m["kv_heads"], d, -1)
    q[..., :2], k[..., :2] = 0.0, 0.0
    q[..., 0], k[..., 1] = way, way
    t["l0.mix.g"][:, 0] = 1.0
    if sink is not None:
        t["l0.mix.sink"][:] = torch.tensor(sink)
    t = {n: v.to(torch.bfloat16) for n, v in t.items()}
    folder = H.tmp_root() / f"fuzazen-planted-{name}"
    register(folder, cfg, t)
    return folder, cfg


def moved(folder, cfg, ids, other, at) -> float:
    """How far the logits at `at` move when the tokens are `other` instead."""
    return H.row_error(P.forward(cfg, _tensors[str(folder)], other)[at], plain_logits(folder, ids)[at])
