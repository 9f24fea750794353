"""Small Sizitar configurations with random weights made here (names and shapes written out from
the configuration, independent of the engine's own list), their model folders, and the comparison
of replayed logits with the plain implementation."""

from __future__ import annotations

import copy
import functools
import json
from typing import Dict, List, Sequence, Tuple

import torch

import helpers as H
import plain_sizitar as P


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
            "shared": {"ff": ff if shared is None else shared}}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def channel_delta(heads, kv_heads, dim, vdim, conv, rank, mlp=None):
    """`rank` = (of the decays, of the gate) or one number for both; the configuration itself does not state it."""
    ranks = (rank, rank) if isinstance(rank, int) else rank
    return {"type": "channel_delta", "mlp": mlp, "test_ranks": list(ranks),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv_heads, dim, vdim, conv, rot_dims, base=10000.0, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                      "rot": {"base": base, "dims": rot_dims}, "scale": dim ** -0.5 if scale is None else scale}}


def config(layers, vocab, width, eps=1e-6, logit_scale=1.0, loop=None):
    return {"architecture": "Sizitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": copy.deepcopy(layers)}


def _cfg_a():
    layers = [channel_delta(4, 2, 16, 32, 3, 8, mlp=moe(5, 2, 24, 40)),
              attention(4, 2, 16, 24, 4, 8, base=500.0, scale=0.3, mlp=dense(48)),
              delta(6, 2, 24, 16, 2, mlp=moe(3, 1, 16)),
              attention(3, 3, 32, 32, 2, 32, scale=0.2),                          # no feed-forward
              delta(2, 2, 10, 6, 5, mlp=dense(40))]                               # sizes that line up with nothing
    return config(layers, 97, 64, eps=1e-5, logit_scale=0.7, loop=(1, 3, 3))


def _cfg_b():
    # what another model makes equal or 1: one head, a convolution of one tap, every expert chosen, no loop
    layers = [delta(1, 1, 32, 48, 1, mlp=dense(80)),
              channel_delta(3, 1, 32, 16, 4, (16, 24), mlp=moe(4, 4, 8, 16)),
              attention(6, 1, 64, 64, 1, 2, base=20.0, scale=0.1, mlp=moe(7, 3, 32)),
              channel_delta(2, 2, 48, 64, 2, 5),
              attention(2, 1, 128, 16, 3, 64, mlp=dense(24))]
    return config(layers, 131, 96, logit_scale=3.0)


CFG_A, CFG_B = _cfg_a(), _cfg_b()
CONFIGS = {"A": (CFG_A, 16), "B": (CFG_B, 32)}


def every_expert_chosen(cfg):
    """The same model with routers that choose every expert: a router's choice is a discontinuity, and where two
    logits nearly tie the rounding of a bfloat16 run may pick the other expert, which says nothing about the
    kernels.  bfloat16 runs are compared on this variant, with the same tensors; the choice itself is compared
    in float32, where a tie within rounding is rare enough to be drawn around (`clear_ids`)."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer.get("mlp") is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


def config_for(name: str, dtype: str):
    cfg, page = CONFIGS[name]
    return (every_expert_chosen(cfg) if dtype == "bfloat16" else cfg), page


def tensor_shapes(cfg) -> Dict[str, Tuple[int, ...]]:
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        n, g, d, e, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        out.update({p + "norm1": (W,), p + "ls1": (W,)})
        values = g * e if layer["type"] == "attention" else n * e
        queries = n * d if layer["type"] == "attention" else g * d
        for name, rows in (("q", queries), ("k", g * d), ("v", values)):
            out.update({f"{p}mix.{name}": (rows, W), f"{p}mix.{name}.conv": (rows, taps)})
        out[p + "mix.o"] = (W, n * e)
        if layer["type"] == "attention":
            out.update({p + "mix.q.norm": (n * d,), p + "mix.k.norm": (g * d,)})
        else:
            out.update({p + "mix.b": (n, W), p + "mix.A_log": (n,), p + "mix.norm": (e,)})
        if layer["type"] == "delta":
            out.update({p + "mix.a": (n, W), p + "mix.dt_bias": (n,), p + "mix.g": (n * e, W)})
        elif layer["type"] == "channel_delta":
            ra, rg = layer["test_ranks"]
            out.update({p + "mix.a1": (ra, W), p + "mix.a2": (n * d, ra), p + "mix.dt_bias": (n * d,),
                        p + "mix.g1": (rg, W), p + "mix.g2": (n * e, rg)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        out.update({p + "norm2": (W,), p + "ls2": (W,)})
        if mlp["kind"] == "dense":
            out.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
            continue
        r = mlp["router"]
        out.update({p + "mlp.router": (r["experts"], W), p + "mlp.router.b": (r["experts"],)})
        for e_, ff in [(f"e{j}", mlp["expert"]["ff"]) for j in range(r["experts"])] + [("shared", mlp["shared"]["ff"])]:
            out.update({f"{p}mlp.{e_}.up": (ff, W), f"{p}mlp.{e_}.down": (W, ff)})
    return out


def random_tensors(cfg, seed: int) -> Dict[str, torch.Tensor]:
    """Values of a size that keeps every activation of order one; bfloat16, as files store them."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        x = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or name == "final.norm":
            x = 0.2 * x                                   # stored around zero
        elif last == "norm":
            x = 1.0 + 0.2 * x
        elif last in ("ls1", "ls2"):
            x = 0.6 + 0.2 * x
        elif name.endswith("router.b"):
            x = 0.5 * x
        elif last == "router":
            x = 2.0 * x / shape[1] ** 0.5
        elif last == "conv":
            x = x / shape[1] ** 0.5
        elif last == "A_log":
            x = 0.8 * x - 1.0
        elif last == "dt_bias":
            x = x - 1.0
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


@functools.lru_cache(maxsize=None)
def model_folder(name: str, seed: int = 3, dtype: str = "float32"):
    """The folder of configuration `name`; for bfloat16 runs the variant whose routers choose every expert."""
    cfg, _page = config_for(name, dtype)
    folder = H.tmp_root() / f"sizitar{name}-{seed}-{dtype}"
    register(folder, cfg, random_tensors(CONFIGS[name][0], seed))
    return folder


def register(folder, cfg, tensors) -> None:
    write_folder(folder, cfg, tensors)
    _tensors[str(folder)] = tensors


# Per logits row: max |got - want| / max |want| against the float64 plain implementation.  A logic fault (a
# key, a state, a tap of the convolution, an expert, a decay, the one in the denominator lost or shifted)
# shows at 1e-2 and more in float32, where every row has to be within the tolerance.  A bfloat16 run has to
# have `BF16_SHARE` of its rows within the tolerance and none beyond `BF16_WORST`.
TOLERANCE = {"float32": 1e-4, "bfloat16": 6e-2}
BF16_SHARE, BF16_WORST = 0.95, 0.3

_plain: Dict[Tuple, torch.Tensor] = {}


def plain_logits(folder, ids: Sequence[int]) -> torch.Tensor:
    key = (str(folder), tuple(ids))
    if key not in _plain:
        cfg = json.loads((folder / "config.json").read_text())
        _plain[key] = P.forward(cfg, _tensors[str(folder)], list(ids))
    return _plain[key]


CLEAR_MARGIN = 2e-4


def clear_ids(folder, rng, n: int, vocab: int) -> List[int]:
    """`n` random ids on which no router of the model in `folder` makes a close call (one that float32 rounding
    could decide the other way): such a draw is thrown away and the next one taken."""
    cfg = json.loads((folder / "config.json").read_text())
    for _ in range(200):
        ids = H.random_ids(rng, n, vocab)
        margins: list = []
        logits = P.forward(cfg, _tensors[str(folder)], ids, None, margins)
        if all(float(m.min()) > CLEAR_MARGIN for m in margins):
            _plain[(str(folder), tuple(ids))] = logits
            return ids
    raise AssertionError("no draw without a close call of a router")


def check(folder, requests: Dict[str, List[int]], got, dtype: str, expect_all: bool = True) -> None:
    errors = []
    for rid, ids in requests.items():
        want = plain_logits(folder, ids)
        places = sorted(p for (r, p) in got if r == rid)
        if expect_all:
            assert places == list(range(len(ids))), f"request {rid}: places {places}"
        for p in places:
            err = H.row_error(got[(rid, p)], want[p])
            assert err == err, f"request {rid} position {p}: not a number"
            errors.append(err)
            if dtype == "float32":
                assert err <= TOLERANCE[dtype], f"request {rid} position {p} of {len(ids)}: error {err:.3e}"
    if dtype != "float32":
        errors.sort()
        over = sum(e > TOLERANCE[dtype] for e in errors)
        assert errors[-1] <= BF16_WORST, f"worst row: error {errors[-1]:.3e}"
        assert over <= (1.0 - BF16_SHARE) * len(errors) or over <= 1, \
            f"{over} of {len(errors)} rows beyond {TOLERANCE[dtype]:.0e}: {errors[-5:]}"
