"""The Sizitar decoder without a GPU: tensor names and shapes against a list written out
independently, what every run of a layer keeps per request, the run order, configuration errors by
key, the plain implementation's mechanisms against hand-made cases, and mistakes planted in it that
must move the tests' logits."""

import copy
import math

import pytest
import torch

import plain_sizitar as P
import sizitar_helpers as U
from bare_cuda_4gib_b200 import models  # noqa: F401
from bare_cuda_4gib_b200.config.registry import resolve_architecture
from bare_cuda_4gib_b200.config.sizitar import SizitarConfig
from bare_cuda_4gib_b200.engine.model import expected_weights
from bare_cuda_4gib_b200.errors import ConfigError
from bare_cuda_4gib_b200.parts.base import KVCacheRequest, StateRequest

F64 = torch.float64


def _spec(cfg):
    arch = resolve_architecture(cfg)
    return arch.build_spec(arch.config_class.from_dict(cfg))


@pytest.mark.parametrize("name", ["A", "B"])
def test_tensor_names_and_shapes(name):
    cfg = U.CONFIGS[name][0]
    expected, _ = expected_weights(_spec(cfg))
    want = U.tensor_shapes(cfg)
    assert set(expected) == set(want)
    for key, shape in want.items():      # -1: a rank, which only the file knows
        got = tuple(expected[key].shape)
        assert len(got) == len(shape) and all(a in (b, -1) for a, b in zip(got, shape)), key
        assert -1 not in got or key.rsplit(".", 1)[-1] in ("a1", "a2", "g1", "g2")


def test_run_order_caches_and_states():
    spec = _spec(U.CFG_A)
    assert [c.layer for c in spec.order] == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert all(c.cache_from is None for c in spec.order)
    _, model = expected_weights(spec)
    demands = model.cache_demands()
    # a delta layer keeps its matrix state and the convolution's last inputs (a ring of `taps` entries), no pages
    assert [d.kv for d in demands[0]] == [None, None]
    assert demands[0][0].state == StateRequest((4, 16, 32), torch.float32)
    assert demands[0][1].state == StateRequest((3, 2 * 2 * 16 + 4 * 32), torch.float32)
    # an attention layer keeps pages with value heads of their own size, and the convolution's last taps - 1 inputs
    assert demands[1][0].kv == KVCacheRequest(2, 16, None, v_head_dim=24)
    assert demands[1][0].state == StateRequest((3, 4 * 16 + 2 * 16 + 2 * 24), torch.float32)
    from bare_cuda_4gib_b200.cache.manager import CacheManager
    cache = CacheManager(demands, page_tokens=16, max_seqs=2, max_tokens=64, allocate=False)
    assert sum(len(g.members) for g in cache.groups) == 4           # every run of an attention layer has its own
    assert len({id(s) for s in cache.states.values()}) == 4 + 2 * 5     # ... and so has every run of a delta layer
    assert [c.layer for c in _spec(U.CFG_B).order] == [0, 1, 2, 3, 4]
    for loop, want in (((0, 5, 2), [0, 1, 2, 3, 4] * 2), ((4, 5, 3), [0, 1, 2, 3, 4, 4, 4]), ((2, 2, 4), [0, 1, 2, 3, 4]),
                       ((1, 4, 1), [0, 1, 2, 3, 4])):
        cfg = dict(U.CFG_B, loop=dict(zip(("start", "stop", "times"), loop)))
        assert [c.layer for c in _spec(cfg).order] == want == P.run_order(cfg)


def test_configuration_errors_name_the_key():
    def broken(change):
        cfg = copy.deepcopy(U.CFG_A)
        change(cfg)
        with pytest.raises(ConfigError) as e:
            SizitarConfig.from_dict(cfg)
        return str(e.value)

    assert "layers[0].mixer.kv_heads" in broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    assert "layers[0].mixer.conv" in broken(lambda c: c["layers"][0]["mixer"].pop("conv"))
    assert "layers[1].mixer.scale" in broken(lambda c: c["layers"][1]["mixer"].pop("scale"))
    assert "layers[1].mixer.rot.dims" in broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))
    assert "layers[1].mixer.rot.dims" in broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18))
    assert "layers[1].mixer.rot.base" in broken(lambda c: c["layers"][1]["mixer"]["rot"].pop("base"))
    assert "layers[2].mixer.vdim" in broken(lambda c: c["layers"][2]["mixer"].pop("vdim"))
    assert "layers[3].type" in broken(lambda c: c["layers"][3].update(type="mamba2"))
    assert "layers[3].mixer" in broken(lambda c: c["layers"][3].update(mixer=None))
    assert "layers[0].mlp.router.top" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=6))
    assert "layers[0].mlp.expert.ff" in broken(lambda c: c["layers"][0]["mlp"].pop("expert"))
    assert "layers[0].mlp.shared.ff" in broken(lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"))
    assert "layers[1].mlp.ff" in broken(lambda c: c["layers"][1]["mlp"].pop("ff"))
    assert "layers[1].mlp.kind" in broken(lambda c: c["layers"][1]["mlp"].update(kind="glu"))
    assert "loop.times" in broken(lambda c: c["loop"].update(times=0))
    assert "loop.stop" in broken(lambda c: c["loop"].pop("stop"))
    assert "loop" in broken(lambda c: c["loop"].update(stop=6))
    assert "loop" in broken(lambda c: c["loop"].update(start=4))
    assert "logit_scale" in broken(lambda c: c.pop("logit_scale"))
    assert "norm.eps" in broken(lambda c: c.pop("norm"))
    assert "vocab" in broken(lambda c: c.update(vocab="many"))


def test_configuration_round_trip_and_random_weights(tmp_path):
    from bare_cuda_4gib_b200.models.presets import preset_config
    from bare_cuda_4gib_b200.weights.random_init import write_random_model
    from bare_cuda_4gib_b200.weights.safetensors_io import SafetensorsFile
    cfg = preset_config("sizitar-tiny")
    assert SizitarConfig.from_dict(cfg.to_dict()) == cfg
    write_random_model(tmp_path, cfg, seed=1)
    with SafetensorsFile(tmp_path / "model.safetensors") as f:
        tensors = {name: f.tensor(name) for name in f.entries}
    logits = P.forward(cfg.to_dict(), tensors, [3, 1, 4, 1, 5, 9, 2, 6])
    assert torch.isfinite(logits).all() and float(logits.std()) > 0


# ------------------------------------------------------------------------- the plain mechanisms by hand

def test_plain_delta_rule_by_hand():
    one = lambda *v: torch.tensor([v], dtype=F64)
    # one key channel, one value column: S = 0.5 S; u = beta (v - S k); S += k u; o = S q
    q, k, v = one(2.0, 1.0, 1.0).T, one(1.0, 1.0, -1.0).T, one(4.0, 0.0, 2.0).T
    g, beta = torch.full((3, 1), 0.5, dtype=F64), torch.tensor([1.0, 0.5, 1.0], dtype=F64)
    out, S = P.delta_rule(q, k, v, g, beta)
    # t0: u = 4, S = 4, o = 8.  t1: S = 2, u = -1, S = 1, o = 1.  t2: S = 0.5, u = 2 + 0.5, S = 0.5 - 2.5 = -2, o = -2
    assert out.view(-1).tolist() == [8.0, 1.0, -2.0] and S.item() == -2.0
    # with beta 1, no decay and a unit key, a key written again forgets what it held
    k = torch.tensor([[0.6, 0.8], [0.6, 0.8]], dtype=F64)
    v = torch.tensor([[5.0, -1.0, 2.0], [7.0, 3.0, 1.0]], dtype=F64)
    out, S = P.delta_rule(k, k, v, torch.ones(2, 1, dtype=F64), torch.ones(2, dtype=F64))
    assert torch.allclose(out, v) and torch.allclose(S, torch.outer(k[0], v[1]))
    # a decay per channel acts on the rows of S that belong to key channels
    k = torch.tensor([[1.0, 0.0], [0.0, 0.0]], dtype=F64)
    g = torch.tensor([[1.0, 1.0], [0.25, 0.5]], dtype=F64)
    _, S = P.delta_rule(k, k, torch.tensor([[8.0], [0.0]], dtype=F64), g, torch.ones(2, dtype=F64))
    assert S.view(-1).tolist() == [2.0, 0.0]


def test_plain_pieces_by_hand():
    u = torch.tensor([[1.0], [2.0], [3.0]], dtype=F64)
    w = torch.tensor([[10.0, 1.0]], dtype=F64)      # the last column meets the current token
    assert P.short_convolution(u, w).view(-1).tolist() == [1.0, 12.0, 23.0]
    x = torch.tensor([3.0, 4.0], dtype=F64)
    assert torch.allclose(P.unit_vector(x, 0.0), torch.tensor([0.6, 0.8], dtype=F64))
    assert torch.allclose(P.unit_rms(x, 0.0), x / math.sqrt(12.5))
    s = torch.tensor([[0.0, math.log(3.0)]], dtype=F64)
    assert torch.allclose(P.softmax_and_one(s), torch.tensor([[0.2, 0.6]], dtype=F64))      # 1 + 1 + 3 below
    assert torch.allclose(P.softmax_and_one(torch.full((1, 3), -50.0, dtype=F64)), torch.zeros(1, 3, dtype=F64), atol=1e-12)
    # pairs of neighbours, position 1, first pair by one radian, the rest stays
    x = torch.tensor([1.0, 0.0, 1.0, 0.0, 9.0], dtype=F64).view(1, 1, 5)
    got = P.turn_neighbours(x, torch.tensor([1]), 4, 100.0).view(-1)
    want = [math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1), 9.0]
    assert torch.allclose(got, torch.tensor(want, dtype=F64))
    t = {"r.router": torch.eye(3, dtype=F64), "r.router.b": torch.tensor([0.0, 1.0, 0.0], dtype=F64)}
    ids, weights = P.route(t, "r.", {"experts": 3, "top": 2}, torch.tensor([[1.0, 0.5, -2.0]], dtype=F64))
    assert ids.tolist() == [[1, 0]]
    a, b = math.exp(1.5), math.exp(1.0)
    assert torch.allclose(weights, torch.tensor([[a / (a + b), b / (a + b)]], dtype=F64))


# ------------------------------------------------------------------------- planted mistakes

def _forward(cfg, tensors, ids):
    return P.forward(cfg, tensors, ids)


def _moved(monkeypatch, patches, name="A", n=70, change=None):
    """How far a mistake moves the logits of a random request, rows in the unit of the tests' errors."""
    import random
    cfg = U.CONFIGS[name][0]
    tensors = U.random_tensors(cfg, 3)
    rng = random.Random(5)
    ids = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    want = P.forward(cfg, tensors, ids)
    for attr, fn in patches.items():
        monkeypatch.setattr(P, attr, fn)
    wrong_cfg = copy.deepcopy(cfg)
    if change:
        change(wrong_cfg)
    got = P.forward(wrong_cfg, tensors, ids)
    return float(((got - want).abs().amax(-1) / want.abs().amax(-1)).max())


def _delta_rule_reading_before(q, k, v, g, beta, start=None):
    n, d, dv = q.shape[0], q.shape[1], v.shape[1]
    S, out = torch.zeros(d, dv, dtype=q.dtype), torch.zeros(n, dv, dtype=q.dtype)
    for i in range(n):
        S = S * g[i][:, None]
        out[i] = S.T @ q[i]
        S = S + torch.outer(k[i], beta[i] * (v[i] - S.T @ k[i]))
    return out, S


def _delta_rule_decay_last(q, k, v, g, beta, start=None):
    n, d, dv = q.shape[0], q.shape[1], v.shape[1]
    S, out = torch.zeros(d, dv, dtype=q.dtype), torch.zeros(n, dv, dtype=q.dtype)
    for i in range(n):
        u = beta[i] * (v[i] - S.T @ k[i])
        S = S * g[i][:, None] + torch.outer(k[i], u)
        out[i] = S.T @ q[i]
    return out, S


def _delta_rule_plain_writes(q, k, v, g, beta, start=None):
    n, d, dv = q.shape[0], q.shape[1], v.shape[1]
    S, out = torch.zeros(d, dv, dtype=q.dtype), torch.zeros(n, dv, dtype=q.dtype)
    for i in range(n):
        S = S * g[i][:, None] + torch.outer(k[i], beta[i] * v[i])
        out[i] = S.T @ q[i]
    return out, S


def _halves(x, positions, dims, base):
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * freq
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., : dims // 2], x[..., dims // 2: dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


def _route_all_softmax(t, p, r, h, margins=None):
    z = h @ t[p + "router"].T + t[p + "router.b"]
    s = torch.softmax(z, -1).topk(r["top"], -1)
    return s.indices, s.values


_ROUTE, _CONV, _NORM = P.route, P.short_convolution, P.norm_around_zero

MISTAKES = {
    "read_before_write": {"delta_rule": _delta_rule_reading_before},
    "decay_after_the_write": {"delta_rule": _delta_rule_decay_last},
    "writes_without_the_difference": {"delta_rule": _delta_rule_plain_writes},
    "plain_softmax": {"softmax_and_one": lambda s: torch.softmax(s, -1)},
    "turned_in_halves": {"turn_neighbours": _halves},
    "weights_from_all_experts": {"route": _route_all_softmax},
    "router_without_bias": {"route": lambda t, p, r, h, margins=None: _ROUTE({**t, p + "router.b": 0.0 * t[p + "router.b"]}, p, r, h)},
    "taps_reversed": {"short_convolution": lambda u, w: _CONV(u, w.flip(-1))},
    "last_tap_only": {"short_convolution": lambda u, w: u * w[:, -1]},
    "norm_weights_used_as_stored": {"norm_around_zero": lambda x, w, eps: P.unit_rms(x, eps) * w},
    "keys_and_queries_of_any_length": {"unit_vector": lambda x, tiny=1e-6: x},
}


@pytest.mark.parametrize("which", sorted(MISTAKES))
def test_a_planted_mistake_shows(which, monkeypatch):
    assert _moved(monkeypatch, MISTAKES[which]) > 2 * U.TOLERANCE["bfloat16"]


def test_a_wrong_size_or_constant_shows(monkeypatch):
    assert _moved(monkeypatch, {}, change=lambda c: c.update(loop=None)) > 0.1
    assert _moved(monkeypatch, {}, change=lambda c: c.update(logit_scale=0.5)) > 0.1
    assert _moved(monkeypatch, {}, change=lambda c: c["layers"][1]["mixer"].update(scale=0.25)) > 0.01
    assert _moved(monkeypatch, {}, change=lambda c: c["layers"][1]["mixer"]["rot"].update(base=10000.0)) > 0.01
    assert _moved(monkeypatch, {}, change=lambda c: c["layers"][0]["mlp"]["router"].update(top=3)) > 0.01
