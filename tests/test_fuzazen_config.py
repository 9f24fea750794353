"""The Fuzazen decoder without a GPU: tensor names and shapes against a list written out
independently, the run order of layers that share tensors, what each run keeps per request,
configuration errors by key, the plain implementation's mechanisms against hand-made cases, that a
mistake in any of them moves the tests' logits, and random weights."""

import copy
import math

import pytest
import torch

import fuzazen_helpers as U
import helpers as H
import plain_fuzazen as P
from bare_cuda_4gib_b200 import models  # noqa: F401
from bare_cuda_4gib_b200.config.fuzazen import FuzazenConfig
from bare_cuda_4gib_b200.config.registry import resolve_architecture
from bare_cuda_4gib_b200.engine.model import expected_weights
from bare_cuda_4gib_b200.errors import ConfigError
from bare_cuda_4gib_b200.parts.base import KVCacheRequest

F64 = torch.float64


def _spec(cfg):
    arch = resolve_architecture(cfg)
    return arch.build_spec(arch.config_class.from_dict(cfg))


@pytest.mark.parametrize("name", ["F", "G"])
def test_tensor_names_and_shapes(name):
    cfg = U.CONFIGS[name][0]
    expected, _ = expected_weights(_spec(cfg))
    assert {k: tuple(v.shape) for k, v in expected.items()} == U.tensor_shapes(cfg)


def test_layers_that_share_tensors_run_again_with_a_cache_of_their_own():
    spec = _spec(U.CFG_F)
    assert len(spec.layers) == 3 and [c.layer for c in spec.order] == [0, 1, 0, 2, 1, 0]
    assert all(c.cache_from is None for c in spec.order)
    _, model = expected_weights(spec)
    demands = model.cache_demands()
    # a query never looks back further than one block of positions
    assert demands[0][0].kv == KVCacheRequest(2, 16, 20, v_head_dim=24) == demands[5][0].kv
    assert demands[3][0].kv == KVCacheRequest(1, 64, 50)
    from bare_cuda_4gib_b200.cache.manager import CacheManager
    cache = CacheManager(demands, page_tokens=16, max_seqs=2, max_tokens=64, allocate=False)
    assert sorted(len(g.members) for g in cache.groups) == [1, 2, 3]
    # a layer may run with a later one's tensors, and a chain of names leads to the layer that has them
    assert [c.layer for c in _spec(U.CFG_G).order] == [0, 1, 1, 2, 2]
    one = U.attention(2, 1, 8, 8, 5, 4)
    chain = U.model([U.again(one, 2), one, U.again(one, 1)], 32, 40)
    spec = _spec(chain)
    assert len(spec.layers) == 1 and [c.layer for c in spec.order] == [0, 0, 0]
    assert all(not n.startswith(("l0.", "l2.")) for n in expected_weights(spec)[0])


def test_configuration_errors_name_the_key():
    def broken(change):
        cfg = copy.deepcopy(U.CFG_F)
        change(cfg)
        with pytest.raises(ConfigError) as e:
            FuzazenConfig.from_dict(cfg)
        return str(e.value)

    assert "layers[0].mixer.kv_heads" in broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    assert "layers[0].mixer.vdim" in broken(lambda c: c["layers"][0]["mixer"].pop("vdim"))
    assert "layers[0].mixer.mask.size" in broken(lambda c: c["layers"][0]["mixer"].pop("mask"))
    assert "layers[0].mixer.mask.size" in broken(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    assert "layers[0].mixer.rot.dims" in broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    assert "layers[0].mixer.rot.dims" in broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18))
    assert "layers[0].mixer.scale" in broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    assert "layers[1].type" in broken(lambda c: c["layers"][1].update(type="mlstm"))
    assert "layers[2].weights_of" in broken(lambda c: c["layers"][2].update(weights_of=9))
    assert "layers[2].weights_of" in broken(lambda c: c["layers"][2].update(weights_of=2))
    assert "layers[2].mixer" in broken(lambda c: c["layers"][2]["mixer"].update(scale=0.9))
    assert "layers[2].mlp" in broken(lambda c: c["layers"][2].update(mlp=None))
    assert "layers[0].mlp.kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    assert "norm.eps" in broken(lambda c: c.pop("norm"))
    assert "embedding.scale" in broken(lambda c: c.pop("embedding"))
    assert "residual_mult" in broken(lambda c: c.pop("residual_mult"))
    assert "logit_softcap" in broken(lambda c: c.pop("logit_softcap"))
    assert "logit_softcap" in broken(lambda c: c.update(logit_softcap=-1.0))
    assert FuzazenConfig.from_dict(dict(U.CFG_F, logit_softcap=None)).logit_softcap is None
    for cfg in (U.CFG_F, U.CFG_G):
        assert FuzazenConfig.from_dict(cfg).to_dict() == cfg


def test_plain_mask_and_turning():
    seen = P.seen(7, 3)
    assert seen[4].tolist() == [False, False, False, True, True, False, False]
    assert seen[3].tolist() == [False, False, False, True, False, False, False]
    assert P.seen(3, None).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    # entries 2i and 2i + 1 turn together; entries from dims on stay; position 0 turns nothing
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]], [[1.0, 0.0, 0.0, 1.0, 5.0]]], dtype=F64)
    y = P.turn_pairs(x, torch.tensor([0, 2]), 100.0, 4)
    assert torch.equal(y[0], x[0])
    want = torch.tensor([math.cos(2.0), math.sin(2.0), -math.sin(0.2), math.cos(0.2), 5.0], dtype=F64)
    assert torch.allclose(y[1, 0], want)


def test_plain_sink_gate_norms_and_cap():
    s = torch.tensor([[0.0, math.log(3.0)]], dtype=F64)
    w = P.softmax_with_sink(s, torch.tensor(math.log(4.0), dtype=F64))
    assert torch.allclose(w, torch.tensor([[1.0, 3.0]], dtype=F64) / 8.0)
    assert torch.allclose(P.softmax_with_sink(s - 900.0, torch.tensor(-900.0, dtype=F64)).sum(), torch.tensor(0.8, dtype=F64))
    y = torch.tensor([[3.0, 4.0]], dtype=F64)
    out = P.add_normed(torch.ones(1, 2, dtype=F64), y, torch.tensor([1.0, 2.0], dtype=F64), 0.5, 0.0)
    assert torch.allclose(out, torch.tensor([[1.0 + 1.5 / math.sqrt(12.5), 1.0 + 4.0 / math.sqrt(12.5)]], dtype=F64))
    assert torch.allclose(P.capped(torch.tensor([0.5, 1e9], dtype=F64), 2.0), torch.tensor([2 * math.tanh(0.25), 2.0], dtype=F64))
    # one token: it sees itself and the sink, so a head is its value times e^s / (e^s + e^sink) times its gate
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 0.5, "mask": {"size": 4}, "rot": {"dims": 2, "base": 10.0}}
    one = torch.ones(1, 1, dtype=F64)
    t = {"q": torch.tensor([[3.0], [0.0]], dtype=F64), "k": torch.tensor([[0.0], [7.0]], dtype=F64), "v": 5.0 * one, "g": 0.3 * one,
         "o": one, "sink": torch.tensor([0.4], dtype=F64)}
    got = P.attention(t, "", m, one, 0.0)         # q and k of size sqrt(2) at a right angle: score 0
    assert torch.allclose(got, 5.0 * one / (1.0 + math.exp(0.4)) / (1.0 + math.exp(-0.3)))
    t["k"] = torch.tensor([[2.0], [0.0]], dtype=F64)                       # the same direction: score 2 * 0.5
    got = P.attention(t, "", m, one, 0.0)
    assert torch.allclose(got, 5.0 * one * math.e / (math.e + math.exp(0.4)) / (1.0 + math.exp(-0.3)))


MISTAKES = {
    "block_one_shorter": lambda mp: mp.setattr(P, "seen", lambda n, c, f=P.seen: f(n, c - 1)),
    "block_one_longer": lambda mp: mp.setattr(P, "seen", lambda n, c, f=P.seen: f(n, c + 1)),
    "no_blocks": lambda mp: mp.setattr(P, "seen", lambda n, c, f=P.seen: f(n, None)),
    "no_sink": lambda mp: mp.setattr(P, "softmax_with_sink", lambda s, sink: torch.softmax(s, -1)),
    "sink_twice": lambda mp: mp.setattr(P, "softmax_with_sink", lambda s, sink, f=P.softmax_with_sink: f(s, sink + math.log(2.0))),
    "sink_scaled": lambda mp: mp.setattr(P, "softmax_with_sink", lambda s, sink, f=P.softmax_with_sink: f(s, 0.5 * sink)),
    "halves_instead_of_pairs": lambda mp: mp.setattr(P, "turn_pairs", lambda x, p, b, d, f=P.turn_pairs: f(
        torch.cat([x[..., :d].unflatten(-1, (2, d // 2)).transpose(-1, -2).flatten(-2), x[..., d:]], -1), p, b, d)),
    "positions_stretched": lambda mp: mp.setattr(P, "turn_pairs", lambda x, p, b, d, f=P.turn_pairs: f(x, p * 1.03, b, d)),
    "no_gate": lambda mp: mp.setattr(P, "attention", lambda t, p, m, h, e, f=P.attention: f({**t, p + "g": 0.0 * t[p + "g"]}, p, m, h, e)),
    "no_factor_on_the_result": lambda mp: mp.setattr(P, "add_normed", lambda x, y, w, m, e, f=P.add_normed: f(x, y, w, 1.0, e)),
    "no_embedding_factor": lambda mp: mp.setattr(P, "scaled_embedding", lambda t, i, s, f=P.scaled_embedding: f(t, i, 1.0)),
    "no_cap": lambda mp: mp.setattr(P, "capped", lambda z, c: z),
}


@pytest.mark.parametrize("which", sorted(MISTAKES))
def test_a_mistake_would_show(which, monkeypatch):
    """The random weights of the GPU tests are such that each of these mistakes moves some logits far
    beyond the bfloat16 tolerance."""
    import random
    ids = H.random_ids(random.Random(2), 70, 97)
    tensors = U.random_tensors(U.CFG_F, 3)
    want = P.forward(U.CFG_F, tensors, ids)
    MISTAKES[which](monkeypatch)
    wrong = P.forward(U.CFG_F, tensors, ids)
    worst = max(H.row_error(a, b) for a, b in zip(wrong, want))
    assert worst > 1.5 * U.TOLERANCE["bfloat16"], worst


def test_random_weights_of_a_preset():
    from bare_cuda_4gib_b200.models.presets import preset_config
    from bare_cuda_4gib_b200.weights.random_init import random_tensors

    config = preset_config("fuzazen-tiny")
    expected, _ = expected_weights(resolve_architecture(config.to_dict()).build_spec(config))
    tensors = random_tensors(expected, 5)
    assert set(tensors) == set(expected)
    assert abs(float(tensors["l0.norm1"].float().mean()) - 1.0) < 0.05
