"""The Sizitar decoder laid out as parts.

Pre-norm layers whose sublayer results are multiplied element by element by a learned scale before they are
added (block "scaled_prenorm"); the norms' weights are stored around zero (the factor is 1 + w).  Mixers, by
the layer's `type`: "delta" and "channel_delta" (the gated delta rule behind short convolutions, with one decay
per head and a silu gate on the output, or one per key channel and a sigmoid gate, both of the latter through a
low rank), and "attention" (grouped-query softmax attention whose q, k and v pass a short convolution, whose q
and k are normed over all heads at once and turned in neighbouring pairs, with one in the softmax's
denominator).  Feed-forwards: a gated one (silu), or a mixture of ungated experts W_down relu(W_up h)^2 with a
biased router, weights from the softmax over the chosen experts, and a shared expert.  `loop` names layers
that run several times in a row, which is the model's run order.  The logits' constant rides in the final
norm's factor.

Tensor names: `embed`, `final.norm`, `head`, and per layer i `l<i>.norm1|norm2`, `l<i>.ls1|ls2`,
`l<i>.mix.q|k|v` (+ `.conv`; attention's q and k + `.norm`), `l<i>.mix.o`; delta mixers `l<i>.mix.b|A_log|
dt_bias|norm` and `.a|g` or `.a1|a2|g1|g2`; `l<i>.mlp.gate|up|down`, or `l<i>.mlp.router` (+ `.b`),
`l<i>.mlp.e<j>.up|down`, `l<i>.mlp.shared.up|down`.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sizitar import SizitarConfig
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _attention(cfg: SizitarConfig, m, p: str) -> PartSpec:
    names = {n: p + n for n in ("q", "k", "v", "o")}
    names.update({f"{n}_conv": f"{p}{n}.conv" for n in ("q", "k", "v")})
    names.update({f"{n}_norm": f"{p}{n}.norm" for n in ("q", "k")})
    return PartSpec("general_attention",
                    {"hidden": cfg.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                     "scale": m["scale"], "eps": cfg.norm_eps, "taps": m["conv"], "qk_norm": "all", "sink_score": 0.0,
                     "position": PartSpec("rotary_pairs", {"dims": m["rot"]["dims"], "base": m["rot"]["base"]})}, names)


def _delta(cfg: SizitarConfig, m, p: str, channel: bool) -> PartSpec:
    names = {n: p + n for n in ("q", "k", "v", "b", "A_log", "dt_bias", "norm", "o")}
    names.update({f"{n}_conv": f"{p}{n}.conv" for n in ("q", "k", "v")})
    names.update({n: p + n for n in (("a1", "a2", "g1", "g2") if channel else ("a", "g"))})
    return PartSpec("gated_delta",
                    {"hidden": cfg.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                     "taps": m["conv"], "eps": cfg.norm_eps, "unit_eps": 1e-6, "decay": "channel" if channel else "head",
                     "gate": "sigmoid" if channel else "silu", "rank": m.get("rank")}, names)


def _feed_forward(cfg: SizitarConfig, mlp, p: str) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("glu", {"hidden": cfg.width, "intermediate": mlp["ff"], "activation": "silu"},
                        {t: p + t for t in ("gate", "up", "down")})
    r, shared = mlp["router"], mlp.get("shared")
    names = {"router": p + "router", "router_bias": p + "router.b"}
    for e in [f"e{e}" for e in range(r["experts"])] + (["shared"] if shared else []):
        names.update({f"{e}.{t}": f"{p}{e}.{t}" for t in ("up", "down")})
    return PartSpec("moe", {"hidden": cfg.width, "experts": r["experts"], "top": r["top"], "router_scale": 1.0,
                            "intermediate": mlp["expert"]["ff"], "shared_intermediate": shared["ff"] if shared else None,
                            "shared_gate": False, "expert_form": "relu2", "router_bias": True, "weights": "chosen"}, names)


def sizitar_spec(cfg: SizitarConfig) -> ModelSpec:
    def norm(name, mult=1.0):
        return PartSpec("gated_sandwich_rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "one_plus": True, "mult": mult},
                        {"weight": name})

    def scale(name):
        return PartSpec("layer_scale", {"size": cfg.width}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        name = f"l{i}."
        m, mlp = layer["mixer"], layer.get("mlp")
        mixer = (_attention(cfg, m, name + "mix.") if layer["type"] == "attention"
                 else _delta(cfg, m, name + "mix.", layer["type"] == "channel_delta"))
        extras = {"scale1": scale(name + "ls1")}
        if mlp is not None:
            extras["scale2"] = scale(name + "ls2")
        layers.append(LayerSpec(
            mixer_norm=norm(name + "norm1"), mixer=mixer, ffn_norm=norm(name + "norm2") if mlp is not None else None,
            ffn=_feed_forward(cfg, mlp, name + "mlp.") if mlp is not None else None, block="scaled_prenorm", extras=extras))
    sizes = {"vocab": cfg.vocab, "hidden": cfg.width}
    return ModelSpec(
        architecture=SizitarConfig.ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=None,
        embed=PartSpec("table", sizes, {"weight": "embed"}), layers=layers, order=[LayerCall(i) for i in cfg.run_order()],
        final_norm=norm("final.norm", cfg.logit_scale), head=PartSpec("linear", sizes, {"weight": "head"}))


register_architecture(SizitarConfig.ARCHITECTURE, SizitarConfig, sizitar_spec)
