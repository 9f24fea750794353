"""The Fuzazen decoder laid out as parts.

The embedding is multiplied by a constant.  A sublayer reads the residual stream itself, without a norm
ahead of it, and its result is RMS-normed and multiplied by a constant before it is added:
x <- x + m * norm(f(x)), first with the mixer and then, where the layer has one, with a gated (silu)
feed-forward.  That is the "sandwich" block with nothing but the hand-over of the stream on its inner
side (norm "stream_input").  The mixer is grouped-query softmax attention inside blocks of positions:
pairwise rotation of the first entries of queries and keys, both then divided by their root mean square
per head, values of their own size, a learned sink per head in the softmax's denominator, and one
sigmoid gate per head on its output.  The logits are capped with a tanh.  A layer that names another with
`weights_of` is a second run of that layer's parts with a cache of its own, so the model's run order
names that layer again.

Tensor names: `embed`, `final.norm`, `head`, and per layer i with tensors of its own `l<i>.norm1|norm2`,
`l<i>.mix.q|k|v|g|o|sink`, `l<i>.mlp.gate|up|down`.
"""

from __future__ import annotations

from ..config.fuzazen import FuzazenConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _attention(cfg: FuzazenConfig, m, p: str) -> PartSpec:
    return PartSpec("general_attention",
                    {"hidden": cfg.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                     "scale": m["scale"], "eps": cfg.norm_eps, "unit_qk": True, "chunk": m["mask"]["size"], "sink": True,
                     "head_gate": True,
                     "position": PartSpec("rotary_pairs", {"dims": m["rot"]["dims"], "base": m["rot"]["base"]})},
                    {n: p + n for n in ("q", "k", "v", "g", "o", "sink")})


def fuzazen_spec(cfg: FuzazenConfig) -> ModelSpec:
    def norm(name, mult=1.0):
        return PartSpec("sandwich_rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "mult": mult}, {"weight": name})

    stream = PartSpec("stream_input", {"size": cfg.width})
    layers, own = [], {}
    for i, layer in enumerate(cfg.layers):
        if cfg.source(i) != i:
            continue
        name = f"l{i}"
        mlp = layer.get("mlp")
        extras = {"post1": norm(name + ".norm1", cfg.residual_mult)}
        if mlp is not None:
            extras["post2"] = norm(name + ".norm2", cfg.residual_mult)
        own[i] = len(layers)
        layers.append(LayerSpec(
            mixer_norm=stream, mixer=_attention(cfg, layer["mixer"], name + ".mix."),
            ffn_norm=stream if mlp is not None else None,
            ffn=PartSpec("glu", {"hidden": cfg.width, "intermediate": mlp["ff"], "activation": "silu"},
                         {t: f"{name}.mlp.{t}" for t in ("gate", "up", "down")}) if mlp is not None else None,
            block="sandwich", extras=extras))
    sizes = {"vocab": cfg.vocab, "hidden": cfg.width}
    return ModelSpec(
        architecture=FuzazenConfig.ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=None,
        embed=PartSpec("table_positions", dict(sizes, scale=cfg.embedding_scale, positions=None, streams=1), {"weight": "embed"}),
        layers=layers, order=[LayerCall(own[cfg.source(i)]) for i in range(len(cfg.layers))], final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(sizes, softcap=cfg.logit_softcap), {"weight": "head"}))


register_architecture(FuzazenConfig.ARCHITECTURE, FuzazenConfig, fuzazen_spec)
