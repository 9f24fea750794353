"""Causal grouped-query attention over the paged cache.

q = h Wq^T, k = h Wk^T, v = h Wv^T (no bias); q and k rotated by position; k and v appended to
the request's cache pages; scores (q . k) / sqrt(head_dim) over the keys at positions
<= the query's (and, with `window`, newer than position - window); softmax; weighted values;
output projection (cuongvng/bare-cuda-4gib engine/src/model.cpp:540-572,
engine/kernels/attention_qk.cu:49-68, softmax.cu:28-42, attention_av.cu:24-44).
The three projections are one matrix product against [Wq; Wk; Wv], fused at load.

params: `hidden`, `heads`, `kv_heads`, `head_dim`, `window` (None = every key), `position`
(a `PartSpec` of the position family).  tensors: `q`, `k`, `v`, `o`.
"""

from __future__ import annotations

import math

import torch

from ..errors import ConfigError
from ..kernels import lib as K
from .base import KVCacheRequest, Part, StateRequest
from .linear import Linear
from .registry import build_part, register_mixer
from ..weights.loader import fused_rows


@register_mixer("attention")
class Attention(Part):
    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden, self.heads, self.kv_heads, self.head_dim = (
            int(p["hidden"]), int(p["heads"]), int(p["kv_heads"]), int(p["head_dim"]))
        self.window = p.get("window")
        if self.heads % self.kv_heads:
            raise ConfigError(f"attention: {self.heads} heads cannot share {self.kv_heads} key/value heads")
        self.position = build_part("position", p["position"])
        self.scale = 1.0 / math.sqrt(self.head_dim)

    def children(self):
        return [self.position]

    def local_weights(self):
        qd, kvd = self.heads * self.head_dim, self.kv_heads * self.head_dim
        return {"q": ((qd, self.hidden), "matrix"), "k": ((kvd, self.hidden), "matrix"),
                "v": ((kvd, self.hidden), "matrix"), "o": ((self.hidden, qd), "matrix")}

    def adjacent_weights(self):
        return [("q", "k", "v")]

    def cache_request(self):
        return KVCacheRequest(self.kv_heads, self.head_dim, self.window)

    def state_request(self):
        return None

    def prepare(self, dtype, device) -> None:
        t = self.tensors
        self.qkv = Linear(fused_rows([t.pop("q"), t.pop("k"), t.pop("v")]), "qkv")
        self.o = Linear(t.pop("o"), "o")
        self.qkv.prepare(dtype)
        self.o.prepare(dtype)
        self.position.prepare(dtype, device)
        if dtype == torch.bfloat16 and device.type == "cuda":
            from ..kernels import attention as fast
            self.fast = fast.plan_for(self.head_dim, self.heads, self.kv_heads)
        else:
            self.fast = None

    def plan_step(self, ctx) -> None:
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.step_tiles(ctx, self.fast)

    takes_lazy_input = True

    def forward(self, ctx, call, h):
        n = ctx.n_tokens
        qd = self.heads * self.head_dim
        # few rows: float32 partial results let the product split its inner dimension over more SMs
        qkv_dtype = torch.float32 if n <= 256 else ctx.dtype
        q = ctx.ws.get("q", (n, qd), ctx.dtype)
        inv_freq = self.position.fused_rotation()
        apply = getattr(self.position, "apply", None)
        if apply is not None:
            # a position encoding with kernels of its own: it changes q and k in place, as [tokens, heads,
            # head_dim] views of the finished projection, before k and v go into the cache
            qkv = self.qkv.forward(ctx, h, n, ctx.dtype, "qkv")
            kvd = self.kv_heads * self.head_dim
            apply(ctx, qkv.tensor[:, :qd].unflatten(1, (self.heads, self.head_dim)),
                  qkv.tensor[:, qd: qd + kvd].unflatten(1, (self.kv_heads, self.head_dim)))
        else:
            rotate = K.RotateAndCache(q, call.cache, ctx.positions, ctx.row_seq, inv_freq, self.heads, call.writes_cache)
            qkv = self.qkv.forward(ctx, h, n, qkv_dtype, "qkv", allow_partials=True, epilogue=rotate)
        if qkv is not None:
            K.rope_cache_write(qkv, q, call.cache, ctx.positions, ctx.row_seq, inv_freq, self.heads,
                               call.writes_cache, n, ctx.stream)
        out = ctx.ws.get("attn_out", (n, qd), ctx.dtype)
        window = int(self.window) if self.window else 0
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.run(ctx, self.fast, q, out, call.cache, self.scale, window)
        else:
            K.attention_plain(q, out, call.cache, ctx.positions, ctx.row_seq, self.heads, n,
                              self.scale, window, ctx.stream)
        residual = getattr(ctx, "residual", None)
        return self.o.forward(ctx, out, n, torch.float32, "attn_proj", allow_partials=True,
                              epilogue=K.AddTo(residual, getattr(ctx, "following_norm", None)) if residual is not None else None)


@register_mixer("gated_attention")
class GatedAttention(Part):
    """Grouped-query softmax attention whose queries and keys are RMS-normed per head (one weight
    per projection, shared by its heads) before the position encoding turns them, whose scores are
    (q . k) * `scale`, and whose concatenated heads are multiplied by sigmoid(Wg h) before the output
    projection.  With `values` = "keys" there is no value projection: a token's value is its key as
    projected, before norm and rotation.  `window` (None = every key) keeps the last positions.

    One product makes [q | k (| v) | g]; one kernel norms, turns and caches; then the engine's paged
    attention kernels run as they do for "attention".

    params: `hidden`, `heads`, `kv_heads`, `head_dim`, `window`, `scale`, `eps`, `values`
    ("keys" | "projection"), `position` (a `PartSpec`; "rotary_pairs" or "none").
    tensors: `q`, `k`, (`v`,) `g`, `o`, `q_norm` [head_dim], `k_norm` [head_dim]."""

    takes_lazy_input = False

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden, self.heads, self.kv_heads, self.head_dim = (
            int(p["hidden"]), int(p["heads"]), int(p["kv_heads"]), int(p["head_dim"]))
        self.window = p.get("window")
        self.own_values = p.get("values", "projection") != "keys"
        if self.heads % self.kv_heads:
            raise ConfigError(f"gated_attention: {self.heads} heads cannot share {self.kv_heads} key/value heads")
        self.position = build_part("position", p["position"])
        self.scale = float(p.get("scale") or 1.0 / math.sqrt(self.head_dim))
        self.eps = float(p["eps"])

    def children(self):
        return [self.position]

    def _projections(self):
        return ("q", "k", "v", "g") if self.own_values else ("q", "k", "g")

    def local_weights(self):
        qd, kvd = self.heads * self.head_dim, self.kv_heads * self.head_dim
        out = {"q": ((qd, self.hidden), "matrix"), "k": ((kvd, self.hidden), "matrix"),
               "g": ((qd, self.hidden), "matrix"), "o": ((self.hidden, qd), "matrix"),
               "q_norm": ((self.head_dim,), "norm"), "k_norm": ((self.head_dim,), "norm")}
        if self.own_values:
            out["v"] = ((kvd, self.hidden), "matrix")
        return out

    def adjacent_weights(self):
        return [self._projections()]

    def cache_request(self):
        return KVCacheRequest(self.kv_heads, self.head_dim, self.window)

    def state_request(self):
        return None

    def prepare(self, dtype, device) -> None:
        t = self.tensors
        self.proj = Linear(fused_rows([t[n] for n in self._projections()]), "gated_attention.in")
        self.o = Linear(t["o"], "gated_attention.o")
        self.proj.prepare(dtype)
        self.o.prepare(dtype)
        self.q_norm, self.k_norm = t["q_norm"].to(dtype).contiguous(), t["k_norm"].to(dtype).contiguous()
        self.position.prepare(dtype, device)
        self.inv_freq = getattr(self.position, "inv_freq", None)
        self.rot_dims = int(getattr(self.position, "dims", 0)) if self.inv_freq is not None else 0
        if self.rot_dims > self.head_dim:
            raise ConfigError(f"gated_attention: {self.rot_dims} rotated entries in a head of {self.head_dim}")
        self.magnitude = float(getattr(self.position, "magnitude", 1.0))
        self.fast = None
        if dtype == torch.bfloat16 and device.type == "cuda":
            from ..kernels import attention as fast
            self.fast = fast.plan_for(self.head_dim, self.heads, self.kv_heads)

    def plan_step(self, ctx) -> None:
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.step_tiles(ctx, self.fast)

    def forward(self, ctx, call, h):
        from ..kernels import head_prepare as HP
        n = ctx.n_tokens
        qd, kvd = self.heads * self.head_dim, self.kv_heads * self.head_dim
        u = self.proj.forward(ctx, h, n, ctx.dtype, "mixer_in").tensor
        q = ctx.ws.get("q", (n, qd), ctx.dtype)
        HP.headnorm_rope_cache(ctx, u, 0, qd, qd + kvd if self.own_values else -1, self.q_norm, self.k_norm, self.eps,
                               self.inv_freq, self.rot_dims, self.magnitude, q, call.cache, self.heads, call.writes_cache)
        out = ctx.ws.get("attn_out", (n, qd), ctx.dtype)
        window = int(self.window) if self.window else 0
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.run(ctx, self.fast, q, out, call.cache, self.scale, window)
        else:
            K.attention_plain(q, out, call.cache, ctx.positions, ctx.row_seq, self.heads, n, self.scale, window, ctx.stream)
        HP.sigmoid_gate(ctx, out, u[:, u.shape[1] - qd:], n)
        return self.o.forward(ctx, out, n, torch.float32, "attn_proj", allow_partials=True)


@register_mixer("general_attention")
class GeneralAttention(Part):
    """Grouped-query causal softmax attention with the options several designs combine: biases on the
    q, k and v projections; an RMS norm per head on q and k (one weight per projection, used as stored)
    before the rotation; any position part that the norm-and-cache kernel turns (`rotary_halves`,
    `rotary_pairs`, `none`); a `scale` of its own; a cap on the scaled scores, cap * tanh(score / cap);
    value heads of their own size; a `window`; and value mixing: with `v_mix` = "source" the values this
    layer caches are also left for later layers of the step, with "mix" the cached value is (1 - l) v +
    l v_source of the same token, l the scalar tensor `v_lambda`; queries and keys divided by their root
    mean square per head after the rotation (`unit_qk`, without weights); blocks of positions (`chunk`: a
    query sees its own block only, blocks counted from position 0); a learned number per head whose
    exponential joins the softmax's denominator (`sink`); and one sigmoid gate per head on its output,
    read from the mixer's input (`head_gate`); a short causal convolution over time on every channel of q, k
    and v ahead of norm and rotation (`taps`: its length; the last taps - 1 projected rows of a request are its
    state); `qk_norm` "all", one RMS norm over all heads of q and one over all heads of k, with a weight per
    channel (with `taps`); and a constant in the place of the learned sink (`sink_score`: 0 adds one to the
    denominator).

    One product makes [q | k | v (| g)]; one kernel adds the biases, norms, turns, mixes and caches; then the
    engine's tensor-core attention kernels run in bfloat16 steps (all three for equal key and value sizes
    without a cap, the mma.sync kernel built for the value size and the cap otherwise), the plain kernel in
    float32 steps and for sizes that are no multiples of 16 up to 128.  All of them join the sink and apply
    the gate where they finish a row.

    params: `hidden`, `heads`, `kv_heads`, `dim`, `vdim`, `scale`, `eps`, `bias` (bool), `qk_norm` (bool or
    "all"), `unit_qk` (bool), `softcap` (None: no cap), `window`, `chunk` (None: every key), `sink` (bool),
    `sink_score` (None: no constant), `head_gate` (bool), `v_mix` (None | "source" | "mix"), `taps` (None: no
    convolution), `position`.
    tensors: `q`, `k`, `v`, `o`, (`q_bias`, `k_bias`, `v_bias`,) (`q_norm`, `k_norm` [dim], or [channels] for
    "all",) (`q_conv`, `k_conv`, `v_conv` [channels, taps],) (`v_lambda` [],) (`sink` [heads],) (`g` [heads, hidden])."""

    takes_lazy_input = False

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim = int(p["dim"]), int(p.get("vdim") or p["dim"])
        if self.heads % self.kv_heads:
            raise ConfigError(f"general_attention: {self.heads} heads cannot share {self.kv_heads} key/value heads")
        if self.vdim > 256:
            raise ConfigError(f"general_attention: value head size {self.vdim} exceeds the 256 the kernels take")
        self.window = p.get("window")
        self.chunk = p.get("chunk")
        self.has_bias, self.qk_norm, self.unit_qk = bool(p.get("bias")), bool(p.get("qk_norm")), bool(p.get("unit_qk"))
        if self.qk_norm and self.unit_qk:
            raise ConfigError("general_attention: queries and keys are normed with weights or without, not both")
        self.has_sink, self.head_gate = bool(p.get("sink")), bool(p.get("head_gate"))
        self.sink_score = p.get("sink_score")
        if self.has_sink and self.sink_score is not None:
            raise ConfigError("general_attention: the sink is learned or a constant, not both")
        self.norm_all, self.taps = p.get("qk_norm") == "all", int(p.get("taps") or 0)
        # the kernel with the convolution norms over all heads and has none of the other steps ahead of the scores
        if self.norm_all != (self.taps > 0) or (self.taps and (self.has_bias or self.unit_qk or p.get("v_mix"))):
            raise ConfigError("general_attention: a convolution (`taps`) goes with qk_norm 'all' and without biases, "
                              "unit_qk and v_mix")
        self.softcap = float(p["softcap"]) if p.get("softcap") else 0.0
        self.v_mix = p.get("v_mix")
        if self.v_mix not in (None, "source", "mix"):
            raise ConfigError(f"general_attention: v_mix must be None, 'source' or 'mix', got {self.v_mix!r}")
        self.position = build_part("position", p["position"])
        self.scale = float(p.get("scale") or 1.0 / math.sqrt(self.dim))
        self.eps = float(p.get("eps", 1e-6))
        self.qd, self.kd, self.vd = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim

    def children(self):
        return [self.position]

    def local_weights(self):
        out = {"q": ((self.qd, self.hidden), "matrix"), "k": ((self.kd, self.hidden), "matrix"),
               "v": ((self.vd, self.hidden), "matrix"), "o": ((self.hidden, self.heads * self.vdim), "matrix")}
        if self.has_bias:
            out.update({"q_bias": ((self.qd,), "zero"), "k_bias": ((self.kd,), "zero"), "v_bias": ((self.vd,), "zero")})
        if self.qk_norm:
            out.update({"q_norm": ((self.qd if self.norm_all else self.dim,), "norm"),
                        "k_norm": ((self.kd if self.norm_all else self.dim,), "norm")})
        if self.taps:
            out.update({"q_conv": ((self.qd, self.taps), "unit"), "k_conv": ((self.kd, self.taps), "unit"),
                        "v_conv": ((self.vd, self.taps), "unit")})
        if self.v_mix is not None:
            out["v_lambda"] = ((), "zero")      # the source layer has the tensor too and does not use it
        if self.has_sink:
            out["sink"] = ((self.heads,), "unit")
        if self.head_gate:
            out["g"] = ((self.heads, self.hidden), "matrix")
        return out

    def _projections(self):
        return ("q", "k", "v", "g") if self.head_gate else ("q", "k", "v")

    def adjacent_weights(self):
        return [self._projections()]

    def _span(self):
        """How many keys a query sees at most: its window, and never more than one block of `chunk` positions."""
        spans = [int(s) for s in (self.window, self.chunk) if s]
        return min(spans) if spans else None

    def cache_request(self):
        return KVCacheRequest(self.kv_heads, self.dim, self._span(), None if self.vdim == self.dim else self.vdim)

    def state_request(self):
        if not self.taps:
            return None
        return StateRequest((max(self.taps - 1, 1), self.qd + self.kd + self.vd), torch.float32)

    def prepare(self, dtype, device) -> None:
        t = self.tensors
        self.proj = Linear(fused_rows([t[n] for n in self._projections()]), "general_attention.in")
        self.o = Linear(t["o"], "general_attention.o")
        self.proj.prepare(dtype)
        self.o.prepare(dtype)
        self.bias = (torch.cat([t[n].to(torch.float32).reshape(-1) for n in ("q_bias", "k_bias", "v_bias")]).contiguous()
                     if self.has_bias else None)
        norm_dtype = torch.float32 if self.norm_all else dtype
        self.q_norm = t["q_norm"].to(norm_dtype).contiguous() if self.qk_norm else None
        self.k_norm = t["k_norm"].to(norm_dtype).contiguous() if self.qk_norm else None
        self.conv_w = (torch.cat([t[n] for n in ("q_conv", "k_conv", "v_conv")], 0).to(torch.float32).contiguous()
                       if self.taps else None)
        self.v_lambda = float(t["v_lambda"].to(torch.float32).reshape(-1)[0].item()) if self.v_mix == "mix" else 0.0
        self.position.prepare(dtype, device)
        self.inv_freq = getattr(self.position, "inv_freq", None)
        self.rot_dims = int(getattr(self.position, "dims", 0)) if self.inv_freq is not None else 0
        if self.rot_dims > self.dim:
            raise ConfigError(f"general_attention: {self.rot_dims} rotated entries in a head of {self.dim}")
        self.halves = bool(getattr(self.position, "halves", False))
        self.magnitude = float(getattr(self.position, "magnitude", 1.0))
        if self.unit_qk and self.magnitude != 1.0:
            raise ConfigError("general_attention: queries and keys of unit size take a rotation that keeps their size")
        if self.taps and self.magnitude != 1.0:
            raise ConfigError("general_attention: the kernel with the convolution takes a rotation that keeps the heads' size")
        self.sink = t["sink"].to(torch.float32).contiguous() if self.has_sink else None
        if self.sink_score is not None:
            self.sink = torch.full((self.heads,), float(self.sink_score), dtype=torch.float32, device=device)
        self.fast = None
        if dtype == torch.bfloat16 and device.type == "cuda":
            # equal head sizes without a cap: the engine's tcgen05 prefill, cluster decode and mma.sync kernels;
            # otherwise the mma.sync kernel built for this value size and with the cap (sizes it takes)
            from ..kernels import attention as fast
            self.fast = fast.plan_for(self.dim, self.heads, self.kv_heads, False, self.vdim, self.softcap, self.window, self.chunk)

    def plan_step(self, ctx) -> None:
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.step_tiles(ctx, self.fast)

    def forward(self, ctx, call, h):
        from ..kernels import biased_attention as BA
        n = ctx.n_tokens
        u = self.proj.forward(ctx, h, n, ctx.dtype, "mixer_in").tensor
        q = ctx.ws.get("q", (n, self.qd), ctx.dtype)
        shared = ctx.ws.get("mixed_values", (n, self.vd), torch.float32) if self.v_mix else None
        if self.taps:
            kept = BA.conv_norm_cache(ctx, u, self.conv_w, call.state, self.q_norm, self.k_norm, q, call.cache, self.heads,
                                      self.eps, 0.0, 1, call.writes_cache, self.inv_freq, self.rot_dims, self.halves,
                                      write_ring=call.writes_cache and ctx.max_q_len == 1)
            if call.writes_cache and not kept:
                BA.conv_ring_write(ctx, u, call.state, self.taps, self.qd + self.kd + self.vd)
        else:
            self._prepare_heads(ctx, call, u, q, shared)
        out = ctx.ws.get("attn_out", (n, self.heads * self.vdim), ctx.dtype)
        window = int(self.window) if self.window else 0
        extras = K.AttentionExtras(self.chunk or 0, self.sink, u[:, u.shape[1] - self.heads:] if self.head_gate else None)
        if self.fast is not None and ctx.use_fast_attention:
            from ..kernels import attention as fast
            fast.run(ctx, self.fast, q, out, call.cache, self.scale, window, extras=extras)
        else:
            BA.attention(ctx, q, out, call.cache, None, self.heads, self.scale, window, 1.0, self.softcap, extras)
        return self.o.forward(ctx, out, n, torch.float32, "attn_proj", allow_partials=True)

    def _prepare_heads(self, ctx, call, u, q, shared) -> None:
        from ..kernels import head_prepare as HP
        HP.headnorm_rope_cache(ctx, u, 0, self.qd, self.qd + self.kd, self.q_norm, self.k_norm, self.eps, self.inv_freq,
                               self.rot_dims, self.magnitude, q, call.cache, self.heads, call.writes_cache,
                               halves=self.halves, bias=self.bias, v_mix_in=shared if self.v_mix == "mix" else None,
                               v_mix=self.v_lambda, v_mix_out=shared if self.v_mix == "source" else None,
                               unit_norm=self.unit_qk)
