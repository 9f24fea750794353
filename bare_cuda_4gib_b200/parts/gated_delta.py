"""The gated delta rule as a mixer over state slots.

q, k (kv_heads x dim) and v (heads x vdim) are projections behind a short causal convolution per channel and
silu; q and k become unit vectors per head, q also / sqrt(dim).  With step size beta = sigmoid(W_b h) and decay
g = exp(-exp(A_log) softplus(z + dt_bias)), per head (head i reads q/k head i / (heads / kv_heads)):

    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            (S dim x vdim, float32)

and every head's o is RMS-normed by itself, multiplied by one weight [vdim] that the heads share and by a gate
of the mixer's input, and projected.  Options:

* `decay` "head": z = W_a h, one number per head; "channel": one per head and key channel, which acts on the
  rows of S, through a low rank, z = W_a2 (W_a1 h);
* `gate` "silu" or "sigmoid", of W_g h; with the channel decay of W_g2 (W_g1 h).

One product makes everything that reads h; with low ranks a second one multiplies both of them by their upper
halves ([a2 0; 0 g2] over [a1 h | g1 h], float32 results).  A request keeps S as a float32 state and the
convolution's last inputs as a second one (a ring of `taps` entries by position).  Steps of one token per request
run one kernel with a block per (request, head); other steps prepare operands, walk the state, and norm
and gate.  The walk goes token by token over float32 operands, or in bfloat16 steps with a portion of `kernels.gated_delta.
CHUNKED_MIN_TOKENS` or more (sizes that are multiples of 16) in chunks on the tensor cores.

params: `hidden`, `heads`, `kv_heads`, `dim`, `vdim`, `taps`, `decay`, `gate`, `rank` (None: from the file),
`eps`, `unit_eps` (under the root of the unit vectors).
tensors: `q`, `k`, `v`, `q_conv`, `k_conv`, `v_conv` [channels, taps], `b` [heads, hidden], `A_log` [heads], `norm`
[vdim], `o`; "head": `a` [heads, hidden], `dt_bias` [heads], `g`; "channel": `a1`, `a2`, `dt_bias` [heads * dim],
`g1`, `g2`.
"""

from __future__ import annotations

import torch

from ..errors import ConfigError
from ..kernels import gated_delta as GD, linear_attention as LA
from .base import Part, StateRequest
from .linear import Linear
from .registry import register_mixer
from ..weights.loader import fused_rows


@register_mixer("gated_delta")
class GatedDelta(Part):
    takes_lazy_input = False

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim, self.taps = int(p["dim"]), int(p["vdim"]), int(p["taps"])
        self.eps, self.unit_eps = float(p["eps"]), float(p["unit_eps"])
        if self.heads % self.kv_heads:
            raise ConfigError(f"gated_delta: {self.heads} heads cannot share {self.kv_heads} query/key heads")
        if self.dim > GD.MAX_KEY_DIM:
            raise ConfigError(f"gated_delta: key size {self.dim} exceeds the {GD.MAX_KEY_DIM} the scan kernel takes")
        if self.taps < 1:
            raise ConfigError("gated_delta: the convolution needs at least one tap")
        if p["decay"] not in ("head", "channel") or p["gate"] not in ("silu", "sigmoid"):
            raise ConfigError(f"gated_delta: decay '{p['decay']}' or gate '{p['gate']}' is not known")
        self.channel, self.gate_kind = p["decay"] == "channel", p["gate"]
        self.kd, self.vd = self.kv_heads * self.dim, self.heads * self.vdim
        self.conv_channels = 2 * self.kd + self.vd

    def local_weights(self):
        H, W = self.heads, self.hidden
        out = {"q": ((self.kd, W), "matrix"), "k": ((self.kd, W), "matrix"), "v": ((self.vd, W), "matrix"),
               "q_conv": ((self.kd, self.taps), "unit"), "k_conv": ((self.kd, self.taps), "unit"),
               "v_conv": ((self.vd, self.taps), "unit"), "b": ((H, W), "matrix"), "A_log": ((H,), "zero"),
               "norm": ((self.vdim,), "norm"), "o": ((W, self.vd), "matrix")}
        if self.channel:
            rank, zd = int(self.params.get("rank") or -1), H * self.dim
            out.update({"a1": ((rank, W), "matrix"), "a2": ((zd, rank), "matrix"), "dt_bias": ((zd,), "unit"),
                        "g1": ((rank, W), "matrix"), "g2": ((self.vd, rank), "matrix")})
        else:
            out.update({"a": ((H, W), "matrix"), "dt_bias": ((H,), "unit"), "g": ((self.vd, W), "matrix")})
        return out

    def _projections(self):
        """What is multiplied with h, in the order of the product's columns."""
        return ("q", "k", "v", "a1", "g1", "b") if self.channel else ("q", "k", "v", "g", "a", "b")

    def adjacent_weights(self):
        return [self._projections()]

    def cache_request(self):
        return None

    def state_request(self):
        return StateRequest((self.heads, self.dim, self.vdim), torch.float32)

    def cache_demands(self):
        """Two states per request: S, and the ring of the convolution's last inputs."""
        return [(None, self.state_request()),
                (None, StateRequest((self.taps, self.conv_channels), torch.float32))]

    def prepare(self, dtype, device) -> None:
        t = self.tensors
        self.columns, at = {}, 0
        for name in self._projections():
            self.columns[name] = (at, at + int(t[name].shape[0]))
            at += int(t[name].shape[0])
        self.proj = Linear(fused_rows([t[n] for n in self._projections()]), "gated_delta.in")
        self.o = Linear(t["o"], "gated_delta.o")
        self.proj.prepare(dtype)
        self.o.prepare(dtype)
        f = lambda x: x.to(torch.float32).contiguous()
        self.conv_w = f(torch.cat([t["q_conv"], t["k_conv"], t["v_conv"]], 0))
        self.a_log, self.dt_bias, self.norm_w = f(t["A_log"]), f(t["dt_bias"]), f(t["norm"])
        if self.channel:
            a2, g2 = t["a2"], t["g2"]
            both = torch.zeros((a2.shape[0] + g2.shape[0], a2.shape[1] + g2.shape[1]), dtype=a2.dtype, device=a2.device)
            both[: a2.shape[0], : a2.shape[1]] = a2
            both[a2.shape[0]:, a2.shape[1]:] = g2
            self.expand = Linear(both, "gated_delta.expand")
            # the fast products read their input in 16-byte pieces: a view that does not start or step so takes the plain one
            first, width = self.columns["a1"][0], at
            if first % 8 == 0 and width % 8 == 0:
                self.expand.prepare(dtype)
        self.one_step = device.type == "cuda" and GD.step_takes(self.dim, self.vdim)
        self.chunked = device.type == "cuda" and dtype == torch.bfloat16 and GD.chunked_takes(self.dim, self.vdim)
        if self.chunked:
            GD.chunked_lib(self.dim)      # compiled with the model, not at its first long portion
        self.tensors = {}

    def forward(self, ctx, call, h):
        n, H, G, dk, dv = ctx.n_tokens, self.heads, self.kv_heads, self.dim, self.vdim
        f32 = torch.float32
        u = self.proj.forward(ctx, h, n, ctx.dtype, "mixer_in").tensor
        col = lambda name: u[:, self.columns[name][0]: self.columns[name][1]]
        if self.channel:
            low = u[:, self.columns["a1"][0]: self.columns["g1"][1]]
            high = self.expand.forward(ctx, low, n, f32, "delta_high").tensor
            z, gate = high[:, : H * dk], high[:, H * dk:]
        else:
            z, gate = col("a"), col("g")
        gates = GD.Gates(z, col("b"), self.a_log, self.dt_bias, self.channel)
        state, ring = call.states[0], call.states[1]
        out = ctx.ws.get("mixer_act", (n, self.vd), ctx.dtype)
        if ctx.max_q_len == 1 and self.one_step:
            GD.step(ctx, u, self.conv_w, ring, gates, state, gate, self.gate_kind, self.norm_w, out, H, G, dk, dv,
                    self.unit_eps, self.eps, call.writes_cache)
            return self.o.forward(ctx, out, n, f32, "mixer_out", allow_partials=True)
        scanned = ctx.ws.get("delta_scan", (n, self.vd), f32)
        chunked = self.chunked and ctx.max_q_len >= GD.CHUNKED_MIN_TOKENS and ctx.use_fast_attention
        if chunked:
            compact = ctx.ws.get("delta_compact", (n, self.conv_channels), torch.bfloat16)
            lengths = ctx.ws.get("delta_lengths", (n, 2 * G), f32)
            GD.operands(ctx, u, self.conv_w, ring, None, None, None, G, dk, H, dv, self.unit_eps, compact, lengths)
        else:
            qn, kn = ctx.ws.get("delta_q", (n, self.kd), f32), ctx.ws.get("delta_k", (n, self.kd), f32)
            vn = ctx.ws.get("delta_v", (n, self.vd), f32)
            GD.operands(ctx, u, self.conv_w, ring, qn, kn, vn, G, dk, H, dv, self.unit_eps)
        if call.writes_cache:
            from ..kernels import mamba2 as MK
            MK.ring_write(ctx, u[:, : self.conv_channels], ring, self.taps, self.conv_channels)
        if chunked:
            GD.chunked(ctx, compact, lengths, gates, state, scanned, H, G, dk, dv)
        else:
            GD.scan(ctx, qn, kn, vn, gates, state, scanned, H, G, dk, dv)
        LA.gated_group_norm(scanned, gate, self.norm_w, out, n, dv, self.gate_kind, self.eps, 1.0, ctx.stream)
        return self.o.forward(ctx, out, n, f32, "mixer_out", allow_partials=True)
