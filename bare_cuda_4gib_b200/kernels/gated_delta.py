"""Launchers of `csrc/gated_delta.cu` and `csrc/gated_delta_chunked.cu`: the gated delta rule over a step's
tokens (operands, scan, chunks on the tensor cores) and in one kernel for steps of one token per request."""

from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Optional

import torch

from . import build
from .lib import _check, _dev, _ptr, dtype_code

MAX_KEY_DIM = 1024
STEP_MAX_SHARED = 160 * 1024
_lib = None


def lib():
    global _lib
    if _lib is None:
        l = build.load_library("gated_delta.cu")
        P, I, L, F = c_void_p, c_int, c_longlong, c_float
        l.llm_gated_delta_operands.argtypes = [P, I, L, P, I, P, P, P, P, P, P, P, P, I, I, I, I, I, F, F, P, P, P]
        l.llm_gated_delta_scan.argtypes = [P, P, P, P, L, I, P, L, I, P, P, I, P, P, P, P, P, I, I, I, I, I, P]
        l.llm_gated_delta_step.argtypes = [P, I, L, P, I, P, P, L, I, P, L, I, P, P, I, P, P, L, I, I, P, P, L, P, P, P, I, I, I,
                                           I, I, I, F, F, F, P]
        l.llm_gated_delta_step_shared_bytes.argtypes = [I, I]
        l.llm_gated_delta_step_shared_bytes.restype = c_longlong
        for name in ("llm_gated_delta_operands", "llm_gated_delta_scan", "llm_gated_delta_step"):
            getattr(l, name).restype = c_int
        _lib = l
    return _lib


class Gates:
    """Where a token's decays and step size come from: `z` [rows, heads] or (with `channel`) [rows, heads * dim]
    and `b` [rows, heads], pre-activations that may be column views; `a_log` [heads], `dt_bias` like z's
    columns, float32.  decay = exp(-exp(a_log) softplus(z + dt_bias)), step size = sigmoid(b)."""

    __slots__ = ("z", "b", "a_log", "dt_bias", "channel")

    def __init__(self, z: torch.Tensor, b: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, channel: bool):
        _dev(z, b, a_log, dt_bias)
        if z.stride(-1) != 1 or b.stride(-1) != 1 or a_log.dtype != torch.float32 or dt_bias.dtype != torch.float32:
            raise TypeError("gated delta: gates not as the kernels need")
        self.z, self.b, self.a_log, self.dt_bias, self.channel = z, b, a_log, dt_bias, channel

    def arguments(self):
        return (self.z.data_ptr(), self.z.stride(0), dtype_code(self.z.dtype), self.b.data_ptr(), self.b.stride(0),
                dtype_code(self.b.dtype), self.a_log.data_ptr(), self.dt_bias.data_ptr(), 1 if self.channel else 0)


def _floats(what: str, *tensors: Optional[torch.Tensor]) -> None:
    _dev(*tensors)
    for t in tensors:
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError(f"gated delta {what}: constants, states and operands must be contiguous float32")


def operands(ctx, u: torch.Tensor, conv_w: torch.Tensor, ring: torch.Tensor, qn, kn, vn, kv_heads: int, dk: int,
             heads: int, dv: int, unit_eps: float, compact: Optional[torch.Tensor] = None,
             lengths: Optional[torch.Tensor] = None) -> None:
    """u [rows, q | k | v | ...]: the convolution (history before the step from `ring`) and silu; qn, kn [rows,
    kv_heads * dk] the unit vectors (q also / sqrt(dk)), vn [rows, heads * dv].  All float32.  With `compact`
    (bfloat16 [rows, q | k | v]) these are left out: the activations go there, and to `lengths` (float32 [rows,
    2 * kv_heads], the q heads first) the factors that make the unit vectors of the rounded q and k heads."""
    _floats("operands", conv_w, ring, qn, kn, vn, lengths)
    if compact is not None and (compact.dtype != torch.bfloat16 or not compact.is_contiguous() or lengths is None):
        raise TypeError("gated delta operands: the compact form is contiguous bfloat16 with float32 factors beside it")
    _check(lib().llm_gated_delta_operands(
        u.data_ptr(), dtype_code(u.dtype), u.stride(0), conv_w.data_ptr(), conv_w.shape[1], ring.data_ptr(), _ptr(qn),
        _ptr(kn), _ptr(vn), ctx.positions.data_ptr(), ctx.row_seq.data_ptr(), ctx.seq_slot.data_ptr(),
        ctx.seq_q_start.data_ptr(), ctx.n_tokens, kv_heads, dk, heads, dv, float(unit_eps), dk ** -0.5, _ptr(compact),
        _ptr(lengths), ctx.stream), "gated_delta_operands")


def scan(ctx, qn: torch.Tensor, kn: torch.Tensor, vn: torch.Tensor, gates: Gates, state: torch.Tensor, out: torch.Tensor,
         heads: int, kv_heads: int, dk: int, dv: int) -> None:
    """Every request's new tokens in order: S = g S; u = beta (v - S^T k); S += k u^T; out = S^T q, with S in
    `state[slot]` ([heads, dk, dv] float32) read at the start and left at the end.  out [rows, heads * dv]."""
    _floats("scan", qn, kn, vn, state, out)
    _check(lib().llm_gated_delta_scan(
        qn.data_ptr(), kn.data_ptr(), vn.data_ptr(), *gates.arguments(), state.data_ptr(), out.data_ptr(),
        ctx.seq_slot.data_ptr(), ctx.seq_q_start.data_ptr(), ctx.seq_q_len.data_ptr(), ctx.n_seqs, heads, kv_heads, dk, dv,
        ctx.stream), "gated_delta_scan")


def step_takes(dk: int, dv: int) -> bool:
    """Whether the kernel for steps of one token per request takes these head sizes."""
    need = int(lib().llm_gated_delta_step_shared_bytes(dk, dv))
    return 0 < need <= STEP_MAX_SHARED


def step(ctx, u: torch.Tensor, conv_w: torch.Tensor, ring: torch.Tensor, gates: Gates, state: torch.Tensor,
         gate: torch.Tensor, gate_kind: str, norm_w: torch.Tensor, out: torch.Tensor, heads: int, kv_heads: int, dk: int,
         dv: int, unit_eps: float, eps: float, write_ring: bool) -> None:
    """A step of one token per request, a block per (request, head): everything from the stored projections to
    what the output projection reads.  `gate` [rows, heads * dv] pre-activations of `gate_kind` ("silu" or
    "sigmoid"), possibly a column view; out [rows, heads * dv] = rms_norm per head * norm_w * gate."""
    _floats("step", conv_w, ring, state, norm_w)
    _dev(u, gate, out)
    if out.dtype != u.dtype or gate.stride(1) != 1:
        raise TypeError("gated delta step: element types or layout not as the kernel needs")
    _check(lib().llm_gated_delta_step(
        u.data_ptr(), dtype_code(u.dtype), u.stride(0), conv_w.data_ptr(), conv_w.shape[1], ring.data_ptr(),
        *gates.arguments(), state.data_ptr(), gate.data_ptr(), gate.stride(0), dtype_code(gate.dtype),
        {"silu": 1, "sigmoid": 0}[gate_kind], norm_w.data_ptr(), out.data_ptr(), out.stride(0), ctx.positions.data_ptr(),
        ctx.seq_slot.data_ptr(), ctx.seq_q_start.data_ptr(), ctx.n_seqs, heads, kv_heads, dk, dv, 1 if write_ring else 0,
        float(unit_eps), dk ** -0.5, float(eps), ctx.stream), "gated_delta_step")


CHUNKED_MIN_TOKENS = 32      # steps with a portion at least this long take the chunked walk
CHUNK = 64
_chunked_libs = {}


def chunked_takes(dk: int, dv: int) -> bool:
    """Head sizes the chunked walk on the tensor cores takes (a library per key size)."""
    return dk % 16 == 0 and 16 <= dk <= 128 and dv % 16 == 0


def chunked_columns(heads: int, dv: int) -> int:
    """Value columns of a block: 32, or 16 where one request's blocks would not come near the number of SMs."""
    from .lib import sm_count
    return 32 if dv % 32 == 0 and heads * (dv // 32) >= sm_count() // 2 else 16


def chunked_lib(dk: int):
    l = _chunked_libs.get(dk)
    if l is None:
        l = build.load_library("gated_delta_chunked.cu", (f"-DGD_DK={dk}",))
        P, I, L = c_void_p, c_int, c_longlong
        l.llm_gated_delta_prepare.argtypes = [P, P, P, L, I, P, L, I, P, P, I, P, P, P, L, P, L, P, P, P, P, I, I, I, I, I, I, P]
        l.llm_gated_delta_walk.argtypes = [P, P, P, L, P, L, P, P, P, P, P, P, P, I, I, I, I, I, P]
        l.llm_gated_delta_prepare.restype = l.llm_gated_delta_walk.restype = c_int
        _chunked_libs[dk] = l
    return l


def chunked(ctx, compact: torch.Tensor, lengths: torch.Tensor, gates: Gates, state: torch.Tensor, out: torch.Tensor,
            heads: int, kv_heads: int, dk: int, dv: int, columns: int = 0) -> None:
    """What `scan` does, in chunks of 64 tokens on the tensor cores, from the compact operands: two kernels, one over
    all chunks side by side for everything that does not depend on the state, one that walks every request's
    chunks in order."""
    _floats("chunked", lengths, state, out)
    if compact.dtype != torch.bfloat16 or not compact.is_contiguous():
        raise TypeError("gated delta chunked: the operands must be contiguous bfloat16")
    columns = columns or chunked_columns(heads, dv)
    n = ctx.n_tokens
    tiles = ctx.ws.get("delta_tiles", (6, n, heads * dk), torch.bfloat16, max_lead=6)      # (W, Q', K'') x (rounded, rest)
    pairs = ctx.ws.get("delta_pairs", (2, n, heads * CHUNK), torch.bfloat16, max_lead=2)
    u = ctx.ws.get("delta_u", (n, heads * dv), torch.float32)
    most = ctx.max_rows // CHUNK + ctx.max_seqs + 1
    end = ctx.ws.get("delta_end", (n // CHUNK + ctx.n_seqs + 1, heads * dk), torch.float32, max_rows=most)
    l = chunked_lib(dk)
    plane = tiles.stride(0)
    at = [tiles.data_ptr() + 2 * plane * i for i in range(6)]
    where = (at[0], at[1], at[2], 3 * plane, pairs.data_ptr(), pairs.stride(0), u.data_ptr(), end.data_ptr())
    _check(l.llm_gated_delta_prepare(
        compact.data_ptr(), lengths.data_ptr(), *gates.arguments(), *where, ctx.seq_q_start.data_ptr(),
        ctx.seq_q_len.data_ptr(), ctx.n_seqs, int(ctx.max_q_len), heads, kv_heads, dk, dv, ctx.stream), "gated_delta_prepare")
    _check(l.llm_gated_delta_walk(
        *where, state.data_ptr(), out.data_ptr(), ctx.seq_slot.data_ptr(), ctx.seq_q_start.data_ptr(),
        ctx.seq_q_len.data_ptr(), ctx.n_seqs, heads, dk, dv, columns, ctx.stream), "gated_delta_walk")
