"""The Sizitar decoder in the engine against the plain implementation (`plain_sizitar`): kernels and
mechanisms alone, every way of cutting requests into steps, slots and pages used again, planted
weights where random ones would hide a fault, and greedy generation through the entry point."""

import copy
import json
import random

import pytest
import torch

import helpers as H
import plain_sizitar as P
import sizitar_helpers as U

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
LENGTHS = {"A": [1, 2, 3, 17, 33, 70, 150], "B": [2, 5, 31, 64, 65, 200]}


def _requests(name, seed, lengths, dtype="float32"):
    rng = random.Random(seed)
    vocab = U.CONFIGS[name][0]["vocab"]
    return {f"r{i}": U.clear_ids(U.model_folder(name, 3, dtype), rng, n, vocab) for i, n in enumerate(lengths)}


# ------------------------------------------------------------------------------- the kernels alone

F32 = dict(dtype=torch.float32, device="cuda")


def _ctx(lengths, dtype=torch.bfloat16, slots=None):
    """A step of requests that bring `lengths` tokens each, from position 0, in slots taken backwards."""
    from bare_cuda_4gib_b200.engine.step import Workspace
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    n, k = sum(lengths), len(lengths)

    class Ctx:
        pass
    c = Ctx()
    c.stream = torch.cuda.current_stream().cuda_stream
    c.dtype, c.use_fast_attention = dtype, True
    c.n_tokens, c.n_seqs, c.max_q_len, c.max_rows, c.max_seqs = n, k, max(lengths), n, k
    c.positions = i32([p for q in lengths for p in range(q)])
    c.row_seq = i32([s for s, q in enumerate(lengths) for _ in range(q)])
    c.slots = list(range(k))[::-1] if slots is None else slots
    c.seq_slot = i32(c.slots)
    c.starts = [sum(lengths[:s]) for s in range(k)]
    c.seq_q_start, c.seq_q_len, c.seq_kv_len = i32(c.starts), i32(lengths), i32(lengths)
    c.ws = Workspace(torch.device("cuda"), n)
    return c


def _inputs(n, heads, kv_heads, dk, dv, channel, seed, strength=0.0):
    """Keys, queries and values that bfloat16 holds exactly, and gates; `strength` shifts the decays' logarithms
    towards faster decay."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    q, k, v = (r(n, h, d).to(torch.bfloat16).double() for h, d in ((kv_heads, dk), (kv_heads, dk), (heads, dv)))
    b = 2.0 * r(n, heads)
    zd = heads * dk if channel else heads
    z, a_log, dt_bias = r(n, zd), 0.5 * r(heads) + strength - 1.0, r(zd)
    return q, k, v, z, b, a_log, dt_bias


def _decays(z, a_log, dt_bias, heads, channel):
    s = P.softplus(z.double() + dt_bias.double())
    s = s.view(z.shape[0], heads, -1)
    return torch.exp(-torch.exp(a_log.double())[None, :, None] * s)


def _want(q, k, v, z, b, a_log, dt_bias, channel, lengths, slots, start):
    """The plain rule per request and head; returns (outputs, states by slot)."""
    heads, kv_heads = v.shape[1], q.shape[1]
    g, beta = _decays(z, a_log, dt_bias, heads, channel), torch.sigmoid(b.double())
    out, states, at = torch.zeros(v.shape, dtype=torch.float64), start.double().clone(), 0
    for s, n in enumerate(lengths):
        rows = slice(at, at + n)
        for h in range(heads):
            kv = h // (heads // kv_heads)
            out[rows, h], states[slots[s], h] = P.delta_rule(q[rows, kv].double(), k[rows, kv].double(), v[rows, h].double(),
                                                             g[rows, h], beta[rows, h], start[slots[s], h].double())
        at += n
    return out, states


SIZES = [(4, 2, 16, 32), (3, 3, 48, 16), (2, 1, 128, 64), (2, 2, 80, 96), (6, 2, 32, 32)]
ODD_SIZES = [(2, 1, 10, 6), (3, 1, 7, 33), (1, 1, 200, 20), (2, 2, 600, 8), (4, 4, 64, 130), (2, 1, 1, 1)]


def _run(lengths, sizes, channel, seed, form, strength=0.0):
    from bare_cuda_4gib_b200.kernels import gated_delta as GD
    heads, kv_heads, dk, dv = sizes
    n = sum(lengths)
    ctx = _ctx(lengths)
    q, k, v, z, b, a_log, dt_bias = _inputs(n, heads, kv_heads, dk, dv, channel, seed, strength)
    start = 0.3 * torch.randn(len(lengths) + 1, heads, dk, dv, generator=torch.Generator().manual_seed(seed + 1))
    qn, kn = P.unit_vector(q) * dk ** -0.5, P.unit_vector(k)
    want, want_state = _want(qn, kn, v, z, b, a_log, dt_bias, channel, lengths, ctx.slots, start)
    c = lambda t: t.reshape(t.shape[0], -1).float().cuda().contiguous()
    state, out = start.cuda(), torch.full((n, heads * dv), float("nan"), **F32)
    gates = GD.Gates(c(z), c(b), a_log.cuda(), dt_bias.cuda(), channel)
    if form == "scan":
        GD.scan(ctx, c(qn), c(kn), c(v), gates, state, out, heads, kv_heads, dk, dv)
    else:
        compact = torch.cat([c(q), c(k), c(v)], 1).to(torch.bfloat16).contiguous()
        factors = torch.cat([dk ** -0.5 / torch.sqrt((q * q).sum(-1) + 1e-6), 1.0 / torch.sqrt((k * k).sum(-1) + 1e-6)], 1)
        GD.chunked(ctx, compact, c(factors), gates, state, out, heads, kv_heads, dk, dv, form)
    torch.cuda.synchronize()
    assert torch.equal(state[-1].cpu(), start[-1])              # a slot that no request of the step holds
    scale, sscale = float(want.abs().max()), float(want_state[:-1].abs().max())
    err = float((out.view(n, heads, dv).cpu().double() - want).abs().max()) / scale
    serr = float((state[:-1].cpu().double() - want_state[:-1]).abs().max()) / sscale
    assert err == err and serr == serr
    return err, serr


@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("sizes", SIZES + ODD_SIZES)
def test_scan_against_the_plain_rule(sizes, channel):
    """Three requests of unequal length, states that are not empty, sizes that fill no warp or piece."""
    err, serr = _run([19, 1, 34], sizes, channel, 3, "scan")
    assert err < 2e-5 and serr < 2e-5, (err, serr)


@pytest.mark.parametrize("columns", [16, 32])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("sizes", SIZES)
def test_chunks_against_the_plain_rule(sizes, channel, columns):
    """Portions that end before, at and after a chunk's and a block of 16's edge, next to single tokens."""
    if sizes[3] % columns:
        pytest.skip("the value size is no multiple of the block's columns")
    for lengths in ([200, 1, 37, 64], [65], [16, 17, 15, 128, 2]):
        err, serr = _run(lengths, sizes, channel, 5, columns)
        assert err < 3e-4 and serr < 3e-4, (lengths, err, serr)


@pytest.mark.parametrize("strength", [2.0, 4.0, 7.0])
@pytest.mark.parametrize("channel", [False, True])
def test_chunks_with_decays_that_leave_nothing(channel, strength):
    """Decays so strong that the factors against a common token leave float32's range inside 16 tokens for some
    channels, while others keep most of what they hold."""
    err, serr = _run([130, 20], (4, 2, 32, 32), channel, 7, 16, strength)
    assert err < 2e-3 and serr < 2e-3, (err, serr)      # (a difference of two sums of large logarithms has fewer digits)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("sizes", SIZES + ODD_SIZES + [(2, 1, 256, 256), (1, 1, 512, 300)])
def test_one_token_step_against_operands_and_scan(sizes, channel, dtype):
    """The kernel for single tokens against convolution, scan, norm and gate one after the other: its results,
    its state and its ring, over a few tokens from the sequence's first one on."""
    from bare_cuda_4gib_b200.kernels import gated_delta as GD, linear_attention as LA, mamba2 as MK
    heads, kv_heads, dk, dv = sizes
    taps, seqs, eps = 4, 3, 1e-5
    kd, vd = kv_heads * dk, heads * dv
    C, zd = 2 * kd + vd, heads * dk if channel else heads
    g = torch.Generator().manual_seed(dk)
    f = lambda t: t.cuda().contiguous()
    conv_w = f(torch.randn(C, taps, generator=g) / 2.0)
    a_log, dt_bias, norm_w = f(0.5 * torch.randn(heads, generator=g)), f(torch.randn(zd, generator=g)), f(1.0 + 0.2 * torch.randn(dv, generator=g))
    rings = [torch.zeros(seqs + 1, taps, C, **F32) for _ in range(2)]
    states = [torch.zeros(seqs + 1, heads, dk, dv, **F32) for _ in range(2)]
    for step in range(6):
        ctx = _ctx([1] * seqs)
        ctx.positions += step
        ctx.seq_kv_len += step
        u = f(torch.randn(seqs, C + 2 * heads + vd, generator=g).to(dtype))
        z = f(torch.randn(seqs, zd, generator=g)) if channel else u[:, C: C + heads]
        b, gate = u[:, C + heads: C + 2 * heads], u[:, C + 2 * heads:]
        gates = GD.Gates(z, b, a_log, dt_bias, channel)
        kind = "sigmoid" if channel else "silu"
        got = torch.full((seqs, vd), float("nan"), dtype=dtype, device="cuda")
        assert GD.step_takes(dk, dv)
        GD.step(ctx, u, conv_w, rings[0], gates, states[0], gate, kind, norm_w, got, heads, kv_heads, dk, dv, 1e-6, eps, True)
        qn, kn, vn, o = (torch.empty(seqs, w, **F32) for w in (kd, kd, vd, vd))
        GD.operands(ctx, u, conv_w, rings[1], qn, kn, vn, kv_heads, dk, heads, dv, 1e-6)
        MK.ring_write(ctx, u[:, :C], rings[1], taps, C)
        GD.scan(ctx, qn, kn, vn, gates, states[1], o, heads, kv_heads, dk, dv)
        want = torch.empty(seqs, vd, dtype=dtype, device="cuda")
        LA.gated_group_norm(o, gate, norm_w, want, seqs, dv, kind, eps)
        torch.cuda.synchronize()
        assert torch.equal(rings[0], rings[1])
        assert torch.allclose(states[0], states[1], rtol=1e-4, atol=1e-5), float((states[0] - states[1]).abs().max())
        # a head whose outputs nearly cancel is normed up with its rounding: rows go by their largest entry
        assert H.row_error(got, want) < (2e-4 if dtype == torch.float32 else 2e-2), step


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_operands_against_plain_pieces(taps):
    from bare_cuda_4gib_b200.kernels import gated_delta as GD
    heads, kv_heads, dk, dv, n = 4, 2, 12, 9, 21
    kd, C = kv_heads * dk, 2 * kv_heads * dk + heads * dv
    g = torch.Generator().manual_seed(taps)
    u, w = torch.randn(n, C + 5, generator=g), torch.randn(C, taps, generator=g)
    y = P.silu(P.short_convolution(u[:, :C].double(), w.double()))
    qn, kn, vn = (torch.full((n, x), float("nan"), **F32) for x in (kd, kd, heads * dv))
    GD.operands(_ctx([n], torch.float32), u.cuda(), w.cuda(), torch.zeros(2, taps, C, **F32), qn, kn, vn, kv_heads, dk, heads, dv, 1e-6)
    assert H.row_error(qn, (P.unit_vector(y[:, :kd].view(n, kv_heads, dk)) * dk ** -0.5).reshape(n, kd)) < 1e-5
    assert H.row_error(kn, P.unit_vector(y[:, kd: 2 * kd].view(n, kv_heads, dk)).reshape(n, kd)) < 1e-5
    assert H.row_error(vn, y[:, 2 * kd:]) < 1e-5


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("heads,kv_heads,dk,dv", [(4, 2, 16, 20), (2, 2, 128, 64), (3, 1, 48, 16), (6, 3, 32, 36), (2, 1, 64, 130)])
def test_compact_operands_over_two_steps(heads, kv_heads, dk, dv, taps):
    """Activations and unit factors of requests that go on from a ring, cut inside the convolution's reach, in the
    form that walks rows and in the one with a block per token."""
    from bare_cuda_4gib_b200.kernels import gated_delta as GD, mamba2 as MK
    kd, C = kv_heads * dk, 2 * kv_heads * dk + heads * dv
    cuts, total = ([19, 1, 3, 40], [2, 5, 1, 20]), [21, 6, 4, 60]
    g = torch.Generator().manual_seed(taps)
    u = [torch.randn(n, C + 8, generator=g).to(torch.bfloat16) for n in total]
    w = torch.randn(C, taps, generator=g)
    want = [P.silu(P.short_convolution(x[:, :C].double(), w.double())).to(torch.bfloat16).double() for x in u]
    ring = torch.full((5, taps, C), float("nan"), **F32)
    done = [0] * 4
    for cut in cuts:
        ctx = _ctx(cut)
        ctx.positions = torch.cat([torch.arange(d, d + n) for d, n in zip(done, cut)]).to(torch.int32).cuda()
        ctx.seq_kv_len = torch.tensor([d + n for d, n in zip(done, cut)], dtype=torch.int32, device="cuda")
        rows = torch.cat([x[d: d + n] for x, d, n in zip(u, done, cut)]).cuda()
        compact = torch.full((sum(cut), C), float("nan"), dtype=torch.bfloat16, device="cuda")
        factors = torch.full((sum(cut), 2 * kv_heads), float("nan"), **F32)
        GD.operands(ctx, rows, w.cuda(), ring, None, None, None, kv_heads, dk, heads, dv, 1e-6, compact, factors)
        MK.ring_write(ctx, rows[:, :C], ring, taps, C)
        y = torch.cat([x[d: d + n] for x, d, n in zip(want, done, cut)])
        got = compact.double().cpu()
        assert float((got - y).abs().max()) < 2e-2 * float(y.abs().max()) and float((got != y).double().mean()) < 0.02
        heads_ = got[:, : 2 * kd].view(sum(cut), 2 * kv_heads, dk)
        f = 1.0 / torch.sqrt((heads_ * heads_).sum(-1) + 1e-6)
        f[:, :kv_heads] *= dk ** -0.5
        assert H.row_error(factors, f) < 1e-5
        done = [d + n for d, n in zip(done, cut)]


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dk,dv,rot", [(4, 2, 16, 24, 8), (2, 1, 128, 128, 128), (16, 4, 128, 64, 32), (3, 3, 10, 7, 6),
                                                      (32, 8, 128, 128, 64)])
def test_convolution_norm_rotation_and_cache(heads, kv_heads, dk, dv, rot, dtype, taps):
    """What stands between the projection and the scores, over three steps of requests that go on from their rings,
    the last one of single tokens: queries, and keys and values in their pages."""
    from bare_cuda_4gib_b200.kernels import biased_attention as BA
    from bare_cuda_4gib_b200.kernels.lib import CacheView
    qd, kd, vd, page, eps, base = heads * dk, kv_heads * dk, kv_heads * dv, 16, 1e-5, 300.0
    C, hist = qd + kd + vd, max(taps - 1, 1)
    if (heads, dk) == (4, 16):      # long portions: a block of the kernel walks several rows
        cuts = ([700, 1, 400], [2, 5, 30], [1, 1, 1])
    else:
        cuts = ([19, 1, 7], [2, 5, 30], [1, 1, 1])
    total = [sum(c[i] for c in cuts) for i in range(3)]
    g = torch.Generator().manual_seed(taps)
    u = [torch.randn(n, C + 8, generator=g).to(dtype) for n in total]
    w, qw, kw = torch.randn(C, taps, generator=g), 1 + 0.2 * torch.randn(qd, generator=g), 1 + 0.2 * torch.randn(kd, generator=g)
    want = []
    for x, n in zip(u, total):
        y = P.short_convolution(x[:, :C].double(), w.double())
        pos = torch.arange(n)
        q = P.turn_neighbours((P.unit_rms(y[:, :qd], eps) * qw.double()).view(n, heads, dk), pos, rot, base)
        k = P.turn_neighbours((P.unit_rms(y[:, qd: qd + kd], eps) * kw.double()).view(n, kv_heads, dk), pos, rot, base)
        want.append((q.reshape(n, qd), k, y[:, qd + kd:].view(n, kv_heads, dv)))
    per = kv_heads * page * (dk + dv)
    blocks = max(total) // page + 1
    pool = torch.full((3 * blocks, per), float("nan"), dtype=dtype, device="cuda")
    table = torch.randperm(3 * blocks, generator=g).view(3, blocks).to(torch.int32).cuda()
    cache = CacheView(pool.data_ptr(), pool.data_ptr() + kv_heads * page * dk * pool.element_size(), table, per, blocks, page, kv_heads,
                      dk, dtype, v_dim=dv)
    ring = torch.zeros(4, hist, C, **F32)
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], **F32)
    done = [0] * 3
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for cut in cuts:
        ctx = _ctx(cut, dtype)
        ctx.positions = torch.cat([torch.arange(d, d + n) for d, n in zip(done, cut)]).to(torch.int32).cuda()
        ctx.seq_kv_len = torch.tensor([d + n for d, n in zip(done, cut)], dtype=torch.int32, device="cuda")
        rows = torch.cat([x[d: d + n] for x, d, n in zip(u, done, cut)]).cuda()
        q_out = torch.full((sum(cut), qd), float("nan"), dtype=dtype, device="cuda")
        kept = BA.conv_norm_cache(ctx, rows, w.cuda(), ring, qw.cuda(), kw.cuda(), q_out, cache, heads, eps, 0.0, 1, True, freq, rot,
                                  False, write_ring=max(cut) == 1)
        if not kept:
            BA.conv_ring_write(ctx, rows, ring, taps, C)
        assert H.row_error(q_out, torch.cat([x[0][d: d + n] for x, d, n in zip(want, done, cut)])) < tol
        done = [d + n for d, n in zip(done, cut)]
    table, pool = table.cpu(), pool.cpu()
    for s in range(3):
        for p in range(total[s]):
            row = pool[int(table[s, p // page])]
            k = row[: kv_heads * page * dk].view(kv_heads, page, dk)[:, p % page]
            v = row[kv_heads * page * dk:].view(kv_heads, page, dv)[:, p % page]
            assert H.row_error(k, want[s][1][p]) < tol and H.row_error(v, want[s][2][p]) < tol, (s, p)
        for p in range(max(0, total[s] - (taps - 1)), total[s]):
            assert torch.equal(ring[ctx.slots[s], p % hist].cpu(), u[s][p, :C].float())


@pytest.mark.parametrize("n,experts,top", [(70, 5, 2), (9, 16, 4), (300, 3, 1), (40, 33, 7), (5, 6, 6)])
def test_router_with_bias_and_weights_over_the_chosen(n, experts, top):
    from bare_cuda_4gib_b200.kernels import moe as M
    g = torch.Generator().manual_seed(experts)
    hidden = 48
    h = torch.randn(n, hidden, generator=g)
    # logits far apart: the softmax over all experts would round the smaller ones to the same zero
    t = {"r.router": 40.0 * torch.randn(experts, hidden, generator=g) / hidden ** 0.5, "r.router.b": 5.0 * torch.randn(experts, generator=g)}
    margins = []
    want_ids, want_w = P.route({k: v.double() for k, v in t.items()}, "r.", {"experts": experts, "top": top}, h.double(), margins)
    clear = margins[0] > 1e-3
    ids, weights = torch.empty(n, top, dtype=torch.int32, device="cuda"), torch.empty(n, top, device="cuda")

    class Ctx:
        stream = torch.cuda.current_stream().cuda_stream
    M.route(Ctx, h.cuda(), t["r.router"].cuda(), None, top, 1.0, ids, weights, None, n, bias=t["r.router.b"].cuda(), chosen_softmax=True)
    assert clear.sum() > 0.8 * n
    assert torch.equal(ids.cpu().long()[clear].sort(-1).values, want_ids[clear].sort(-1).values)
    order, want_order = ids.cpu().long().argsort(-1), want_ids.argsort(-1)
    assert float((weights.cpu().gather(1, order) - want_w.gather(1, want_order))[clear].abs().max()) < 1e-4
    assert torch.allclose(weights.sum(-1).cpu(), torch.ones(n), atol=1e-5)


@pytest.mark.parametrize("rows,width", [(37, 200), (5, 202), (9, 2048), (70, 4096), (3, 6000)])
def test_scaled_add_and_norm_alone(rows, width):
    """x += s * y, then the norm, in the kernel's entry-by-entry, piece-by-piece and wide forms."""
    from bare_cuda_4gib_b200.kernels import gated_sandwich as GS
    from bare_cuda_4gib_b200.kernels.lib import Partials
    g = torch.Generator().manual_seed(2)
    x, y = torch.randn(rows, width, generator=g), torch.randn(3, rows, width, generator=g)
    s, w = 0.5 * torch.randn(width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    new = x.double() + y.double().sum(0) * s.double()
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        res, out = x.clone().cuda(), torch.empty(rows, width, dtype=dtype, device="cuda")
        GS.step(res, GS.GatedDelta(Partials(y.cuda(), 3), None, None, s.cuda(), None), w.cuda(), out, 1e-6, rows)
        assert H.row_error(res, new) < 1e-5
        assert H.row_error(out, P.unit_rms(new, 1e-6) * w.double()) < tol


# --------------------------------------------------------------------- mechanisms, one at a time

def _model(name, layers, seed, width=72, vocab=61, eps=1e-5, logit_scale=1.5, loop=None):
    cfg = U.config(layers, vocab, width, eps, logit_scale, loop)
    folder = H.tmp_root() / f"sizitar-one-{name}"
    U.register(folder, cfg, U.random_tensors(cfg, seed))
    return folder, cfg


ALONE = {
    "attention": [U.attention(4, 2, 16, 24, 4, 8)],
    "attention_one_tap_whole_turn": [U.attention(3, 1, 48, 16, 1, 48, base=300.0, scale=0.3)],
    "attention_odd_sizes": [U.attention(2, 2, 10, 33, 3, 4)],
    "attention_heads_of_64": [U.attention(4, 2, 64, 64, 3, 32)],          # equal heads of 64 and 128: the engine's fast kernels
    "attention_heads_of_128": [U.attention(8, 1, 128, 128, 5, 16, scale=0.2)],
    "attention_wide_values": [U.attention(2, 1, 32, 256, 2, 16)],
    "attention_twice": [U.attention(2, 1, 16, 16, 6, 4), U.attention(6, 3, 32, 16, 2, 32)],
    "delta": [U.delta(4, 2, 16, 24, 4)],
    "delta_one_head_one_tap": [U.delta(1, 1, 32, 16, 1)],
    "delta_shared_by_five": [U.delta(5, 1, 16, 16, 3)],
    "delta_odd_sizes": [U.delta(3, 3, 6, 10, 3)],
    "delta_wide": [U.delta(2, 1, 128, 128, 4)],
    "delta_wider_than_the_chunks": [U.delta(2, 2, 160, 48, 4)],
    "delta_twice_long_taps": [U.delta(2, 2, 16, 16, 7), U.delta(4, 1, 48, 32, 2)],
    "channel_delta": [U.channel_delta(4, 2, 16, 24, 4, 8)],
    "channel_delta_two_ranks": [U.channel_delta(2, 2, 32, 32, 4, (8, 24))],
    "channel_delta_odd_sizes": [U.channel_delta(3, 1, 6, 10, 3, 5)],
    "channel_delta_wide": [U.channel_delta(2, 2, 128, 128, 4, 32)],
    "channel_delta_wider_than_the_chunks": [U.channel_delta(2, 1, 144, 16, 2, 16)],
    "channel_delta_many_heads": [U.channel_delta(8, 8, 16, 16, 2, 16)],
    "both_kinds": [U.delta(2, 1, 16, 32, 3), U.channel_delta(4, 4, 32, 16, 2, 8), U.delta(4, 2, 48, 16, 4)],
    "dense": [U.delta(2, 2, 8, 8, 2, mlp=U.dense(56))],
    "experts_two_of_five": [U.attention(2, 1, 16, 16, 2, 8, mlp=U.moe(5, 2, 24))],
    "experts_one_of_three_wide_shared": [U.delta(2, 2, 16, 16, 2, mlp=U.moe(3, 1, 32, 136))],
    "experts_all": [U.attention(2, 1, 16, 16, 2, 8, mlp=U.moe(4, 4, 16, 8))],
    "experts_many_small": [U.delta(2, 1, 8, 8, 2, mlp=U.moe(33, 3, 8, 12))],
    "experts_odd_width": [U.attention(2, 1, 16, 16, 2, 8, mlp=U.moe(4, 2, 20, 21))],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(ALONE))
def test_each_mechanism_alone(which, dtype):
    layers = ALONE[which]
    if dtype == "bfloat16":      # routers that choose every expert: see `every_expert_chosen`
        layers = U.every_expert_chosen({"layers": layers})["layers"]
    folder, cfg = _model(f"{which}-{dtype}", layers, 11)
    rng = random.Random(5)
    requests = {"a": U.clear_ids(folder, rng, 90, cfg["vocab"]), "b": U.clear_ids(folder, rng, 1, cfg["vocab"])}
    steps = H.trace_whole(requests)
    got = H.Replayer(folder, dtype, 16, H.peak_tokens(steps, 16)).run(steps)
    U.check(folder, requests, got, dtype)
    # the same tokens in portions and one by one give the same logits
    steps = H.trace_portions({"a": requests["a"]}, random.Random(1))
    got = H.Replayer(folder, dtype, 16, 96, shuffle_seed=2).run(steps)
    U.check(folder, {"a": requests["a"]}, got, dtype)
    steps = H.trace_decode_tail({"a": requests["a"]}, 50)
    got = H.Replayer(folder, dtype, 16, 96, shuffle_seed=3).run(steps)
    U.check(folder, {"a": requests["a"]}, got, dtype, expect_all=False)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_width_that_no_fast_kernel_takes(dtype):
    """Width 50: no product, norm or copy in pieces of 16 bytes fits; every part takes its entry-by-entry form."""
    layers = [U.attention(2, 1, 16, 16, 3, 8, scale=0.4, mlp=U.moe(3, 2, 8)), U.delta(2, 1, 16, 16, 2, mlp=U.dense(12)),
              U.channel_delta(3, 3, 16, 16, 3, 7, mlp=U.moe(2, 1, 9, 11))]
    if dtype == "bfloat16":
        layers = U.every_expert_chosen({"layers": layers})["layers"]
    folder, cfg = _model(f"width50-{dtype}", layers, 17, width=50, vocab=37, loop=(0, 2, 2))
    rng = random.Random(4)
    requests = {"a": U.clear_ids(folder, rng, 70, 37), "b": U.clear_ids(folder, rng, 3, 37)}
    got = H.Replayer(folder, dtype, 16, 96).run(H.trace_whole(requests))
    U.check(folder, requests, got, dtype)
    got = H.Replayer(folder, dtype, 16, 96, shuffle_seed=3).run(H.trace_decode_tail({"a": requests["a"]}, 20))
    U.check(folder, {"a": requests["a"]}, got, dtype, expect_all=False)


@pytest.mark.parametrize("loop", [None, (0, 3, 2), (2, 3, 4), (0, 1, 1), (1, 1, 3)])
def test_layers_that_run_again(loop):
    """Every pass has a cache, a state and a ring of its own."""
    layers = [U.delta(2, 1, 16, 16, 3), U.attention(2, 1, 16, 16, 3, 8), U.channel_delta(2, 2, 16, 16, 2, 8, mlp=U.dense(24))]
    folder, cfg = _model(f"loop{loop}", layers, 19, loop=loop)
    ids = H.random_ids(random.Random(7), 60, cfg["vocab"])
    got = H.Replayer(folder, "float32", 16, 64, shuffle_seed=1).run(H.trace_portions({"a": ids}, random.Random(2)))
    U.check(folder, {"a": ids}, got, "float32")
    got = H.Replayer(folder, "float32", 16, 64).run(H.trace_decode_tail({"a": ids}, 30))
    U.check(folder, {"a": ids}, got, "float32", expect_all=False)


# ------------------------------------------------------------------ every cutting, two configs

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_whole(name, dtype):
    folder, page = U.model_folder(name, 3, dtype), U.CONFIGS[name][1]
    requests = _requests(name, 1, LENGTHS[name], dtype)
    steps = H.trace_whole(requests)
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page)).run(steps)
    U.check(folder, requests, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_prefill_then_token_by_token(name, dtype):
    folder, page = U.model_folder(name, 3, dtype), U.CONFIGS[name][1]
    requests = _requests(name, 2, LENGTHS[name][3:], dtype)
    steps = H.trace_decode_tail(requests, 45)
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page), shuffle_seed=3).run(steps)
    U.check(folder, requests, got, dtype, expect_all=False)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_down_to_two_tokens(name, dtype):
    folder, page = U.model_folder(name, 3, dtype), U.CONFIGS[name][1]
    requests = _requests(name, 3, LENGTHS[name][2:], dtype)
    steps = H.trace_portions(requests, random.Random(5))
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page), shuffle_seed=4).run(steps)
    U.check(folder, requests, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [2, 31, 32, 33, 63, 65])
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_of_one_size(name, size, dtype):
    """All portions of one size: shorter than the convolutions' reach, and around the sizes at which a portion goes
    to the tensor cores or starts another chunk."""
    folder, page = U.model_folder(name, 3, dtype), U.CONFIGS[name][1]
    ids = _requests(name, 12, [75 if size == 2 else 150], dtype)["r0"]
    steps = [{"step": i, "entries": [{"id": "r0", "tokens": ids[at: at + size], "want": list(range(len(ids[at: at + size])))}], "end": []}
             for i, at in enumerate(range(0, len(ids), size))]
    got = H.Replayer(folder, dtype, page, 160, shuffle_seed=8).run(steps)
    U.check(folder, {"r0": ids}, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_mixed_batches_reuse_slots_and_pages(name, dtype):
    """Unequal requests side by side, four slots and a small pool for eleven requests: every logit equals the
    request's alone, whatever slot and pages it got and whoever held them before (a state that was not emptied,
    or a ring of convolution inputs left by the slot's last owner, shows here)."""
    folder, page = U.model_folder(name, 3, dtype), U.CONFIGS[name][1]
    longest = 160
    rng = random.Random(11)
    requests = _requests(name, 4, [rng.randrange(3, longest // 2) for _ in range(10)] + [longest], dtype)
    budget = 2 * longest
    steps = H.trace_mixed(requests, random.Random(6), live=4, budget_tokens=budget, page=page)
    rep = H.Replayer(folder, dtype, page, budget, max_live=4, shuffle_seed=9)
    got = rep.run(steps)
    U.check(folder, requests, got, dtype)
    for group in rep.cache.groups:
        assert group.pool.acquired_total > group.pool.num_pages and group.pool.pages_in_use == 0
    assert rep.cache.free_slots == 4


@pytest.mark.parametrize("name", ["A", "B"])
def test_long_portions_beside_single_tokens(name):
    """A prompt's long portions on the tensor cores in the same steps as another request's single tokens."""
    folder, page = U.model_folder(name, 3, "bfloat16"), U.CONFIGS[name][1]
    requests = _requests(name, 15, [180, 40], "bfloat16")
    a, b = requests["r0"], requests["r1"]
    steps, at = [{"step": 0, "entries": [{"id": "r1", "tokens": b[:37], "want": [36]}], "end": []}], 0
    for i, size in enumerate((70, 45, 65)):
        steps.append({"step": i + 1, "entries": [{"id": "r1", "tokens": [b[37 + i]], "want": [0]},
                                                 {"id": "r0", "tokens": a[at: at + size], "want": list(range(size))}], "end": []})
        at += size
    got = H.Replayer(folder, "bfloat16", page, 256, shuffle_seed=2).run(steps)
    U.check(folder, requests, got, "bfloat16", expect_all=False)


@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_in_graphs(name):
    """Three tokens of prompt, then a hundred and more one by one (captured as CUDA graphs after the
    second step), two requests of different age side by side."""
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    requests = _requests(name, 8, [140, 120])
    a, b = requests["r0"], requests["r1"]
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": a[:3], "want": [2]}], "end": []}]
    for i in range(3, 140):
        entries = [{"id": "r0", "tokens": [a[i]], "want": [0]}]
        j = i - 20
        if 0 <= j < 120:
            entries.append({"id": "r1", "tokens": [b[j]], "want": [0]})
        steps.append({"step": i, "entries": entries, "end": []})
    rep = H.Replayer(folder, "float32", page, 320, max_live=4)
    got = rep.run(steps)
    assert rep.runner._graphs, "no step was replayed from a CUDA graph"
    U.check(folder, requests, got, "float32", expect_all=False)


# ------------------------------------------------------------------------------ planted weights

def _planted(layer, seed, vocab=53, width=64):
    """Token 1's embedding lies along one direction, token 0's along a second one, every other token's is
    orthogonal to both; the convolutions pass the current token alone."""
    cfg = U.config([layer], vocab, width)
    t = {k: v.float() for k, v in U.random_tensors(cfg, seed).items()}
    t["embed"][:, :2] = 0.0
    t["embed"][:2] = 0.0
    t["embed"][1, 0] = 1.0
    t["embed"][0, 1] = 1.0
    t["l0.norm1"][:] = 0.0
    for n in "qkv":
        t[f"l0.mix.{n}.conv"][:] = 0.0
        t[f"l0.mix.{n}.conv"][:, -1] = 1.0
    return cfg, t


def _register(cfg, t, name):
    folder = H.tmp_root() / f"sizitar-planted-{name}"
    U.register(folder, cfg, {k: v.to(torch.bfloat16) for k, v in t.items()})
    return folder, cfg


def planted_attention(layer, seed, name):
    """Scores decided by two tokens: the query of a token 1 and the key of a token 0 point the same way in the
    entries that no rotation turns, so a token 1 finds the earlier tokens 0, however far back."""
    cfg, t = _planted(layer, seed)
    m = layer["mixer"]
    d = m["dim"]
    way = torch.zeros(d)
    way[m["rot"]["dims"]:] = 1.0
    q, k = t["l0.mix.q"].view(m["heads"], d, -1), t["l0.mix.k"].view(m["kv_heads"], d, -1)
    q[..., :2], k[..., :2] = 0.0, 0.0
    q[:, :, 0] = way
    k[:, :, 1] = way
    t["l0.mix.q.norm"][:], t["l0.mix.k.norm"][:] = 1.0, 1.0
    return _register(cfg, t, name)


def planted_state(layer, seed, name):
    """A delta layer that forgets almost nothing and in which only token 0 writes: its step size is one, every
    other token's nearly zero; the query of a token 1 is the key of a token 0."""
    cfg, t = _planted(layer, seed)
    m = layer["mixer"]
    t["l0.mix.A_log"][:] = -9.0
    t["embed"][2:, 2] = 2.0
    t["embed"][1, 2] = 1.0
    t["l0.mix.b"][:] = 0.0
    t["l0.mix.b"][:, 1] = 2.0
    t["l0.mix.b"][:, 2] = -5.0
    way = torch.randn(m["dim"], generator=torch.Generator().manual_seed(seed)).abs() + 0.2      # silu keeps what is positive
    q, k = t["l0.mix.q"].view(m["kv_heads"], m["dim"], -1), t["l0.mix.k"].view(m["kv_heads"], m["dim"], -1)
    q[..., :3], k[..., :3] = 0.0, 0.0
    q[:, :, 0] = way
    k[:, :, 1] = way
    return _register(cfg, t, name)


FAR = {"attention": (planted_attention, U.attention(2, 1, 64, 32, 2, 16, scale=0.5)),
       "attention_heads_of_128": (planted_attention, U.attention(4, 2, 128, 128, 3, 32, scale=0.2)),
       "delta": (planted_state, U.delta(4, 2, 16, 32, 3)),
       "channel_delta": (planted_state, U.channel_delta(2, 2, 32, 16, 2, 8)),
       "channel_delta_wide": (planted_state, U.channel_delta(2, 1, 128, 64, 2, 8))}


def moved(folder, cfg, ids, other, at):
    return H.row_error(P.forward(cfg, U._tensors[str(folder)], other)[at], U.plain_logits(folder, ids)[at])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(FAR))
def test_far_token_decides(kind, dtype):
    make, layer = FAR[kind]
    folder, cfg = make(layer, 21, "far-" + kind)
    rng = random.Random(2)
    filler = lambda n: [rng.randrange(2, cfg["vocab"]) for _ in range(n)]
    ids = filler(9) + [0] + filler(290) + [1] + filler(3)      # the far token is 291 positions back, pages and chunks away
    without = list(ids)
    without[9] = 5
    assert moved(folder, cfg, ids, without, 300) > 0.1
    requests = {"p": ids}
    got = H.Replayer(folder, dtype, 16, 304).run(H.trace_whole(requests))
    U.check(folder, requests, got, dtype)
    got = H.Replayer(folder, dtype, 16, 304, shuffle_seed=5).run(H.trace_decode_tail(requests, 8))
    U.check(folder, requests, got, dtype, expect_all=False)
    got = H.Replayer(folder, dtype, 16, 304, shuffle_seed=6).run(H.trace_portions(requests, random.Random(3)))
    U.check(folder, requests, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [U.attention(2, 1, 64, 64, 2, 8, scale=0.25), U.attention(4, 1, 128, 128, 2, 16, scale=0.2),
                                   U.attention(3, 3, 32, 16, 2, 8, scale=0.4)], ids=["64", "128", "values16"])
def test_one_in_the_denominator(layer, dtype, monkeypatch):
    """Every score far below zero: nearly all weight goes to the one, and the mixer adds almost nothing.  A plain
    softmax would average the values: the oracle with one moves the logits."""
    cfg, t = _planted(layer, 8)
    m = layer["mixer"]
    way = torch.zeros(m["dim"])
    way[m["rot"]["dims"]:] = 1.0
    t["embed"][:, 2] = 3.0
    q, k = t["l0.mix.q"].view(m["heads"], m["dim"], -1), t["l0.mix.k"].view(m["kv_heads"], m["dim"], -1)
    q *= 0.05
    k *= 0.05
    q[:, :, 2] += way
    k[:, :, 2] -= way
    t["l0.mix.q.norm"][:], t["l0.mix.k.norm"][:] = 1.0, 1.0
    t["l0.ls1"][:] = 2.0
    folder, cfg = _register(cfg, t, f"one-{m['dim']}-{m['vdim']}")
    ids = H.random_ids(random.Random(3), 150, cfg["vocab"])
    want = U.plain_logits(folder, ids)
    with monkeypatch.context() as patch:
        patch.setattr(P, "softmax_and_one", lambda s: torch.softmax(s, -1))
        other = P.forward(cfg, U._tensors[str(folder)], ids)
    assert H.row_error(other[149], want[149]) > 0.2 and H.row_error(other[0], want[0]) > 0.2
    requests = {"p": ids}
    got = H.Replayer(folder, dtype, 16, 160).run(H.trace_whole(requests))
    U.check(folder, requests, got, dtype)
    got = H.Replayer(folder, dtype, 16, 160, shuffle_seed=5).run(H.trace_decode_tail(requests, 40))
    U.check(folder, requests, got, dtype, expect_all=False)


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_at_page_borders(dtype):
    """The key that decides sits at a page's last or the next page's first position; it is asked for right
    behind the border, in the middle of the next page and from pages away, in prompts and in decoding."""
    folder, cfg = planted_attention(U.attention(2, 1, 64, 64, 2, 16, scale=0.5), 5, "borders")
    rng = random.Random(1)
    for at in (15, 16, 31, 32):
        for ask in (at + 1, at + 9, at + 40):
            ids = [rng.randrange(2, cfg["vocab"]) for _ in range(ask + 2)]
            ids[at], ids[ask] = 0, 1
            requests = {"p": ids}
            got = H.Replayer(folder, dtype, 16, 80, shuffle_seed=at).run(H.trace_whole(requests))
            U.check(folder, requests, got, dtype)
            got = H.Replayer(folder, dtype, 16, 80, shuffle_seed=at).run(H.trace_decode_tail(requests, 5))
            U.check(folder, requests, got, dtype, expect_all=False)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "channel_delta", "attention"])
def test_first_tokens_and_every_tap_of_the_convolution(kind, dtype):
    """A convolution of six taps whose every tap matters (equal weights): prompts shorter than its reach,
    portions that end inside it, and single tokens right after a slot's first token."""
    layer = {"delta": U.delta(2, 1, 8, 8, 6), "channel_delta": U.channel_delta(2, 2, 8, 8, 6, 4),
             "attention": U.attention(2, 1, 16, 16, 6, 8)}[kind]
    cfg = U.config([layer], 41, 48, eps=1e-5)
    t = U.random_tensors(cfg, 4)
    for n in "qkv":
        t[f"l0.mix.{n}.conv"] = torch.full_like(t[f"l0.mix.{n}.conv"], 0.5)
    folder = H.tmp_root() / f"sizitar-taps-{kind}"
    U.register(folder, cfg, t)
    ids = H.random_ids(random.Random(9), 23, 41)
    short = {f"s{n}": ids[:n] for n in (1, 2, 3, 5, 6, 7)}
    got = H.Replayer(folder, dtype, 16, 64, max_live=8).run(H.trace_whole(short))
    U.check(folder, short, got, dtype)
    for cut in ([1, 1, 1, 1, 1, 1, 1, 16], [2, 3, 1, 4, 13], [5, 1, 6, 11], [7, 16]):
        steps, at = [], 0
        for i, size in enumerate(cut):
            steps.append({"step": i, "entries": [{"id": "p", "tokens": ids[at: at + size], "want": list(range(size))}], "end": []})
            at += size
        got = H.Replayer(folder, dtype, 16, 32, shuffle_seed=1).run(steps)
        U.check(folder, {"p": ids}, got, dtype)


# ------------------------------------------------------------------------------ the entry point

@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(name):
    from bare_cuda_4gib_b200.engine.engine import LLMEngine
    folder, (cfg, page) = U.model_folder(name), U.CONFIGS[name]
    rng = random.Random(13)
    prompts = [H.random_ids(rng, n, cfg["vocab"]) for n in (5, 23, 1, 40, 12, 9)]
    engine = LLMEngine(str(folder), max_tokens=96, max_seqs=4, dtype="float32", page_tokens=page, max_step_tokens=24)
    out = engine.generate_batch(prompts, 24)
    alone = engine.generate(prompts[1], 24)
    assert alone == out[1]
    for prompt, new in zip(prompts, out):
        assert len(new) == 24
        logits = U.plain_logits(folder, prompt + new[:-1])
        for i, token in enumerate(new):
            row = logits[len(prompt) - 1 + i]
            best = int(row.argmax())
            if token != best:        # a tie within float32 rounding, or a router's close call, may go either way
                assert float(row[best] - row[token]) < 1e-3 * float(row.abs().max()), (i, token, best)


@pytest.mark.parametrize("name", ["A", "B"])
def test_layer_by_layer(name):
    """The model cut off after its first layer, its first two, and so on (float32): the first layer
    that differs from the plain implementation is the first cut that fails."""
    cfg, page = U.CONFIGS[name]
    tensors = U.random_tensors(cfg, 3)
    for n in range(1, len(cfg["layers"]) + 1):
        cut = dict(cfg, layers=copy.deepcopy(cfg["layers"][:n]), loop=None)
        kept = {k: v for k, v in tensors.items() if not k.startswith("l") or int(k[1:].split(".")[0]) < n}
        folder = H.tmp_root() / f"sizitar{name}-first{n}"
        U.register(folder, cut, kept)
        ids = U.clear_ids(folder, random.Random(3), 70, cfg["vocab"])
        got = H.Replayer(folder, "float32", page, 96).run(H.trace_whole({"p": ids}))
        U.check(folder, {"p": ids}, got, "float32")


# ------------------------------------------------------------------------- command line tools

def _tool(tool, *args, feed=None):
    import os
    import pathlib
    import subprocess
    import sys

    root = pathlib.Path(__file__).resolve().parents[1]
    done = subprocess.run([sys.executable, str(root / "bin" / tool), *map(str, args)], input=feed, capture_output=True,
                          text=True, env=dict(os.environ, PYTHONDONTWRITEBYTECODE="1"), timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    return done.stdout


def test_tools_run_a_preset_with_random_weights(tmp_path):
    out = _tool("llm-infer", "--model", tmp_path / "m", "--random", "sizitar-tiny", "--prompt", "1,2,3", "--tokens", 5)
    assert len(out.split("generated:")[1].split()) == 5
    out = _tool("llm-bench", "--model", tmp_path / "m", "--random", "sizitar-tiny", "--prompt-len", 24, "--tokens", 8,
                "--runs", 2, "--warmup", 1, "--page-tokens", 16)
    assert "TTFT" in out and "TPOT" in out


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_tool(dtype, tmp_path):
    """bin/trace_run on requests that share steps; the third takes the second one's slot and pages."""
    import numpy as np

    folder = U.model_folder("A", 3, dtype)
    requests = _requests("A", 17, [40, 19, 33], dtype)
    a, b, c = requests["r0"], requests["r1"], requests["r2"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [16]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[30:39], "want": []}, {"id": "c", "tokens": c, "want": [32]}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[39:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    printed = _tool("trace_run", "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", 128, "--page-tokens", 16,
                    feed="".join(json.dumps(s) + "\n" for s in steps))
    assert [l for l in printed.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    want = {0: [("r0", 0), ("r0", 29), ("r1", 1)], 1: [("r1", 18)], 2: [("r2", 32)], 3: [("r0", 39)]}
    vocab = U.CONFIGS["A"][0]["vocab"]
    for step, rows in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), vocab).copy())
        for i, (rid, p) in enumerate(rows):
            err = H.row_error(got[i], U.plain_logits(folder, requests[rid])[p])
            assert err <= U.TOLERANCE[dtype], (step, rid, p, err)
