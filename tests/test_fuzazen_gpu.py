"""The Fuzazen decoder in the engine against the plain implementation (`plain_fuzazen`): every
mechanism alone, every way of cutting requests into steps, slots and pages used again, planted
weights where random ones would hide a fault, and greedy generation through the entry point."""

import copy
import json
import math
import random

import pytest
import torch

import fuzazen_helpers as U
import helpers as H
import plain_fuzazen as P

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
LENGTHS = {"F": [1, 2, 3, 17, 33, 70, 150], "G": [2, 5, 31, 64, 65, 200]}


def _requests(name, seed, lengths):
    rng = random.Random(seed)
    vocab = U.CONFIGS[name][0]["vocab"]
    return {f"r{i}": H.random_ids(rng, n, vocab) for i, n in enumerate(lengths)}


# --------------------------------------------------------------------- mechanisms, one at a time

def _model(name, layers, seed, width=72, vocab=61, **constants):
    cfg = U.model(layers, width, vocab, **constants)
    folder = H.tmp_root() / f"fuzazen-one-{name}"
    U.register(folder, cfg, U.random_tensors(cfg, seed))
    return folder, cfg


ALONE = {
    "attention": ([U.attention(4, 2, 16, 24, 20, 8)], {}),
    "whole_turn_one_key_head": ([U.attention(3, 1, 48, 16, 37, 48, base=300.0, scale=0.3)], {}),
    "two_entries_turned": ([U.attention(2, 2, 32, 32, 40, 2, base=5.0)], {}),
    "odd_sizes": ([U.attention(2, 2, 10, 33, 7, 4, scale=0.5)], {}),                # no tensor-core kernel takes these
    "heads_of_64": ([U.attention(4, 2, 64, 64, 33, 32, scale=0.2)], {}),           # the tcgen05 and cluster decode kernels
    "heads_of_128": ([U.attention(4, 1, 128, 128, 70, 64, scale=0.1)], {}),
    "many_heads_of_64": ([U.attention(20, 1, 64, 64, 50, 16, scale=0.2)], {}),      # one token fills more than one tile of 16 rows
    "many_heads": ([U.attention(24, 2, 16, 48, 45, 16)], {}),
    "wide_values": ([U.attention(2, 1, 64, 256, 33, 32, scale=0.2)], {}),
    "narrow_keys_wide_values": ([U.attention(4, 4, 16, 128, 64, 8)], {}),
    "block_of_one": ([U.attention(2, 2, 16, 16, 1, 16)], {}),                       # every token sees itself and the sink
    "block_beyond_the_request": ([U.attention(4, 2, 32, 48, 4096, 32)], {}),
    "block_of_a_page": ([U.attention(2, 1, 64, 48, 16, 16, scale=0.2)], {}),
    "block_of_a_key_block": ([U.attention(2, 1, 64, 64, 64, 16, scale=0.2)], {}),
    "with_dense": ([U.attention(4, 4, 32, 64, 40, 32, ff=100)], {}),
    "run_again": ([U.attention(4, 2, 16, 32, 30, 8, ff=64), U.again(U.attention(4, 2, 16, 32, 30, 8, ff=64), 0)], {}),
    "run_before_its_owner": ([U.again(U.attention(2, 1, 16, 16, 9, 8), 1), U.attention(2, 1, 16, 16, 9, 8)], {}),
    "factors": ([U.attention(2, 1, 32, 16, 25, 16, ff=40)], dict(scale=6.0, mult=0.11, cap=50.0, eps=1e-2)),
    "tight_cap": ([U.attention(2, 1, 32, 16, 25, 16, ff=40)], dict(cap=1.0, mult=2.0)),
    "no_cap": ([U.attention(2, 1, 32, 16, 25, 16)], dict(cap=None)),
    "width_50": ([U.attention(3, 3, 12, 20, 17, 6, ff=34)], dict(width=50)),        # nothing lines up with 16 bytes
    "width_192": ([U.attention(9, 3, 64, 32, 60, 40, scale=0.15, ff=288)], dict(width=192)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(ALONE))
def test_each_mechanism_alone(which, dtype):
    layers, constants = ALONE[which]
    folder, cfg = _model(which, layers, 11, **constants)
    rng = random.Random(5)
    requests = {"a": H.random_ids(rng, 90, cfg["vocab"]), "b": H.random_ids(rng, 1, cfg["vocab"])}
    steps = H.trace_whole(requests)
    got = H.Replayer(folder, dtype, 16, H.peak_tokens(steps, 16)).run(steps)
    U.check(folder, requests, got, dtype)
    # the same tokens in portions and one by one give the same logits
    steps = H.trace_portions({"a": requests["a"]}, random.Random(1))
    got = H.Replayer(folder, dtype, 16, 96, shuffle_seed=2).run(steps)
    U.check(folder, {"a": requests["a"]}, got, dtype)
    got = H.Replayer(folder, dtype, 16, 96, shuffle_seed=3).run(H.trace_decode_tail({"a": requests["a"]}, 60))
    U.check(folder, {"a": requests["a"]}, got, dtype, expect_all=False)


def _attention_case(seqs, heads, kv_heads, d, dv, page, dtype, window=0, chunk=0, sink=None, gate=False, plain=False, seed=0):
    """(what the attention kernel gives, what it should, the step's plan) for requests (tokens, length)
    over a cache of random keys and values; pages that no query can see are gone, and a page behind a
    request's last key holds NaN.  `sink`: the size of the random sinks, or None."""
    from bare_cuda_4gib_b200.kernels import attention as fast, biased_attention as BA, gemm, lib as K

    g = torch.Generator().manual_seed(seed)
    rnd = lambda *shape: torch.randn(*shape, generator=g).to(dtype)
    blocks = [-(-kv // page) for _, kv in seqs]
    n_pages = sum(blocks) + 1
    k_elems, v_elems = kv_heads * page * d, kv_heads * page * dv
    storage = torch.full((n_pages, k_elems + v_elems), float("nan"), dtype=dtype)
    table = torch.full((len(seqs), max(blocks) + 1), -1, dtype=torch.int32)
    order = torch.randperm(n_pages - 1, generator=g).tolist()
    ks, vs = [], []
    for s, (q_len, kv) in enumerate(seqs):
        k, v = rnd(kv, kv_heads, d), rnd(kv, kv_heads, dv)
        first = kv - q_len                                  # what the step's first query sees is the oldest needed
        oldest = max(0, first - window + 1 if window else 0, first - first % chunk if chunk else 0)
        for b in range(blocks[s]):
            page_id = order.pop()
            lo, hi = b * page, min(kv, (b + 1) * page)
            storage[page_id, :k_elems].view(kv_heads, page, d)[:, : hi - lo] = k[lo:hi].transpose(0, 1)
            storage[page_id, k_elems:].view(kv_heads, page, dv)[:, : hi - lo] = v[lo:hi].transpose(0, 1)
            if hi > oldest:
                table[s, b] = page_id
        ks.append(k.double())
        vs.append(v.double())
    storage, table = storage.cuda(), table.cuda()
    esize = storage.element_size()
    view = K.CacheView(storage.data_ptr(), storage.data_ptr() + k_elems * esize, table, k_elems + v_elems, table.shape[1], page,
                       kv_heads, d, dtype, storage.data_ptr(), storage.numel(), v_dim=dv)
    n = sum(q for q, _ in seqs)
    q = rnd(n, heads, d)
    sinks = torch.randn(heads, generator=g) * sink if sink is not None else None
    wide = rnd(n, heads + 5)                                # the gate is a column view of a wider matrix
    starts = [sum(a for a, _ in seqs[:i]) for i in range(len(seqs))]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")

    from bare_cuda_4gib_b200.engine.step import StepContext, Workspace
    ctx = StepContext()
    ctx.stream = torch.cuda.current_stream().cuda_stream
    ctx.ws, ctx.n_tokens, ctx.max_rows, ctx.max_seqs = Workspace("cuda", n), n, n, len(seqs)
    ctx.seq_q_start, ctx.seq_q_len, ctx.seq_kv_len = i32(starts), i32([a for a, _ in seqs]), i32([b for _, b in seqs])
    ctx.positions = i32([p for a, b in seqs for p in range(b - a, b)])
    ctx.row_seq = i32([s for s, (a, _) in enumerate(seqs) for _ in range(a)])
    ctx.token_ids = i32([0])
    ctx.host_q_len, ctx.host_kv_len = [a for a, _ in seqs], [b for _, b in seqs]
    ctx.max_q_len, ctx.max_kv_len = max(ctx.host_q_len), max(ctx.host_kv_len)
    wide_dev = wide.cuda()
    extras = K.AttentionExtras(chunk, sinks.cuda() if sinks is not None else None, wide_dev[:, 2: 2 + heads] if gate else None)
    out = torch.full((n, heads * dv), float("nan"), dtype=dtype, device="cuda")
    scale = 1.0 / math.sqrt(d)
    if plain:
        BA.attention(ctx, q.cuda().view(n, heads * d), out, view, None, heads, scale, window, 1.0, 0.0, extras)
    else:
        plan = fast.plan_for(d, heads, kv_heads, False, dv, 0.0, window, chunk)
        fast.run(ctx, plan, q.cuda().view(n, heads * d), out, view, scale, window, extras=extras)
        gemm.check_errors()
    want = torch.zeros(n, heads, dv, dtype=torch.float64)
    for s, (q_len, kv) in enumerate(seqs):
        mask = P.seen(kv, chunk or None)
        if window:
            p = torch.arange(kv)
            mask = mask & (p[:, None] - p[None, :] < window)
        mask = mask[kv - q_len:]
        for h in range(heads):
            kvh = h // (heads // kv_heads)
            rows = slice(starts[s], starts[s] + q_len)
            o = P.one_head(q[rows, h].double(), ks[s][:, kvh], vs[s][:, kvh], scale, mask,
                           sinks[h].double() if sinks is not None else torch.tensor(-1e9, dtype=torch.float64))
            want[rows, h] = o * torch.sigmoid(wide[rows, 2 + h: 3 + h].double()) if gate else o
    return out.view(n, heads, dv), want, ctx


def _close(got, want, tol):
    diff = (got.double().cpu() - want).abs()
    assert not torch.isnan(diff).any()
    assert float(diff.max()) <= 1e-7 + tol * float(want.abs().max()), float(diff.max() / want.abs().max())


PREFILL = [(37, 37), (5, 133), (1, 70), (64, 64), (2, 2), (1, 1), (19, 300)]
SINGLE = [(1, 500), (1, 1), (1, 65), (1, 64), (1, 129), (1, 333), (1, 100)]
SHAPES = [(8, 2, 64, 64, 16), (8, 1, 64, 64, 64), (4, 2, 128, 128, 32), (6, 3, 32, 32, 16), (4, 2, 64, 48, 64), (3, 1, 112, 80, 16),
          (20, 1, 64, 64, 16), (12, 1, 16, 128, 32)]


@pytest.mark.parametrize("heads,kv_heads,d,dv,page", SHAPES)
@pytest.mark.parametrize("options", [dict(chunk=50, sink=2.0, gate=True), dict(chunk=64), dict(sink=1.0), dict(gate=True),
                                     dict(chunk=100, window=30, sink=3.0), dict(chunk=1, sink=0.5), dict(window=40, gate=True),
                                     dict(chunk=129, sink=200.0)])
def test_attention_kernels_with_blocks_sinks_and_gates(heads, kv_heads, d, dv, page, options):
    """Each option alone and together, in the tensor-core kernels' prefill and single-token shapes.  Sinks of
    size 200 leave some heads with the sink alone and others without it."""
    for seqs in (PREFILL, SINGLE):
        got, want, _ = _attention_case(seqs, heads, kv_heads, d, dv, page, torch.bfloat16, seed=heads + d + page, **options)
        _close(got, want, 1.5e-2)


@pytest.mark.parametrize("options", [dict(chunk=50, sink=2.0, gate=True), dict(chunk=100, window=30, sink=3.0), dict(gate=True),
                                     dict(chunk=7, sink=200.0, gate=True)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1.5e-2)])
def test_plain_attention_kernel_with_blocks_sinks_and_gates(dtype, tol, options):
    for heads, kv_heads, d, dv, page in [(4, 2, 10, 33, 16), (3, 3, 64, 48, 32), (2, 1, 24, 200, 16)]:
        got, want, _ = _attention_case(PREFILL + [(1, 200)], heads, kv_heads, d, dv, page, dtype, plain=True, seed=d, **options)
        _close(got, want, tol)


def test_single_token_steps_split_keys_no_more_often_than_a_block_has_them():
    """A block of 256 positions has few key blocks: a step at position 3,000 splits them, and every split
    count gives the same."""
    for chunk in (0, 256, 1000):
        got, want, ctx = _attention_case([(1, 3000), (2, 2500)], 4, 1, 48, 64, 64, torch.bfloat16, chunk=chunk, sink=1.0, gate=True, seed=chunk)
        _close(got, want, 1.5e-2)
        (plan,) = [v for k, v in ctx.extras.items() if k[0] == "attention_tiles"]
        assert plan[3] == 16 and 1 < plan[4] <= (-(-chunk // 64) + 1 if chunk else 47), plan[3:]


def test_long_prompts_in_blocks():
    """Prompts of over a thousand tokens whose blocks end inside a tile's keys and rows, after long prefixes."""
    for heads, kv_heads, d in ((8, 2, 64), (4, 2, 128), (4, 2, 96)):
        got, want, _ = _attention_case([(1100, 1100), (300, 1500), (5, 1900), (130, 641)], heads, kv_heads, d, d, 64, torch.bfloat16,
                                       chunk=333, sink=1.0, gate=True, seed=d)
        _close(got, want, 1.5e-2)


@pytest.mark.parametrize("n", [9, 90])
@pytest.mark.parametrize("width", [52, 256, 50, 1100, 2048, 4096, 6000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_stream_kernels(dtype, width, n):
    """x + m * rms_norm(y) * w with the new stream handed on un-normed, and the stream alone."""
    from bare_cuda_4gib_b200.kernels import lib as K, sandwich as SW
    g = torch.Generator().manual_seed(4)
    x = torch.randn(n, width, generator=g)
    y = torch.randn(3, n, width, generator=g)                # three partial sums
    w = torch.randn(width, generator=g).to(dtype)
    want = P.add_normed(x.double(), y.double().sum(0), w.double(), 0.3, 1e-3)
    res, out = x.cuda(), torch.empty(n, width, dtype=dtype, device="cuda")
    SW.postnorm_add_rmsnorm(res, SW.NormedDelta(K.Partials(y.cuda(), 3), w.cuda(), 1e-3, 0.3), None, out, 0.0, n)
    assert H.row_error(res, want) < 1e-6
    assert torch.equal(out.cpu(), res.cpu().to(dtype))
    SW.postnorm_add_rmsnorm(res, None, None, out, 0.0, n)   # nothing to add
    assert H.row_error(res, want) < 1e-6 and torch.equal(out.cpu(), res.cpu().to(dtype))
    rows = torch.tensor([7, 2], dtype=torch.int32, device="cuda")
    res, out = x.cuda(), torch.empty(2, width, dtype=dtype, device="cuda")
    SW.postnorm_add_rmsnorm(res, SW.NormedDelta(K.Partials(y.cuda(), 3), w.cuda(), 1e-3, 0.3), w.cuda(), out, 1e-2, 2, rows)
    normed = P.unit_rms(want[[7, 2]], 1e-2) * w.double()
    assert H.row_error(out, normed) < (1e-6 if dtype == torch.float32 else 5e-3) and torch.equal(res[0].cpu(), x[0])


def test_cap_on_the_logits():
    from bare_cuda_4gib_b200.kernels import lib as K
    for rows, vocab in ((1, 1), (1, 3), (3, 33), (5, 1000), (64, 32000)):
        z = torch.randn(rows, vocab, generator=torch.Generator().manual_seed(vocab)) * 40.0
        x = z.cuda()
        K.softcap_rows(x, 7.5, rows)
        assert float((x.double().cpu() - P.capped(z.double(), 7.5)).abs().max()) < 2e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [11, 300])
@pytest.mark.parametrize("d,rot,dv,spare", [(64, 64, 24, 0), (48, 16, 20, 3), (10, 4, 20, 3), (128, 2, 64, 8), (8, 6, 8, 0), (256, 100, 16, 0),
                                            (16, 16, 40, 5), (32, 10, 32, 8)])
def test_heads_of_unit_size_after_the_turn(dtype, d, rot, dv, spare, n):
    """Queries and keys turned and then divided by their root mean square, written to buffer and page, by the
    kernel in pieces of 16 bytes (where rows and sizes allow it) and by the other; with weights instead, too."""
    from bare_cuda_4gib_b200.kernels import head_prepare as HP, lib as K
    g = torch.Generator().manual_seed(d)
    heads, kv_heads, page, eps = 3, 2, 8, 1e-2
    u = torch.randn(n, heads * d + kv_heads * (d + dv) + spare, generator=g).to(dtype)
    elems = kv_heads * page * (d + dv)
    blocks = -(-n // page)
    pages = torch.randperm(blocks + 1, generator=g)[:blocks]
    storage = torch.zeros(blocks + 1, elems, dtype=dtype, device="cuda")
    table = pages.to(torch.int32)[None].cuda()
    view = K.CacheView(storage.data_ptr(), storage.data_ptr() + kv_heads * page * d * storage.element_size(), table, elems, blocks, page,
                       kv_heads, d, dtype, v_dim=dv)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")

    class Ctx:
        stream = torch.cuda.current_stream().cuda_stream
        positions, row_seq, n_tokens = i32(list(range(n))), i32([0] * n), n

    freq = torch.tensor([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)], device="cuda")
    q = torch.empty(n, heads * d, dtype=dtype, device="cuda")
    HP.headnorm_rope_cache(Ctx, u.cuda(), 0, heads * d, (heads + kv_heads) * d, None, None, eps, freq, rot, 1.0, q, view, heads, True,
                           unit_norm=True)
    tol = 3e-5 if dtype == torch.float32 else 5e-3        # an angle of 300 in float32 is off by 2e-5
    ud, pos = u.double(), torch.arange(n)
    want = P.unit_rms(P.turn_pairs(ud[:, : heads * d].reshape(n, heads, d), pos, 300.0, rot), eps)
    assert H.row_error(q.view(n, heads, d), want) < tol
    want_k = P.unit_rms(P.turn_pairs(ud[:, heads * d: (heads + kv_heads) * d].reshape(n, kv_heads, d), pos, 300.0, rot), eps)
    cells = storage.cpu()[pages]
    keys = torch.cat([c[: kv_heads * page * d].view(kv_heads, page, d) for c in cells], 1)[:, :n].transpose(0, 1)
    values = torch.cat([c[kv_heads * page * d:].view(kv_heads, page, dv) for c in cells], 1)[:, :n].transpose(0, 1)
    assert H.row_error(keys, want_k) < tol
    first = (heads + kv_heads) * d
    assert torch.equal(values, u[:, first: first + kv_heads * dv].reshape(n, kv_heads, dv))
    # with a weight per projection the norm comes before the turn; keys stay away from a cache that is only read
    wq, wk = (1.0 + 0.3 * torch.randn(2, d, generator=g)).to(dtype)
    storage.zero_()
    HP.headnorm_rope_cache(Ctx, u.cuda(), 0, heads * d, (heads + kv_heads) * d, wq.cuda(), wk.cuda(), eps, freq, rot, 1.5, q, view, heads, False)
    normed = P.unit_rms(ud[:, : heads * d].reshape(n, heads, d), eps) * wq.double()
    want = P.turn_pairs(normed, pos, 300.0, rot)
    want[..., :rot] *= 1.5
    assert H.row_error(q.view(n, heads, d), want) < tol and float(storage.abs().max()) == 0.0


# ------------------------------------------------------------------ every cutting, two configs

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_whole(name, dtype):
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    requests = _requests(name, 1, LENGTHS[name])
    steps = H.trace_whole(requests)
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page)).run(steps)
    U.check(folder, requests, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_prefill_then_token_by_token(name, dtype):
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    requests = _requests(name, 2, LENGTHS[name][3:])
    steps = H.trace_decode_tail(requests, 70)          # blocks' edges pass over decoded tokens
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page), shuffle_seed=3).run(steps)
    U.check(folder, requests, got, dtype, expect_all=False)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_portions_down_to_two_tokens(name, dtype):
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    requests = _requests(name, 3, LENGTHS[name][2:])
    steps = H.trace_portions(requests, random.Random(5))
    got = H.Replayer(folder, dtype, page, H.peak_tokens(steps, page), shuffle_seed=4).run(steps)
    U.check(folder, requests, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_portions_of_two(name, dtype):
    """Every step brings two tokens (the last one perhaps one)."""
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    ids = _requests(name, 12, [105])["r0"]
    steps = [{"step": i, "entries": [{"id": "r0", "tokens": ids[at: at + 2], "want": list(range(len(ids[at: at + 2])))}], "end": []}
             for i, at in enumerate(range(0, len(ids), 2))]
    got = H.Replayer(folder, dtype, page, 128, shuffle_seed=8).run(steps)
    U.check(folder, {"r0": ids}, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_mixed_batches_reuse_slots_and_pages(name, dtype):
    """Unequal requests side by side, four slots and a small pool for eleven requests: every logit
    equals the request's alone, whatever slot and pages it got and whoever held them before."""
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    longest = 160
    rng = random.Random(11)
    requests = _requests(name, 4, [rng.randrange(3, longest // 2) for _ in range(10)] + [longest])
    budget = 2 * longest
    steps = H.trace_mixed(requests, random.Random(6), live=4, budget_tokens=budget, page=page)
    rep = H.Replayer(folder, dtype, page, budget, max_live=4, shuffle_seed=9)
    got = rep.run(steps)
    U.check(folder, requests, got, dtype)
    for group in rep.cache.groups:
        assert group.pool.acquired_total > group.pool.num_pages and group.pool.pages_in_use == 0
    assert rep.cache.free_slots == 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F", "G"])
def test_long_decoding_in_graphs(name, dtype):
    """Three tokens of prompt, then well over a hundred one by one (captured as CUDA graphs after the
    second step), two requests of different age side by side, so that their blocks end at different steps."""
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    requests = _requests(name, 8, [210, 180])
    a, b = requests["r0"], requests["r1"]
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": a[:3], "want": [2]}], "end": []}]
    for i in range(3, 210):
        entries = [{"id": "r0", "tokens": [a[i]], "want": [0]}]
        j = i - 20
        if j == 0:
            entries.append({"id": "r1", "tokens": b[:1], "want": [0]})
        elif 0 < j < 180:
            entries.append({"id": "r1", "tokens": [b[j]], "want": [0]})
        steps.append({"step": i, "entries": entries, "end": []})
    rep = H.Replayer(folder, dtype, page, 448, max_live=4)
    got = rep.run(steps)
    assert rep.runner._graphs, "no step was replayed from a CUDA graph"
    U.check(folder, requests, got, dtype, expect_all=False)


@pytest.mark.parametrize("name", ["F", "G"])
def test_pages_of_passed_blocks_are_given_back(name):
    """Long after its blocks have ended a request holds no more pages than one block and the next step take."""
    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    ids = _requests(name, 9, [240])["r0"]
    rep = H.Replayer(folder, "float32", page, 256)
    got = rep.run(H.trace_decode_tail({"r0": ids}, 200)[:-1])
    U.check(folder, {"r0": ids}, got, "float32", expect_all=False)
    for group in rep.cache.groups:
        assert group.pool.pages_in_use <= -(-(group.request.window + 1) // page) + 1


# ------------------------------------------------------------------------------ planted weights

PLANTED_FAR = {"value_size": U.attention(2, 1, 64, 32, 400, 16, scale=0.5), "tensor_memory": U.attention(2, 1, 64, 64, 310, 16, scale=0.5),
               "heads_of_128": U.attention(4, 2, 128, 128, 512, 32, scale=0.2), "plain_kernel": U.attention(2, 1, 40, 33, 350, 8, scale=0.6)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(PLANTED_FAR))
def test_far_key_decides(kind, dtype):
    folder, cfg = U.planted(PLANTED_FAR[kind], 21, "far-" + kind)
    rng = random.Random(2)
    filler = lambda n: [rng.randrange(2, cfg["vocab"]) for _ in range(n)]
    ids = filler(9) + [0] + filler(290) + [1] + filler(3)      # the far key is 291 positions back, pages away
    without = list(ids)
    without[9] = 5
    assert U.moved(folder, cfg, ids, without, 300) > 0.1
    requests = {"p": ids}
    got = H.Replayer(folder, dtype, 16, 304).run(H.trace_whole(requests))
    U.check(folder, requests, got, dtype)
    got = H.Replayer(folder, dtype, 16, 304, shuffle_seed=5).run(H.trace_decode_tail(requests, 8))
    U.check(folder, requests, got, dtype, expect_all=False)
    got = H.Replayer(folder, dtype, 16, 304, shuffle_seed=6).run(H.trace_portions(requests, random.Random(3)))
    U.check(folder, requests, got, dtype)


# (layer, where the planted key is): it opens a block, or is the last of one, at page and key-block borders or not
EDGES = [(U.attention(2, 1, 64, 32, 50, 16, scale=0.5), 100), (U.attention(2, 1, 64, 64, 64, 16, scale=0.5), 128),
         (U.attention(2, 2, 32, 64, 16, 8, scale=0.7), 64), (U.attention(4, 1, 128, 128, 37, 64, scale=0.2), 111),
         (U.attention(3, 3, 40, 24, 21, 8, scale=0.6), 84), (U.attention(8, 1, 64, 64, 129, 4, scale=0.4), 129)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(EDGES)))
def test_block_edges(i, dtype):
    """A planted key at a block's first position, asked for by the block's last position (which sees it)
    and by the next block's first (which does not, though it is nearer than some that did), in a prompt,
    in a portion that starts between the two, and for a token decoded alone."""
    layer, start = EDGES[i]
    size = layer["mixer"]["mask"]["size"]
    folder, cfg = U.planted(layer, 23, f"edge{i}")
    rng = random.Random(6)
    filler = lambda n: [rng.randrange(2, cfg["vocab"]) for _ in range(n)]
    ids = filler(start) + [0] + filler(size - 2) + [1, 1] + filler(5)
    inside, outside = start + size - 1, start + size
    without = list(ids)
    without[start] = 7
    assert U.moved(folder, cfg, ids, without, inside) > 0.1 and U.moved(folder, cfg, ids, without, outside) < 1e-9
    # ... and a key on the last position before the block, one place back, is not seen at all
    before = filler(start - 1) + [0, 1] + filler(3)
    other = list(before)
    other[start - 1] = 7
    assert U.moved(folder, cfg, before, other, start) < 1e-9
    requests = {"p": ids, "b": before}
    got = H.Replayer(folder, dtype, 16, 288).run(H.trace_whole(requests))
    U.check(folder, requests, got, dtype)
    cut = inside - 1
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": ids[:cut], "want": [cut - 1]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": ids[cut: outside + 3], "want": list(range(outside + 3 - cut))}], "end": ["p"]}]
    got = H.Replayer(folder, dtype, 16, 288, shuffle_seed=3).run(steps)
    U.check(folder, requests, got, dtype, expect_all=False)
    got = H.Replayer(folder, dtype, 16, 288, shuffle_seed=4).run(H.trace_decode_tail(requests, 9))
    U.check(folder, requests, got, dtype, expect_all=False)
    assert {("p", inside), ("p", outside)} <= set(got)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(64, 32), (64, 64), (40, 24)])
def test_sink_takes_its_share(dims, dtype):
    """A sink as large as the planted key's score halves that key's weight, here in one head of two (the norm
    behind the mixer would undo it in both); without it the logits would be others.  At a sequence's first
    tokens the sink is most of the sum."""
    d, dv = dims
    layer = U.attention(2, 1, d, dv, 90, 8, scale=0.25)
    level = d * 0.25
    folder, cfg = U.planted(layer, 31, f"sink-{d}-{dv}", sink=[level, -100.0])
    bare, _ = U.planted(layer, 31, f"no-sink-{d}-{dv}", sink=[-100.0, -100.0])
    rng = random.Random(4)
    ids = [1, 0, 1] + [rng.randrange(2, cfg["vocab"]) for _ in range(60)] + [1, 5, 1]
    for at in (0, 1, 2, 63, 65):
        assert H.row_error(U.plain_logits(bare, ids)[at], U.plain_logits(folder, ids)[at]) > 0.1, at
    for f in (folder, bare):
        got = H.Replayer(f, dtype, 16, 80).run(H.trace_whole({"p": ids}))
        U.check(f, {"p": ids}, got, dtype)
        got = H.Replayer(f, dtype, 16, 80, shuffle_seed=2).run(H.trace_decode_tail({"p": ids}, 65))
        U.check(f, {"p": ids}, got, dtype, expect_all=False)


# ----------------------------------------------------------------- the entry point and scheduler

@pytest.mark.parametrize("name", ["F", "G"])
def test_greedy_generation_through_the_engine(name):
    from bare_cuda_4gib_b200.engine.engine import LLMEngine

    folder, page = U.model_folder(name), U.CONFIGS[name][1]
    cfg = U.CONFIGS[name][0]
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
            if token != best:        # a tie within float32 rounding may go either way
                assert float(row[best] - row[token]) < 1e-4 * float(row.abs().max()), (i, token, best)


@pytest.mark.parametrize("name", ["F", "G"])
def test_layer_by_layer(name):
    """The model cut off after its first layer, its first two, and so on (float32): the first layer
    that differs from the plain implementation is the first cut that fails."""
    cfg, page = U.CONFIGS[name]
    tensors = U.random_tensors(cfg, 3)
    ids = H.random_ids(random.Random(3), 70, cfg["vocab"])
    for n in range(1, len(cfg["layers"]) + 1):
        layers = copy.deepcopy(cfg["layers"][:n])
        if any(layer.get("weights_of", 0) >= n for layer in layers):
            continue                 # the tensors' owner stands behind the cut
        owners = [f"l{i}." for i, layer in enumerate(layers) if "weights_of" not in layer]
        kept = {k: v for k, v in tensors.items() if k[:2] not in {f"l{i}" for i in range(9)} or k.startswith(tuple(owners))}
        folder = H.tmp_root() / f"fuzazen{name}-first{n}"
        U.register(folder, dict(cfg, layers=layers), kept)
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


def test_llm_infer_prints_the_plain_greedy_tokens():
    folder = U.model_folder("G")
    prompt = [5, 17, 3, 60, 9, 41, 76]
    out = _tool("llm-infer", "--model", folder, "--prompt", ",".join(map(str, prompt)), "--tokens", 10, "--dtype",
                "float32", "--page-tokens", 32)
    generated = [int(t) for t in out.split("generated:")[1].split()]
    assert len(generated) == 10
    logits = U.plain_logits(folder, prompt + generated[:-1])
    assert generated == [int(logits[len(prompt) - 1 + i].argmax()) for i in range(10)]


def test_tools_run_a_preset_with_random_weights(tmp_path):
    out = _tool("llm-infer", "--model", tmp_path / "m", "--random", "fuzazen-tiny", "--prompt", "1,2,3", "--tokens", 5)
    assert len(out.split("generated:")[1].split()) == 5
    out = _tool("llm-bench", "--model", tmp_path / "m", "--random", "fuzazen-tiny", "--prompt-len", 24, "--tokens", 8,
                "--runs", 2, "--warmup", 1, "--page-tokens", 16)
    assert "TTFT" in out and "TPOT" in out


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_tool(dtype, tmp_path):
    """bin/trace_run on requests that share steps; the third takes the second one's slot and pages."""
    import numpy as np

    folder = U.model_folder("F")
    requests = _requests("F", 17, [40, 19, 33])
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
    vocab = U.CONFIGS["F"][0]["vocab"]
    for step, rows in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), vocab).copy())
        for i, (rid, p) in enumerate(rows):
            err = H.row_error(got[i], U.plain_logits(folder, requests[rid])[p])
            assert err <= U.TOLERANCE[dtype], (step, rid, p, err)
