"""Ludelorn on the GPU against the plain implementation: every mechanism's kernel alone, then whole models cut into
steps in every way, then generation through the entry point.

Kernel tests build their own index arrays and pages (handed out shuffled) and compare with the functions of
``plain_ludelorn`` in float64.  Where random numbers would hide a fault (a window that is one position off, a pooled
block that is seen too early, a sink that is left out) one key or block is made to stand out.  Model tests make small
model folders of four configurations that differ in every size and option and replay requests whole, with a decoded
tail, in portions down to two tokens, and mixed with few pages and slots.
"""

import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_ludelorn as plain
import traces
from ludelorn_models import ludelorn_dir, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def shuffled_table(rows, page, seed, spare=3):
    """(table int32 [1, pages], row -> (page, place)) for one request whose pages lie anywhere in the pool."""
    pages = -(-rows // page)
    perm = torch.randperm(pages + spare, generator=torch.Generator().manual_seed(seed))[:pages]
    return perm.to(torch.int32).reshape(1, -1).to(DEV), lambda r: (int(perm[r // page]), r % page)


def filled_pool(rows, table, place, page, spare=3):
    """A pool [pages, heads, page, size] that holds ``rows`` [n, heads, size]; everything else is NaN."""
    pool = torch.full((table.shape[1] + spare, rows.shape[1], page, rows.shape[2]), float("nan"), dtype=rows.dtype)
    for r in range(rows.shape[0]):
        pg, at = place(r)
        pool[pg, :, at] = rows[r]
    return pool.to(DEV)


# ---- heads between the input product and the attention -----------------------------------------------------------

@pytest.mark.parametrize("dtype, n, nq, nk, d, e, dims, interleaved, over_all, magnitude", [
    (torch.float32, 21, 3, 1, 10, 6, 6, True, True, 1.0), (torch.float32, 21, 4, 2, 16, 16, 16, False, False, 1.3),
    (torch.float32, 5, 6, 3, 12, 20, 12, True, True, 1.2), (torch.bfloat16, 21, 4, 2, 64, 32, 32, True, True, 1.0),
    (torch.bfloat16, 700, 4, 2, 24, 8, 24, False, True, 1.1), (torch.float32, 400, 2, 2, 8, 8, 2, True, True, 0.9)])
def test_heads_are_normed_one_by_one_or_all_at_once_and_turned(dtype, n, nq, nk, d, e, dims, interleaved, over_all, magnitude):
    from yalis_b200.ops.elementwise import qkv_prepare
    g = torch.Generator().manual_seed(d + dims + n)
    page, start = 8, 300
    table, place = shuffled_table(start + n, page, seed=2)
    q_off, k_off, v_off = 8, 8 + nq * d + 3, 8 + nq * d + 3 + nk * d + 5
    src = (torch.randn(n, v_off + nk * e + 3, generator=g) * 2).to(dtype)
    src[:, q_off:q_off + d] *= 3                       # one head larger than the others: the two norms differ
    qn, kn = (1 + 0.3 * torch.randn(h * d if over_all else d, generator=g) for h in (nq, nk))
    freq = plain.plain_frequencies(dims, 50.0)
    k_pool = torch.full((table.shape[1] + 3, nk, page, d), 7.0, dtype=dtype, device=DEV)
    v_pool = torch.full((table.shape[1] + 3, nk, page, e), 7.0, dtype=dtype, device=DEV)
    positions = torch.arange(start, start + n)
    q = qkv_prepare(src.to(DEV), (q_off, k_off, v_off), nq, nk, d, e, i32(positions.tolist()), i32([0] * n), out_dtype=dtype,
                    q_norm=qn.to(DEV), k_norm=kn.to(DEV), norm_eps=1e-3, inv_freq=torch.tensor(freq).float().to(DEV), k_pool=k_pool,
                    v_pool=v_pool, block_table=table, interleaved=interleaved, rot_scale=magnitude, norm_all=over_all)
    x = src.double()

    def heads(off, count, w):
        rows = x[:, off:off + count * d]
        if over_all:
            rows = (plain.rms(rows, 1e-3) * w.double()).reshape(n, count, d)
        else:
            rows = plain.rms(rows.reshape(n, count, d), 1e-3) * w.double()
        return plain.turn(rows, positions, dims, freq, magnitude, interleaved)

    tol = dict(rtol=2e-5, atol=3e-4) if dtype == torch.float32 else dict(rtol=1e-2, atol=4e-2)
    torch.testing.assert_close(q.double().cpu().reshape(n, nq, d), heads(q_off, nq, qn), **tol)
    got_k = torch.stack([k_pool[pg, :, at] for pg, at in map(place, positions.tolist())]).double().cpu()
    got_v = torch.stack([v_pool[pg, :, at] for pg, at in map(place, positions.tolist())]).double().cpu()
    torch.testing.assert_close(got_k, heads(k_off, nk, kn), **tol)
    torch.testing.assert_close(got_v, x[:, v_off:v_off + nk * e].reshape(n, nk, e), rtol=0, atol=0)
    # values that are the raw keys: the same columns, neither normed nor turned
    v_pool2 = torch.zeros((table.shape[1] + 3, nk, page, d), dtype=dtype, device=DEV)
    qkv_prepare(src.to(DEV), (q_off, k_off, k_off), nq, nk, d, d, i32(positions.tolist()), i32([0] * n), out_dtype=dtype,
                q_norm=qn.to(DEV), k_norm=kn.to(DEV), norm_eps=1e-3, k_pool=k_pool, v_pool=v_pool2, block_table=table,
                norm_all=over_all)
    raw = torch.stack([v_pool2[pg, :, at] for pg, at in map(place, positions.tolist())]).cpu()
    assert torch.equal(raw, src[:, k_off:k_off + nk * d].reshape(n, nk, d))


def test_yarn_frequencies_in_the_rotary_part():
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import make_part
    for dims, base, sc in ((16, 100.0, (4.0, 64, 6.0, 1.0)), (40, 4e5, (2.0, 1024, 24.0, 1.0)), (10, 20.0, (3.0, 16, 2.0, 0.25))):
        keys = ("factor", "original", "fast", "slow")
        part = make_part("position", PartSpec("rotary", {"head_dim": dims, "theta": base, "exact_powers": True,
                                                         "scaling": {"kind": "yarn", **dict(zip(keys, sc))}}))
        freq, magnitude = plain.yarn(dims, base, *sc)
        assert part.magnitude == pytest.approx(magnitude, rel=1e-12)
        assert part.frequencies(dims, DEV).tolist() == pytest.approx(freq, rel=1e-6)


@pytest.mark.parametrize("dtype, P, page, block_page, d, e", [
    (torch.float32, 3, 4, 2, 10, 6), (torch.bfloat16, 8, 16, 16, 64, 32), (torch.float32, 1, 8, 8, 8, 12),
    (torch.float32, 20, 8, 4, 150, 200), (torch.bfloat16, 16, 16, 16, 128, 128)])
def test_block_means_are_stored_when_their_last_token_arrives(dtype, P, page, block_page, d, e):
    """The same tokens in one portion, in uneven portions and one by one: the same means to the bit, of the keys and
    values as the pages hold them; unfinished blocks are not touched."""
    from yalis_b200.ops.elementwise import qkv_prepare
    g = torch.Generator().manual_seed(P)
    nk, n = 2, 4 * P + 2
    src = torch.randn(n, nk * (2 * d + e), generator=g).to(dtype)
    table, place = shuffled_table(n, page, seed=3)
    btable, bplace = shuffled_table(n // P + 1, block_page, seed=4)
    results = []
    for cut in ([n], [P - 1, 2, P + 1] if P > 1 else [1, 2], [1] * n):
        cut = [c for c in cut if c > 0]
        cut = cut + ([n - sum(cut)] if sum(cut) < n else [])
        pools = [torch.full((t.shape[1] + 3, nk, pg, s), 9.0, dtype=dtype, device=DEV)
                 for t, pg, s in ((table, page, d), (table, page, e), (btable, block_page, d), (btable, block_page, e))]
        at = 0
        for c in cut:
            qkv_prepare(src[at:at + c].to(DEV), (0, nk * d, 2 * nk * d), nk, nk, d, e, i32(range(at, at + c)), i32([0] * c),
                        out_dtype=dtype, k_pool=pools[0], v_pool=pools[1], block_table=table, pool=P, pooled_k=pools[2],
                        pooled_v=pools[3], pooled_table=btable, single_tokens=c == 1)
            at += c
        results.append([p.cpu() for p in pools])
    for other in results[1:]:
        assert all(torch.equal(a, b) for a, b in zip(results[0], other))
    k_pool, v_pool, pk, pv = (p.double() for p in results[0])
    for pool, means in ((k_pool, pk), (v_pool, pv)):
        rows = torch.stack([pool[pg, :, at] for pg, at in map(place, range(n))])
        for b in range(n // P):
            pg, at = bplace(b)
            want = rows[b * P:(b + 1) * P].mean(dim=0)
            tol = 1e-6 if dtype == torch.float32 else 8e-3
            torch.testing.assert_close(means[pg, :, at], want, rtol=tol, atol=tol)
            means[pg, :, at] = 9.0
        assert bool((means == 9.0).all())


# ---- attention: windows, pooled blocks, distance bias, sink, gates --------------------------------------------------

def attend_rows(q, keys, values, scale, W, **kw):
    return plain.attend(q.double(), keys.double(), values.double(), scale, W, **kw)


CASES = [  # dtype, key size, value size, page, window, block size (None: none), buckets (None: none), heads, kv_heads
    (torch.float32, 12, 20, 16, 9, 4, None, 4, 2), (torch.float32, 8, 8, 8, 30, 30, None, 2, 2), (torch.float32, 10, 10, 4, 1, 1, None, 3, 1),
    (torch.float32, 12, 12, 16, 23, None, 8, 4, 2), (torch.float32, 7, 7, 8, 300, None, 6, 3, 1),
    (torch.bfloat16, 64, 40, 16, 44, 6, None, 4, 2), (torch.bfloat16, 48, 48, 16, 17, 5, None, 6, 3), (torch.bfloat16, 128, 96, 8, 100, 3, None, 2, 1),
    (torch.bfloat16, 64, 64, 64, 64, 64, None, 4, 2), (torch.bfloat16, 40, 24, 16, 37, None, None, 8, 1), (torch.bfloat16, 24, 24, 16, 50, None, 10, 20, 1),
    (torch.bfloat16, 128, 128, 16, 70, None, 32, 4, 2), (torch.bfloat16, 16, 200, 16, 33, 2, None, 2, 2), (torch.bfloat16, 256, 8, 16, 20, 7, None, 2, 1)]


@pytest.mark.parametrize("dtype, hs, vd, page, W, P, buckets, heads, kv_heads", CASES)
def test_attention_sees_exactly_its_window_and_the_blocks_before_it(dtype, hs, vd, page, W, P, buckets, heads, kv_heads):
    """One key is made to stand out.  Inside the window it carries the answer; just outside it does not; once its whole
    block lies before the window its mean does.  All queries in one portion, and each of interest alone as a decoded
    token; the tensor-core kernel, with and without key splits, where the sizes allow it."""
    from yalis_b200.ops.attention import PooledBlocks, mma_extended_supports, paged_attention_generic, paged_attention_mma
    g = torch.Generator().manual_seed(hs + vd + W)
    n, star = 260, 101
    table, place = shuffled_table(n, page, seed=5)
    keys, values = torch.randn(n, kv_heads, hs, generator=g), torch.randn(n, kv_heads, vd, generator=g)
    direction = torch.randn(hs, generator=g)
    direction /= direction.norm()
    keys -= 2 * direction                              # every other key points away from what the queries look for
    keys[star] = direction * 40
    values[star] = 5.0
    q = torch.randn(n, heads, hs, generator=g) * 0.3 + 4 * direction
    q, keys, values = q.to(dtype), keys.to(dtype), values.to(dtype)
    scale = 0.11
    sink = torch.randn(heads, generator=g)
    rel = torch.randn(buckets, heads, generator=g) * 2 if buckets else None
    far = 160 if buckets == 10 else 60
    gate = torch.randn(n, heads * vd if P else heads, generator=g).to(dtype)
    k_pool, v_pool = filled_pool(keys, table, place, page), filled_pool(values, table, place, page)
    pool = None
    if P:
        blocks = n // P
        bpage = 4
        btable, bplace = shuffled_table(blocks, bpage, seed=6)
        means = [x[:blocks * P].float().reshape(blocks, P, kv_heads, -1).mean(1).to(dtype) for x in (keys, values)]
        pool = PooledBlocks(P, *(filled_pool(m, btable, bplace, bpage) for m in means), btable)
    kw = dict(scale=scale, window=W, sink=True, sink_logits=sink.to(DEV), pool=pool)
    if buckets:
        length = min(W, far + 1)
        kw["rel"] = torch.stack([rel[plain.distance_bucket(m, buckets, far)] for m in range(length)]).T.contiguous().to(DEV)
    free = attend_rows(q, keys, values, scale, W, pool=P, sink=sink.double(), rel=None if rel is None else rel.double(), bias_max=far)
    want = free * torch.sigmoid(gate.double()).reshape(n, heads, -1)
    # the oracle itself must show the edges
    last_in = star + W - 1
    block_end = star // P * P + P - 1 if P else n
    seen_again = block_end + W                          # the first position that sees the starred block
    strong = lambda t: float(free[t, :, 0].mean()) > 2.5
    assert strong(star) and strong(min(last_in, n - 1)) and not strong(star - 1)
    if last_in + 1 < min(seen_again, n):
        assert not strong(last_in + 1)
    positions, reqs = i32(range(n)), i32([0] * n)
    qd, gd = q.reshape(n, heads * hs).to(DEV), gate.to(DEV)
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    got = paged_attention_generic(qd, k_pool, v_pool, positions, reqs, table, heads, kv_heads, hs, v_head_dim=vd, gate=gd, **kw)
    torch.testing.assert_close(got.double().cpu().reshape(n, heads, vd), want, **tol)
    places = sorted({t for t in (0, star - 1, star, last_in, last_in + 1, seen_again - 1, seen_again, n - 1) if 0 <= t < n})
    fast = dtype == torch.bfloat16
    if fast:
        assert mma_extended_supports(hs, vd)
        got = paged_attention_mma(qd, k_pool, v_pool, positions, i32([0, n]), reqs, table, n, heads, kv_heads, hs, v_head_dim=vd,
                                  gate=gd, exact_weights=True, **kw)
        torch.testing.assert_close(got.double().cpu().reshape(n, heads, vd), want, **tol)
    for t in places:
        args = (qd[t:t + 1].contiguous(), k_pool, v_pool, i32([t]))
        one = paged_attention_generic(*args, i32([0]), table, heads, kv_heads, hs, v_head_dim=vd, gate=gd[t:t + 1], **kw)
        torch.testing.assert_close(one.double().cpu().reshape(heads, vd), want[t], **tol)
        for splits in ((1, 3) if heads // kv_heads <= 16 else (1,)) if fast else ():
            one = paged_attention_mma(*args, i32([0, 1]), i32([0]), table, 1, heads, kv_heads, hs, v_head_dim=vd, exact_weights=True,
                                      n_splits=splits, gate=gd[t:t + 1].contiguous(), **kw)
            torch.testing.assert_close(one.double().cpu().reshape(heads, vd), want[t], **tol)


def test_a_far_block_among_hundreds_is_found():
    """Block 2 of 340 stands out for the last query of a long sequence, in the exact kernel and in the tensor-core one
    with its tiles divided among blocks."""
    from yalis_b200.ops.attention import PooledBlocks, paged_attention_generic, paged_attention_mma
    g = torch.Generator().manual_seed(1)
    P, W, hs, vd, n = 4, 20, 64, 64, 1400
    b_table, b_place = shuffled_table(n // P, 16, seed=7)
    table, place = shuffled_table(n, 16, seed=8)
    keys, values = (torch.randn(n, 1, s, generator=g).to(torch.bfloat16) for s in (hs, vd))
    bk, bv = (torch.randn(n // P, 1, s, generator=g) * 0.5 for s in (hs, vd))
    q = torch.randn(1, 2 * hs, generator=g).to(torch.bfloat16)
    bk[2, 0] = q[0, :hs].float() * 4
    bk, bv = bk.to(torch.bfloat16), bv.to(torch.bfloat16)
    pool = PooledBlocks(P, filled_pool(bk, b_table, b_place, 16), filled_pool(bv, b_table, b_place, 16), b_table)
    k_pool, v_pool = filled_pool(keys, table, place, 16), filled_pool(values, table, place, 16)
    kw = dict(scale=0.3, window=W, pool=pool)
    exact = paged_attention_generic(q.to(DEV), k_pool, v_pool, i32([n - 1]), i32([0]), table, 2, 1, hs, **kw)
    for splits in (1, 4, 7):
        fast = paged_attention_mma(q.to(DEV), k_pool, v_pool, i32([n - 1]), i32([0, 1]), i32([0]), table, 1, 2, 1, hs, n_splits=splits,
                                   exact_weights=True, **kw)
        torch.testing.assert_close(exact.float(), fast.float(), rtol=2e-2, atol=2e-2)
    assert float((exact[0, :vd].float().cpu() - bv[2, 0].float()).abs().max()) < 0.05


@pytest.mark.parametrize("hs, vd, P, heads, kv_heads", [(64, 32, 6, 4, 2), (48, 48, None, 6, 1)])
def test_unequal_requests_in_one_launch_each_as_alone(hs, vd, P, heads, kv_heads):
    """Three requests of unequal lengths in one launch (a long portion, a single token, a short portion in the middle of
    a block), pages interleaved: every row equals the request run alone, to the bit."""
    from ctx_helper import make_context
    from yalis_b200.ops.attention import PooledBlocks, paged_attention_generic, paged_attention_mma
    page, W = 16, 29
    q_lens, before = [90, 1, 13], [7, 203, 70]
    ctx, num_pages = make_context(q_lens, before, page, seed=4)
    g = torch.Generator().manual_seed(8)
    r = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).to(DEV)
    k_pool, v_pool = r(num_pages, kv_heads, page, hs), r(num_pages, kv_heads, page, vd)
    q = r(sum(q_lens), heads * hs)
    table = ctx.block_tables["kv_all"]
    pool = None
    if P:
        width = 12
        btable = torch.randperm(3 * width, generator=g).to(torch.int32).reshape(3, width).to(DEV)
        pool = PooledBlocks(P, r(3 * width, kv_heads, 4, hs), r(3 * width, kv_heads, 4, vd), btable)
    rel = torch.randn(heads, W, generator=g).to(DEV) if not P else None
    kw = dict(scale=0.2, window=W, sink=True, sink_logits=torch.randn(heads, generator=g).to(DEV), rel=rel, v_head_dim=vd)
    exact = paged_attention_generic(q, k_pool, v_pool, ctx.positions, ctx.req_of_token, table, heads, kv_heads, hs, pool=pool, **kw)
    fast = paged_attention_mma(q, k_pool, v_pool, ctx.positions, ctx.q_start, ctx.req_of_token, table, max(q_lens), heads, kv_heads, hs,
                               exact_weights=True, pool=pool, **kw)
    torch.testing.assert_close(exact.float(), fast.float(), rtol=2e-2, atol=2e-2)
    at = 0
    for i, (ql, b) in enumerate(zip(q_lens, before)):
        own = None if pool is None else PooledBlocks(P, pool.k, pool.v, pool.table[i:i + 1].contiguous())
        alone = paged_attention_mma(q[at:at + ql].contiguous(), k_pool, v_pool, i32(range(b, b + ql)), i32([0, ql]), i32([0] * ql),
                                    table[i:i + 1].contiguous(), max(ql, 17), heads, kv_heads, hs, exact_weights=True, pool=own, **kw)
        assert torch.equal(alone, fast[at:at + ql]), i
        alone = paged_attention_generic(q[at:at + ql].contiguous(), k_pool, v_pool, i32(range(b, b + ql)), i32([0] * ql),
                                        table[i:i + 1].contiguous(), heads, kv_heads, hs, pool=own, **kw)
        assert torch.equal(alone, exact[at:at + ql]), i
        at += ql


# ---- the selective state space --------------------------------------------------------------------------------------

STATE_SIZES = [  # heads, vdim, state, groups, parts, taps
    (4, 12, 10, 2, 3, 3), (5, 3, 9, 1, 1, 1), (2, 16, 128, 2, 2, 4), (6, 16, 20, 6, 6, 6), (8, 8, 260, 1, 4, 2)]


def state_case(dtype, sizes, hidden=40, seed=0):
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import make_part
    H, e, N, G, parts, K = sizes
    part = make_part("mixer", PartSpec("state_space", {"hidden_size": hidden, "heads": H, "vdim": e, "state": N, "groups": G,
                                                       "norm_groups": parts, "conv": K, "eps": 1e-5}))
    g = torch.Generator().manual_seed(seed + H)
    r = lambda *s, std=1.0, mean=0.0: (mean + std * torch.randn(*s, generator=g)).to(torch.bfloat16).float()
    channels = H * e + 2 * G * N
    t = {"in": r(H * e + channels + H, hidden, std=1.5 / hidden ** 0.5), "conv": r(channels, K, std=0.6), "conv.b": r(channels, std=0.4),
         "dt_bias": r(H, mean=-2.0), "A_log": r(H), "D": r(H, mean=1.0, std=0.5), "norm": r(H * e, mean=1.0, std=0.3),
         "o": r(hidden, H * e, std=1.3 / (H * e) ** 0.5)}
    names = {"in": "in_proj", "conv.b": "conv_bias", "o": "o_proj"}
    local = {names.get(k, k): v for k, v in t.items()}
    specs = part.param_specs()
    assert {k: tuple(v.shape) for k, v in local.items()} == {k: tuple(s.shape) for k, s in specs.items()}
    part.load({k: (v if specs[k].keep_float32 else v.to(dtype)).to(DEV) for k, v in local.items()})
    m = {"heads": H, "vdim": e, "state": N, "groups": G, "norm_groups": parts, "conv": K}
    return part, {k: v.double() for k, v in t.items()}, m, g


class StepArrays:
    """What a mixer reads of a step: requests ``[(slot, length)]`` one after the other."""

    def __init__(self, requests):
        starts = [0]
        for _, c in requests:
            starts.append(starts[-1] + c)
        self.q_start, self.slots = i32(starts), i32([s for s, _ in requests])
        self.req_of_token = i32([i for i, (_, c) in enumerate(requests) for _ in range(c)])
        self.host = type("Host", (), {"max_q_len": max(c for _, c in requests)})


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", STATE_SIZES)
def test_the_state_space_in_portions_beside_others(dtype, sizes):
    """Three requests of unequal lengths, cut into portions of 1 to 17 tokens with requests left out of steps: every
    position as the plain recurrence has it, and to the bit as when each request runs alone and whole."""
    from yalis_b200.parts.base import SlotStateCache
    part, t, m, g = state_case(dtype, sizes)
    lengths = {2: 61, 0: 33, 4: 7}
    xs = {s: torch.randn(n, 40, generator=g).to(dtype) for s, n in lengths.items()}
    zs = {s: (x.double() @ part.in_weight().double().cpu().T).to(dtype) for s, x in xs.items()}
    new_state = lambda: SlotStateCache(torch.zeros(6, part.layout.total, device=DEV))
    state = new_state()
    got, done = {s: [] for s in lengths}, {s: 0 for s in lengths}
    rng = random.Random(1)
    while any(done[s] < n for s, n in lengths.items()):
        live = [s for s, n in lengths.items() if done[s] < n]
        take = [(s, min(lengths[s] - done[s], rng.choice([1, 1, 2, 5, 17]))) for s in live if len(live) == 1 or rng.random() < 0.8]
        if not take:
            continue
        z = torch.cat([zs[s][done[s]:done[s] + c] for s, c in take]).to(DEV)
        y = torch.empty(z.shape[0], part.hidden_width, dtype=dtype, device=DEV)
        part.mix(z, StepArrays(take), state, y)
        at = 0
        for s, c in take:
            got[s].append(y[at:at + c].cpu())
            done[s] += c
            at += c
    for s, n in lengths.items():
        alone_state = new_state()
        y = torch.empty(n, part.hidden_width, dtype=dtype, device=DEV)
        part.mix(zs[s].to(DEV), StepArrays([(3, n)]), alone_state, y)
        assert torch.equal(torch.cat(got[s]), y.cpu()) and torch.equal(alone_state.state[3], state.state[s]), s
        want = plain.state_space(xs[s].double(), t, "", m, 1e-5)
        out = torch.cat(got[s]).double() @ t["o"].T
        scale = float(want.abs().max())
        assert float((out - want).abs().max()) / scale < (2e-5 if dtype == torch.float32 else 2.5e-2), s
    assert bool((state.state[[1, 3, 5]] == 0).all())                      # nobody else's slot was touched


def test_a_token_far_back_is_still_in_the_state():
    """A slowly decaying state (A near 0) keeps what one large token wrote 400 tokens ago; with a quick decay it is gone."""
    from yalis_b200.parts.base import SlotStateCache
    sizes, n = (2, 8, 16, 1, 1, 2), 420
    outs = {}
    for a_log in (-9.0, 2.0):
        part, t, m, g = state_case(torch.float32, sizes, seed=3)
        part.a_log.fill_(a_log)
        t["A_log"] = torch.full((2,), a_log, dtype=torch.float64)
        x = torch.randn(n, 40, generator=g)
        for big in (False, True):
            rows = x.clone()
            if big:
                rows[5] *= 20
            y = torch.empty(n, part.hidden_width, device=DEV)
            part.mix(torch.nn.functional.linear(rows.to(DEV), part.in_weight()), StepArrays([(0, n)]),
                     SlotStateCache(torch.zeros(2, part.layout.total, device=DEV)), y)
            want = plain.state_space(rows.double(), t, "", m, 1e-5)
            out = y.double().cpu() @ t["o"].T
            assert float((out - want).abs().max() / want.abs().max()) < 1e-4
            outs[a_log, big] = want[-1]
    gap = lambda a: float((outs[a, True] - outs[a, False]).abs().max())
    assert gap(-9.0) > 0.05 and gap(2.0) < 1e-6


@pytest.mark.parametrize("dtype, parts, width", [(torch.float32, 1, 50), (torch.float32, 7, 3), (torch.bfloat16, 4, 512), (torch.float32, 1, 14000)])
def test_gate_before_the_norm_of_equal_parts(dtype, parts, width):
    from yalis_b200.ops.recurrent import gate_norm
    g = torch.Generator().manual_seed(width)
    n, c = 5, parts * width
    o, z, w = torch.randn(n, c, generator=g), torch.randn(n, c + 8, generator=g).to(dtype), 1 + 0.3 * torch.randn(c, generator=g)
    o[:, :width] *= 30                                 # a part far larger than the others: norms over parts, not over all
    out = torch.full((n, c + 2), 3.0, dtype=dtype, device=DEV)
    gate_norm(o.to(DEV), z.to(DEV)[:, 8:], parts, w.to(DEV), 1e-4, i32([0, 0, -1, 1, 1]), out[:, 1:1 + c])
    zd = z[:, 8:].double()
    want = plain.rms((o.double() * zd * torch.sigmoid(zd)).reshape(n, parts, width), 1e-4).reshape(n, c) * w.double()
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    rows = [0, 1, 3, 4]
    torch.testing.assert_close(out[:, 1:1 + c].double().cpu()[rows], want[rows], rtol=tol, atol=tol)
    assert bool((out[2] == 3).all()) and bool((out[:, 0] == 3).all()) and bool((out[:, -1] == 3).all())     # padding stays


# ---- what stands between a sub-layer and the stream -----------------------------------------------------------------

@pytest.mark.parametrize("width, parts, parts2, dtype, n", [
    (48, 1, 1, torch.float32, 9), (200, 3, 2, torch.float32, 9), (1024, 1, 4, torch.bfloat16, 9), (37, 2, 1, torch.float32, 9),
    (2048, 1, 1, torch.bfloat16, 300), (2048, 4, 1, torch.bfloat16, 5), (4100, 1, 1, torch.bfloat16, 260), (6001, 1, 2, torch.float32, 3),
    (9000, 1, 1, torch.float32, 300)])
def test_two_normed_results_a_factor_and_a_scale_join_the_stream(width, parts, parts2, dtype, n):
    from yalis_b200.ops.elementwise import add_normed_rmsnorm
    g = torch.Generator().manual_seed(width)
    x = torch.randn(n, width, generator=g)

    def result(p, size):
        return torch.randn(p, n, width, generator=g) * size if p > 1 else (torch.randn(n, width, generator=g) * size).to(dtype)

    first, second = result(parts, 3.0), result(parts2, 0.2)
    bias, w1, w2, scale, w = (torch.randn(width, generator=g) * 0.3 + m for m in (0.0, 1.0, 1.0, 1.0, 1.0))
    total = lambda d, p: d.double().sum(0) if p > 1 else d.double()
    d1 = plain.rms(total(first, parts) + bias.double(), 1e-4) * w1.double()
    d2 = plain.rms(total(second, parts2), 1e-3) * w2.double()
    dev = lambda t: t.to(DEV)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    cases = [(dict(delta_norm=(dev(w1), 1e-4), second=(dev(second), (dev(w2), 1e-3)), factor=0.5, scale=dev(scale)), 0.5 * (d1 + d2) * scale.double()),
             (dict(delta_norm=(dev(w1), 1e-4), second=(dev(second), (dev(w2), 1e-3))), d1 + d2),
             (dict(scale=dev(scale)), (total(first, parts) + bias.double()) * scale.double()),
             (dict(factor=0.25), (total(first, parts) + bias.double()) * 0.25)]
    for kw, added in cases:
        want_x = x.double() + added
        want_y = plain.rms(want_x, 1e-5) * w.double()
        xs = dev(x.clone())
        y = add_normed_rmsnorm(xs, dev(first), bias=dev(bias), weight=dev(w), eps=1e-5, out_dtype=dtype, **kw)
        torch.testing.assert_close(xs.double().cpu(), want_x, rtol=2e-5, atol=2e-5)
        torch.testing.assert_close(y.double().cpu(), want_y, rtol=tol, atol=tol)
        xs2 = dev(x.clone())
        rows = add_normed_rmsnorm(xs2, dev(first), bias=dev(bias), weight=dev(w), eps=1e-5, out_dtype=dtype, rows=i32([n - 1, 0]), **kw)
        assert torch.equal(xs2.cpu(), x)
        torch.testing.assert_close(rows.float(), y[[n - 1, 0]].float(), rtol=tol, atol=tol)
        xs3 = dev(x.clone())
        assert add_normed_rmsnorm(xs3, dev(first), bias=dev(bias), **kw) is None
        torch.testing.assert_close(xs3.double().cpu(), want_x, rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("dtype, at", [(torch.float32, 3), (torch.bfloat16, 3), (torch.bfloat16, 8)])
def test_the_dense_feed_forwards_inner_bias(dtype, at):
    from yalis_b200.ops.elementwise import activation
    g = torch.Generator().manual_seed(at)
    z, b = (torch.randn(11, at + 40, generator=g) * 2).to(dtype), torch.randn(40, generator=g)
    got = activation(z.to(DEV)[:, at:], "gelu_tanh", bias=b.to(DEV))
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    torch.testing.assert_close(got.double().cpu(), plain.gelu_tanh(z[:, at:].double() + b.double()), rtol=tol, atol=tol)


# ---- whole models ------------------------------------------------------------------------------------------------------

TOL = {"float32": 2e-4, "bfloat16": 6e-2}
LENGTHS = {"A": [1, 5, 33, 70, 21, 48], "B": [2, 40, 9, 64, 17, 90], "C": [3, 37, 18, 150, 12, 66], "D": [7, 1, 50, 19, 33, 4]}
PAGE = {"A": 16, "B": 8, "C": 64, "D": 16}
_oracle = {}


def requests_for(which):
    cfg, _ = plain.read_folder(ludelorn_dir(which))
    g = torch.Generator().manual_seed(ord(which))
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[which])}


def oracle(which):
    if which not in _oracle:
        cfg, w = plain.read_folder(ludelorn_dir(which))
        _oracle[which] = {rid: plain.forward(cfg, w, t).numpy() for rid, t in requests_for(which).items()}
    return _oracle[which]


def replay(folder, dtype, steps, max_tokens, page, graphs=False):
    from yalis_b200.engine.replay import Replayer
    rep = Replayer(folder, dtype, max_tokens, page_size=page, graphs=graphs)
    out = {}
    for s in steps:
        r = rep.run_step(s)
        if r is not None:
            out[s["step"]] = r
    rep.engine.manager.check()
    for grp in rep.engine.groups:
        assert rep.engine.manager.free_pages(grp.name) == grp.num_pages          # every page came back
    return out, rep


def compare(got, want, tol, what):
    assert set(got) == set(want), what
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        err = np.abs(got[rid] - want[rid]).max(axis=1) / np.abs(want[rid]).max()
        assert err.max() <= tol, (f"{what}: request {rid} differs by {err.max():.3e} (tolerance {tol}); first wrong position "
                                  f"{int(np.argmax(err > tol))} of {len(err)}")


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_requests_cut_four_ways_agree_with_the_plain_model(which, dtype):
    reqs, want = requests_for(which), oracle(which)
    vocab = plain.read_folder(ludelorn_dir(which))[0]["vocab"]
    results = {}
    for name, steps in (("whole", traces.whole(reqs)), ("tail", traces.tail_decoded(reqs, tail=12)),
                        ("portions", traces.portions(reqs, seed=3)), ("mixed", traces.mixed(reqs, seed=5, tail=6))):
        steps = traces.number(steps)
        out, _ = replay(ludelorn_dir(which), dtype, steps, traces.peak_tokens(steps, max(64, PAGE[which])), PAGE[which])
        results[name] = traces.collect(steps, out, vocab)
        compare(results[name], want, TOL[dtype], f"{which} {dtype} {name}")
    # how a request was cut, what ran beside it and which pages and slots it had leave (nearly) no trace
    for name in ("tail", "portions", "mixed"):
        compare(results[name], results["whole"], 2e-5 if dtype == "float32" else 5e-2, f"{which} {dtype} {name} against whole")


@pytest.mark.parametrize("which", ["A", "C"])
def test_steps_replayed_from_recordings_give_the_same(which):
    reqs, want = requests_for(which), oracle(which)
    vocab = plain.read_folder(ludelorn_dir(which))[0]["vocab"]
    steps = traces.number(traces.tail_decoded(reqs, tail=12))
    pages = traces.peak_tokens(steps, max(64, PAGE[which]))
    launched, _ = replay(ludelorn_dir(which), "float32", steps, pages, PAGE[which])
    recorded, rep = replay(ludelorn_dir(which), "float32", steps, pages, PAGE[which], graphs=True)
    assert rep.steps_replayed > 40
    a, b = traces.collect(steps, launched, vocab), traces.collect(steps, recorded, vocab)
    compare(b, want, TOL["float32"], f"{which} recorded")
    compare(b, a, 1e-6, f"{which} recorded against launched")


@pytest.mark.parametrize("which", ["A", "B", "C"])
def test_the_residual_stream_after_every_layer(which):
    from yalis_b200.engine.engine import Engine, StepEntry
    d = ludelorn_dir(which)
    cfg, w = plain.read_folder(d)
    tokens = requests_for(which)["r3"]
    want = []
    plain.forward(cfg, w, tokens, taps=want)
    eng = Engine(d, dtype="float32", page_size=16, num_pages=12, max_slots=2, max_context=192)
    eng.add_request("x")
    seen = []
    inner = eng.model.forward
    eng.model.forward = lambda ctx, caches: inner(ctx, caches, tap=lambda i, x: seen.append(x.double().cpu()))
    eng.run([StepEntry("x", tokens, [len(tokens) - 1])])
    assert len(seen) == len(want) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, want)):
        assert float((a - b).abs().max() / b.abs().max()) < 2e-5, f"layer {i}"


@pytest.mark.parametrize("which, dtype", [("A", "float32"), ("B", "float32"), ("C", "bfloat16")])
def test_long_decoding_keeps_to_the_plain_model(which, dtype):
    """300 tokens one by one after a two-token prompt: every window and block border passes over decoded tokens many
    times, the state is carried through all of them, and the pages behind the windows are given back and used again
    (their pools are far smaller than the sequence)."""
    from yalis_b200.engine.engine import Engine, StepEntry
    d = ludelorn_dir(which)
    cfg, w = plain.read_folder(d)
    tokens = torch.randint(0, cfg["vocab"], (302,), generator=torch.Generator().manual_seed(9)).tolist()
    want = plain.forward(cfg, w, tokens).numpy()
    eng = Engine(d, dtype=dtype, page_size=8, num_pages=48, max_slots=1, max_context=384, max_tokens_per_step=2)
    windows = [grp for grp in eng.groups if grp.window is not None]
    assert windows and all(grp.num_pages * grp.page_size < 150 for grp in windows)
    eng.add_request("x")
    rows = [eng.run([StepEntry("x", tokens[:2], [0, 1])]).logits.cpu().numpy()]
    for t in tokens[2:]:
        rows.append(eng.run([StepEntry("x", [t], [0])]).logits.cpu().numpy())
    eng.check_device_errors()
    err = np.abs(np.concatenate(rows) - want).max(axis=1) / np.abs(want).max()
    assert err.max() < TOL[dtype], int(np.argmax(err))


def test_a_slot_and_its_pages_used_again_start_clean():
    from yalis_b200.engine.engine import Engine, StepEntry
    reqs = requests_for("C")
    eng = Engine(ludelorn_dir("C"), dtype="float32", page_size=64, num_pages=3, max_slots=1, max_context=192)
    first = None
    for rid in ("r3", "r1", "r3"):
        assert eng.add_request(rid) == 0                       # the only slot, every time
        out = eng.run([StepEntry(rid, reqs[rid], [len(reqs[rid]) - 1])]).logits.cpu().numpy()
        eng.finish_request(rid)
        if rid == "r3":
            if first is None:
                first = out
            else:
                assert np.array_equal(first, out)              # what r1 left in slot, pages and blocks does not show


def test_a_pool_too_small_is_refused_before_anything_runs():
    """A request whose tokens would still fit the windows' pages but whose blocks' pages have run out is refused, and
    the engine goes on."""
    from yalis_b200.engine.engine import Engine, OutOfPages, StepEntry
    eng = Engine(ludelorn_dir("A"), dtype="float32", page_size=4, num_pages=12, max_slots=2, max_context=4000, max_tokens_per_step=4)
    eng.add_request("x")
    with pytest.raises(OutOfPages):
        for _ in range(500):
            eng.run([StepEntry("x", [1, 2, 3, 4], [])])
    # windows give their pages back; what ends it is the group of blocks of 3 tokens: (12 / 3 + 2) pages of 4 blocks
    assert eng.length("x") == 6 * 4 * 3
    eng.manager.check()
    eng.finish_request("x")
    eng.add_request("y")
    assert eng.run([StepEntry("y", [1, 2], [1])]).logits is not None


@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_entry_point(which):
    from yalis_b200 import InferenceConfig, LLMEngine, ModelConfig
    d = ludelorn_dir(which)
    cfg, w = plain.read_folder(d)
    g = torch.Generator().manual_seed(4)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (3, 19, 40, 7, 26)]
    engine = LLMEngine(ModelConfig(model_name=f"ludelorn-tiny-{which}", model_path=d, precision="fp32"),
                       InferenceConfig(max_batch_size=3, max_length_of_generated_sequences=64, temperature=0.0, top_p=0.0,
                                       page_size=PAGE[which]))
    tokens, metrics = engine.generate(prompts, tokens_to_generate=10)[:2]
    for p, row in zip(prompts, tokens.cpu().tolist()):
        assert row == plain.greedy(cfg, w, p, 10)


def test_the_replay_program_runs_a_ludelorn_folder(tmp_path):
    reqs = {k: v for k, v in requests_for("B").items() if k in ("r1", "r2")}
    steps = traces.number(traces.portions(reqs, seed=1))
    out_dir = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", ludelorn_dir("B"), "--dtype", "float32",
                           "--out", str(out_dir), "--max-tokens", str(traces.peak_tokens(steps))],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    vocab = plain.read_folder(ludelorn_dir("B"))[0]["vocab"]
    outputs = {s["step"]: np.fromfile(out_dir / f"{s['step']}.f32", dtype="<f4") for s in steps}
    compare(traces.collect(steps, outputs, vocab), {k: oracle("B")[k] for k in reqs}, TOL["float32"], "program")


# ---- configurations drawn at random: other orders of layers, sizes, masks and constants -------------------------------

def random_config(seed):
    """A Ludelorn configuration drawn from ``seed``: three to six layers of any type in any order, head sizes with and
    without a tensor-core kernel, windows from one position to longer than any request, blocks shorter and longer than
    their windows, bucket counts and limits, state sizes, groups, parts and taps."""
    rng = random.Random(seed)

    def heads(same=False):
        kv, dim = rng.choice([1, 2, 3]), rng.choice([6, 8, 12, 16, 24, 32, 40, 48, 64])
        return {"heads": kv * rng.choice([1, 2, 4]), "kv_heads": kv, "dim": dim, "vdim": dim if same else rng.choice([dim, 8, 20, 32, 56]),
                "scale": round(rng.uniform(0.5, 1.5) * dim ** -0.5, 4), "mask": {"size": rng.choice([1, 2, 5, 16, 17, 31, 64, 1000])}}

    def turned(m):
        m["rot"] = {"dims": rng.choice([v for v in (2, 4, 8, m["dim"]) if v <= m["dim"]]), "base": rng.choice([10.0, 777.0, 10000.0])}
        if rng.random() < 0.5:
            m["rot"]["scaling"] = {"factor": rng.choice([1.5, 4.0, 16.0]), "original": rng.choice([16, 100, 4096]),
                                   "fast": rng.choice([2.0, 32.0]), "slow": rng.choice([0.5, 1.0])}
        return m

    layers = []
    for _ in range(rng.randint(3, 6)):
        kind = rng.choice(["parallel", "attention", "attention_2"])
        if kind == "parallel":
            groups, vdim = rng.choice([1, 2, 3]), rng.choice([4, 5, 8, 16])
            n = groups * rng.choice([1, 2, 3])
            mixer = {"left": turned(heads()), "right": {"heads": n, "vdim": vdim, "groups": groups, "state": rng.choice([3, 8, 16, 40, 64]),
                                                        "norm_groups": rng.choice([1, n, vdim]), "conv": rng.choice([1, 2, 4, 7])}}
        elif kind == "attention":
            mixer = turned(heads())
            mixer["mask"]["pool"] = rng.choice([1, 2, 3, 8, 16, 30])
        else:
            mixer = heads(same=True)
            buckets = rng.choice([2, 4, 10, 16, 32])
            mixer.update(buckets=buckets, bias_max=rng.choice([v for v in (18, 33, 100, 1000) if v > buckets // 2]))
        mlp = None if rng.random() < 0.2 else {"kind": "dense", "ff": rng.choice([24, 57, 90])}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Ludelorn", "width": rng.choice([40, 63, 64, 100]), "vocab": rng.choice([33, 64, 150]),
            "norm": {"eps": rng.choice([1e-5, 1e-6, 1e-3])}, "embedding": {"scale": rng.choice([0.5, 1.0, 4.0])}, "layers": layers}


@pytest.mark.parametrize("seed", [21, 22, 23, 24, 25, 26, 27, 28, 29, 30])
def test_configurations_drawn_at_random(seed, tmp_path):
    d = write_model(random_config(seed), str(tmp_path / "m"), seed)
    cfg, w = plain.read_folder(d)
    g = torch.Generator().manual_seed(seed)
    reqs = {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate([1, 37, 80, 9, 52])}
    want = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for name, steps, dtype in (("whole", traces.whole(reqs), "float32"), ("mixed", traces.mixed(reqs, seed=seed, tail=5), "float32"),
                               ("portions", traces.portions(reqs, seed=seed), "float32"),
                               ("mixed", traces.mixed(reqs, seed=seed, tail=5), "bfloat16")):
        steps = traces.number(steps)
        out, _ = replay(d, dtype, steps, traces.peak_tokens(steps), 16)
        got = traces.collect(steps, out, cfg["vocab"])
        if dtype == "float32":
            compare(got, want, TOL[dtype], f"seed {seed} {name}")
        else:                       # the other kernels over the same steps; how far rounding carries depends on the draw
            errs = np.concatenate([np.abs(got[rid] - want[rid]).max(axis=1) / np.abs(want[rid]).max() for rid in want])
            assert np.isfinite(errs).all() and np.mean(errs > 8e-2) < 0.03, f"seed {seed}: {np.mean(errs > 8e-2):.3f} of the positions differ"
