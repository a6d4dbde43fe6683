"""Lagulorn on the GPU against the plain implementation: every mechanism's kernel alone, then whole models cut into
steps in every way, then generation through the entry point.

Kernel tests build their own index arrays, slots and pages (handed out shuffled, everything else NaN) and compare with the
functions of ``plain_lagulorn`` in float64.  Where random numbers would hide a fault (a window that is one position off,
maps that read each other's keys, a lost state, a group masked with zero) the inputs are made so that it shows.  Model
tests make small model folders of four configurations that differ in every size and option (one to four copies of the
stream or none, shared tensors, layers without feed-forward, every output chosen) and replay requests whole, with a
decoded tail, in portions down to two tokens, and mixed with few pages and slots.
"""

import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_lagulorn as plain
import traces
from lagulorn_models import lagulorn_dir, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def step_arrays(portions):
    """portions: list of (slot, start position, count) -> req_of_token, q_start, slots, positions."""
    req, pos, qs, slots = [], [], [0], []
    for r, (slot, start, count) in enumerate(portions):
        req += [r] * count
        pos += list(range(start, start + count))
        qs.append(qs[-1] + count)
        slots.append(slot)
    return i32(req), i32(qs), i32(slots), i32(pos)


def cuts(total, sizes):
    out, at, i = [], 0, 0
    while at < total:
        c = min(sizes[i % len(sizes)], total - at)
        out.append((at, c))
        at += c
        i += 1
    return out


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


# ---- the copies of the stream with a root-mean-square norm --------------------------------------------------------

@pytest.mark.parametrize("copies, width, y_kind", [(1, 36, "float32"), (2, 64, "bfloat16"), (3, 50, "parts"), (4, 128, "parts"), (4, 2048, "bfloat16"),
                                                   (8, 20, "float32"), (5, 4100, "parts"), (2, 5000, "bfloat16"), (3, 1030, "float32")])
def test_copies_are_written_read_and_normed_in_one_pass(copies, width, y_kind):
    from yalis_b200.ops.streams import stream_step
    g = torch.Generator().manual_seed(copies * 100 + width)
    n, eps = 11, 0.3                                                                     # an eps that shows
    x = torch.randn(n, copies, width, generator=g)
    mix = torch.eye(copies) * 0.7 + 0.3 * torch.randn(copies, copies, generator=g)       # not symmetric: [from, to] shows
    w_out, w_in = torch.randn(copies, generator=g), torch.randn(copies, generator=g)
    w = 0.3 * torch.randn(width, generator=g)
    if y_kind == "parts":
        y = torch.randn(3, n, width, generator=g)
        y_sum = y.double().sum(dim=0)
    else:
        y = torch.randn(n, width, generator=g).to(getattr(torch, y_kind))
        y_sum = y.double()
    want_x = plain.write_copies(x.double().transpose(0, 1), mix.double(), w_out.double(), y_sum)        # [S, N, D]
    want_h = plain.layer_norm(plain.read_copies(want_x, w_in.double()), w.double(), eps)
    write = dict(y=y.to(DEV), mix=mix.to(DEV), out_weights=w_out.to(DEV))
    rms = ((1 + w).to(DEV), eps)
    xd = x.clone().to(DEV)
    h = stream_step(xd, in_weights=w_in.to(DEV), rms=rms, out_dtype=torch.float32, **write)
    torch.testing.assert_close(xd.double().cpu().transpose(0, 1), want_x, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h.double().cpu(), want_h, rtol=1e-5, atol=1e-5)
    # chosen rows, the plain sum of the copies (the last step before the logits): the stream stays
    xd2 = x.clone().to(DEV)
    rows = [n - 1, 0, 7]
    some = stream_step(xd2, rms=rms, rows=i32(rows), out_dtype=torch.float32, **write)
    assert torch.equal(xd2.cpu(), x)
    torch.testing.assert_close(some.double().cpu(), plain.layer_norm(want_x.sum(dim=0), w.double(), eps)[rows], rtol=1e-5, atol=1e-5)
    # a row of no request is skipped
    with_gap = stream_step(xd2, rms=rms, rows=i32([3, -1]), out_dtype=torch.bfloat16)
    torch.testing.assert_close(with_gap[0].double().cpu(), plain.layer_norm(x[3].double().sum(dim=0), w.double(), eps), rtol=1e-2, atol=1e-2)
    # the stream's first pass: all copies are the entering rows, which the pass stores as copies
    src = torch.randn(n, width, generator=g)
    late = torch.full((n, copies, width), float("nan"), device=DEV)
    first = stream_step(late, source=src.to(DEV), in_weights=w_in.to(DEV), rms=rms, out_dtype=torch.float32)
    assert torch.equal(late.cpu(), src[:, None, :].repeat(1, copies, 1))
    want_first = plain.layer_norm(src.double() * w_in.double().sum(), w.double(), eps)
    torch.testing.assert_close(first.double().cpu(), want_first, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("copies", [None, 1, 3])
def test_a_constant_on_the_result(copies):
    """The residual constant multiplies the result on its way into the stream: through the write weights of a stream in
    copies, in the adding pass of a plain one."""
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import ResidualStream, make_part
    g = torch.Generator().manual_seed(5)
    n, width, factor = 9, 40, 0.3
    x, y = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g)
    norm = make_part("norm", PartSpec("rms_norm", {"size": width, "eps": 1e-5, "one_plus": True}))
    w = 0.2 * torch.randn(width, generator=g)
    norm.load({"weight": w.to(DEV)})
    if copies is None:
        part = make_part("connection", PartSpec("scaled_sum", {"hidden_size": width, "learned": False, "factor": factor}))
        part.load({})
        stream = ResidualStream(x.clone().to(DEV), torch.float32)
        want = x.double() + factor * y.double()
    else:
        part = make_part("connection", PartSpec("hyper_connection", {"hidden_size": width, "copies": copies, "mixing": True, "factor": factor}))
        t = {"in": torch.randn(copies, generator=g), "out": torch.randn(copies, generator=g), "mix": torch.randn(copies, copies, generator=g)}
        part.load({k: v.to(DEV) for k, v in t.items()})
        stream = ResidualStream(torch.full((n, copies, width), float("nan"), device=DEV), torch.float32, source=x.clone().to(DEV))
        norm.forward(stream, in_weights=part.read_weights())
        streams = plain.write_copies(x.double()[None].repeat(copies, 1, 1), t["mix"].double(), factor * t["out"].double(), y.double())
        want = streams.sum(dim=0)
    stream.add(part.write(None, y.to(DEV)))
    h = norm.forward(stream)
    torch.testing.assert_close(h.double().cpu(), plain.layer_norm(want, w.double(), 1e-5), rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(stream.total().double().cpu(), want, rtol=1e-5, atol=1e-5)


# ---- lightning attention -------------------------------------------------------------------------------------------

@pytest.mark.parametrize("kind", ["silu", "gelu_erf"])
@pytest.mark.parametrize("dtype, n, cols, pad", [(torch.bfloat16, 33, 64, 8), (torch.bfloat16, 700, 30, 5), (torch.float32, 5, 44, 4), (torch.float32, 3, 7, 0)])
def test_activations_with_float32_results(kind, dtype, n, cols, pad):
    from yalis_b200.ops.elementwise import activation
    x = (torch.randn(n, cols + pad, generator=torch.Generator().manual_seed(cols)) * 3).to(dtype)
    got = activation(x.to(DEV)[:, :cols], kind, out_dtype=torch.float32)
    assert got.dtype == torch.float32
    want = (plain.silu if kind == "silu" else plain.gelu_erf)(x[:, :cols].double())
    torch.testing.assert_close(got.double().cpu(), want, rtol=2e-6, atol=2e-6)


@pytest.mark.parametrize("dtype, heads, vdim", [(torch.float32, 3, 10), (torch.bfloat16, 16, 128), (torch.float32, 1, 7), (torch.bfloat16, 5, 3),
                                                (torch.float32, 40, 300)])
def test_all_heads_normed_together_before_the_gate(dtype, heads, vdim):
    """One head is a hundred times larger than the others: a norm per head would bring all to one size.  The gate comes
    behind the norm: gating first would change the root mean square."""
    from yalis_b200.ops.recurrent import GATE_SIGMOID, gate_norm
    g = torch.Generator().manual_seed(heads * vdim)
    n, width, eps = 13, heads * vdim, 1e-3
    o = torch.randn(n, heads, vdim, generator=g)
    o[:, 0] *= 100.0
    o = o.reshape(n, width)
    z = (torch.randn(n, width + 8, generator=g) * 2).to(dtype)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    out = torch.zeros(n, width, dtype=dtype, device=DEV)
    gate_norm(o.to(DEV), z.to(DEV)[:, 8:], 1, w.to(DEV), eps, i32([0] * n), out, gate_kind=GATE_SIGMOID, after=True)
    want = plain.unit_rms(o.double(), eps) * w.double() * plain.sigmoid(z[:, 8:].double())
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    torch.testing.assert_close(out.double().cpu(), want, rtol=tol, atol=tol)


def lightning_part(hidden, heads, dim, vdim, decay, dtype, seed, eps=1e-5):
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import SlotStateCache, make_part
    g = torch.Generator().manual_seed(seed)
    t = {n: (torch.randn(rows, hidden, generator=g) * (1.5 / hidden ** 0.5)).to(torch.bfloat16)
         for n, rows in (("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim))}
    t["o"] = (torch.randn(hidden, heads * vdim, generator=g) * (1.5 / (heads * vdim) ** 0.5)).to(torch.bfloat16)
    t["norm"] = 1 + 0.3 * torch.randn(heads * vdim, generator=g)
    part = make_part("mixer", PartSpec("retention", {"hidden_size": hidden, "heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rotary": None,
                                                     "eps": eps, "activation": "silu", "norm": "all", "gate": "sigmoid"}))
    local = {f"{n}_proj": t[n].to(dtype).to(DEV) for n in "qkvgo"}
    part.load({**local, "norm": t["norm"].float().to(DEV)})
    return part, {k: v.double() for k, v in t.items()}, lambda slots: SlotStateCache(torch.zeros(slots, part.layout.total, device=DEV))


class _Step:
    """The few facts of a step that a mixer with a state reads."""

    def __init__(self, portions):
        self.req_of_token, self.q_start, self.slots, self.positions = step_arrays(portions)
        self.host = type("Host", (), {"max_q_len": max(c for _, _, c in portions)})()


def result(part_output):
    return (part_output.sum(dim=0) if part_output.dim() == 3 else part_output).double().cpu()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden, heads, dim, vdim", [(64, 2, 16, 12), (40, 3, 10, 7), (96, 4, 64, 16), (72, 1, 20, 130), (64, 5, 7, 1), (128, 2, 300, 24)])
def test_the_lightning_mixer_in_portions_beside_others(dtype, hidden, heads, dim, vdim):
    decay = [0.4, 0.999, 1.0, 0.0, 0.9][:heads]
    part, t, cache_for = lightning_part(hidden, heads, dim, vdim, decay, dtype, seed=heads * 100 + dim)
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    g = torch.Generator().manual_seed(3)
    lengths = [41, 6, 70]
    x = [torch.randn(T, hidden, generator=g).to(torch.bfloat16) for T in lengths]
    want = [plain.lightning_mixer(v.double(), t, "", m, 1e-5) for v in x]

    def run(plan):
        cache = cache_for(5)
        cache.state[0].fill_(3.0)
        cache.state[4].fill_(-2.0)
        got = [torch.zeros(T, hidden, dtype=torch.float64) for T in lengths]
        for step in plan:
            rows = torch.cat([x[r][a:a + c] for r, a, c in step]).to(dtype).to(DEV)
            out = result(part.forward(rows, _Step([(r + 1, a, c) for r, a, c in step]), cache))
            o = 0
            for r, a, c in step:
                got[r][a:a + c] = out[o:o + c]
                o += c
        assert float(cache.state[0, 0]) == 3.0 and float(cache.state[4, -1]) == -2.0               # nobody else's slot
        return got

    whole = run([[(r, 0, T)] for r, T in enumerate(lengths)])
    pieces = {r: cuts(T, s) for (r, T), s in zip(enumerate(lengths), ([2, 1, 17, 3], [1, 2], [16, 1, 2, 30]))}
    plan = []
    for i in range(max(len(p) for p in pieces.values())):
        step = [(r, *pieces[r][i]) for r in pieces if i < len(pieces[r])]
        plan.append(step[::-1] if i % 2 else step)
    cut, single = run(plan), run([[(r, a, 1)] for r, T in enumerate(lengths) for a in range(T)])
    tol = 1e-4 if dtype == torch.float32 else 4e-2
    for r in range(3):
        for got, what in ((whole, "whole"), (cut, "portions"), (single, "one by one")):
            assert float((got[r] - want[r]).abs().max() / want[r].abs().max()) < tol, (r, what)


def test_a_token_far_back_is_still_in_the_slow_heads_state():
    """A pair written at the first token is read 600 tokens later, the later tokens one by one: in the head that keeps
    0.999 of its state a token it is more than half there, in the head that keeps 0.6 it is gone."""
    from yalis_b200.ops.recurrent import StateLayout, state_scan
    g = torch.Generator().manual_seed(8)
    heads, dim, vdim, T = 2, 24, 16, 601
    decay = [0.6, 0.999]
    lay = StateLayout(heads, dim, vdim)
    q, k, v = torch.randn(T, heads, dim, generator=g), 0.01 * torch.randn(T, heads, dim, generator=g), torch.randn(T, heads, vdim, generator=g)
    e = torch.zeros(dim)
    e[5] = 1.0
    k[0], q[T - 1] = 3.0 * e, e
    want, _ = plain.decaying_state(q.double(), k.double(), v.double(), decay)
    rows, got = torch.zeros(3, lay.total, device=DEV), []
    f = lambda t, a, c: t[a:a + c].reshape(c, -1).to(DEV)
    for a, c in cuts(T, [200] + [1] * 500):
        _, qs, slots, _ = step_arrays([(2, a, c)])
        got.append(state_scan(f(q, a, c), f(k, a, c), f(v, a, c), rows, lay, qs, slots, kv_heads=heads, decay=torch.tensor(decay, device=DEV),
                              max_q_len=c).double().cpu())
    got = torch.cat(got).reshape(T, heads, vdim)
    assert float((got - want).abs().max() / want.abs().max()) < 1e-4
    planted = 3.0 * v[0].double()
    assert float((got[-1, 1] - 0.999 ** 600 * planted[1]).abs().max()) < 0.25 * float(planted[1].abs().max())
    assert float(got[-1, 0].abs().max()) < 0.1 * float(planted[0].abs().max())


# ---- differential attention ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype, n, heads, kv_heads, d, e", [(torch.float32, 21, 3, 1, 10, 6), (torch.float32, 5, 4, 2, 16, 24), (torch.bfloat16, 21, 4, 2, 64, 128),
                                                             (torch.bfloat16, 400, 6, 3, 24, 40), (torch.float32, 400, 2, 2, 7, 9)])
def test_every_head_and_map_is_normed_by_itself_and_keys_lie_side_by_side(dtype, n, heads, kv_heads, d, e):
    from yalis_b200.ops.elementwise import qkv_prepare
    g = torch.Generator().manual_seed(d + n)
    page, start, eps = 8, 300, 1e-3
    table, place = shuffled_table(start + n, page, seed=2)
    qd, kd = heads * 2 * d, kv_heads * 2 * d
    src = torch.randn(n, qd + kd + kv_heads * e + 3, generator=g)
    src[:, d:2 * d] *= 50.0                                                       # the first head's second map is far larger than its first
    src = src.to(dtype)
    qn, kn = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    pages = table.shape[1] + 3
    k_pool = torch.zeros(pages, kv_heads, page, 2 * d, dtype=dtype, device=DEV)
    v_pool = torch.zeros(pages, kv_heads, page, e, dtype=dtype, device=DEV)
    q = qkv_prepare(src.to(DEV), (0, qd, qd + kd), heads * 2, kv_heads, d, e, i32(range(start, start + n)), i32([0] * n), out_dtype=dtype,
                    q_norm=qn.to(DEV), k_norm=kn.to(DEV), norm_eps=eps, k_pool=k_pool, v_pool=v_pool, block_table=table, maps=2)
    x = src.double()
    want_q = plain.unit_rms(x[:, :qd].reshape(n, heads, 2, d), eps) * qn.double()
    want_k = plain.unit_rms(x[:, qd:qd + kd].reshape(n, kv_heads, 2, d), eps) * kn.double()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    torch.testing.assert_close(q.double().cpu(), want_q.reshape(n, qd), rtol=tol, atol=tol)
    for t in range(n):
        pg, at = place(start + t)
        torch.testing.assert_close(k_pool[pg, :, at].double().cpu(), want_k[t].reshape(kv_heads, 2 * d), rtol=tol, atol=tol)
        assert torch.equal(v_pool[pg, :, at].cpu(), src[t, qd + kd:qd + kd + kv_heads * e].reshape(kv_heads, e))
    assert int((k_pool != 0).any(dim=-1).sum()) == n * kv_heads                    # nothing else was written


def plain_maps(q, k, v, scale, window, balance, diff, eps, at):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, e]: the heads' results at the positions ``at``."""
    maps = []
    for m in range(2):
        per = q.shape[1] // k.shape[1]
        out = torch.zeros(len(at), q.shape[1], v.shape[-1], dtype=torch.float64)
        for n, i in enumerate(at):
            lo = 0 if window is None else max(0, i - window + 1)
            for h in range(q.shape[1]):
                s = (k[lo:i + 1, h // per, m] @ q[i, h, m]) * scale
                w = torch.exp(s - s.max())
                out[n, h] = (w @ v[lo:i + 1, h // per]) / w.sum()
        maps.append(out)
    return plain.difference_of_maps(maps[0], maps[1], balance, diff, eps)


def test_the_maps_helper_is_the_plain_mixers_attention():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(12, *s, generator=g).double() for s in ((4, 2, 6), (2, 2, 6), (2, 5)))
    want = plain.difference_of_maps(*(plain.windowed_attention(q[:, :, m], k[:, :, m], v, 0.4, 5) for m in range(2)), 0.7, 0.2, 1e-5)
    torch.testing.assert_close(plain_maps(q, k, v, 0.4, 5, 0.7, 0.2, 1e-5, range(12)), want)


MAP_CASES = [(torch.float32, 10, 6, 8, 5, 3, 1), (torch.float32, 16, 24, 16, 64, 4, 2), (torch.float32, 64, 128, 64, 40, 2, 2), (torch.float32, 200, 256, 16, 21, 2, 1),
             (torch.bfloat16, 16, 32, 8, 17, 6, 3), (torch.bfloat16, 32, 48, 16, 50, 8, 2), (torch.bfloat16, 64, 128, 64, 64, 4, 2), (torch.bfloat16, 48, 96, 32, 33, 4, 1),
             (torch.bfloat16, 128, 256, 16, 70, 3, 1), (torch.bfloat16, 16, 24, 8, 1, 20, 1), (torch.bfloat16, 64, 8, 16, 90, 12, 1), (torch.bfloat16, 80, 64, 16, 65, 16, 1),
             (torch.bfloat16, 24, 40, 16, 30, 4, 2), (torch.bfloat16, 64, 64, 16, None, 4, 4)]


@pytest.mark.parametrize("dtype, d, e, page, W, heads, kv_heads", MAP_CASES)
def test_each_map_sees_exactly_its_window(dtype, d, e, page, W, heads, kv_heads):
    """One key stands out for the first map and another for the second: each query finds them from the key's own position
    to the last one of its window and not after; a map that read the other map's keys or queries, or a window that is one
    off, changes the result by more than the tolerance."""
    from yalis_b200.ops import attention as ops
    g = torch.Generator().manual_seed(d + e + heads)
    T, scale, balance, diff, eps = 230, d ** -0.5, 0.85, 0.3, 1e-4
    W_eff = W or 1000
    star1, star2 = 2 * page - 1, 2 * page + 1                                             # on both sides of a page border
    u1, u2 = (torch.nn.functional.normalize(torch.randn(d, generator=g), dim=0) for _ in range(2))
    q, k = torch.randn(T, heads, 2, d, generator=g), torch.randn(T, kv_heads, 2, d, generator=g) * 0.4
    v = torch.randn(T, kv_heads, e, generator=g)
    q[:, :, 0], q[:, :, 1] = q[:, :, 0] * 0.3 + 4 * u1, q[:, :, 1] * 0.3 + 4 * u2
    k[star1, :, 0], k[star2, :, 1] = (3.0 / scale) * u1, (3.0 / scale) * u2
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    ask = sorted({p for s in (star1, star2) for p in (0, s - 1, s, s + 1, s + W_eff - 1, s + W_eff, s + W_eff + 1, T - 2, T - 1) if 0 <= p < T})
    want = plain_maps(q.double(), k.double(), v.double(), scale, W, balance, diff, eps, ask)
    table, place = shuffled_table(T, page, seed=4)
    k_pool, v_pool = filled_pool(k.reshape(T, kv_heads, 2 * d), table, place, page), filled_pool(v, table, place, page)
    qm = q.reshape(T, heads * 2 * d).to(DEV)
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    difference = ops.MapDifference(balance, eps)

    def check(got, rows, what):
        for n, p in enumerate(rows):
            err = float((got[n].double().cpu().reshape(heads, e) - want[ask.index(p)]).abs().max())
            assert err < tol * float(want[ask.index(p)].abs().max()), f"{what}: position {p} off by {err}"

    common = dict(scale=scale, window=W, v_head_dim=e, out_scale=1 - diff, difference=difference)
    out = ops.paged_attention_generic(qm[ask].contiguous(), k_pool, v_pool, i32(ask), i32([0] * len(ask)), table, heads, kv_heads, d, **common)
    check(out, ask, "exact")
    if dtype == torch.bfloat16 and ops.mma_maps_supports(d, e):
        out = ops.paged_attention_mma(qm, k_pool, v_pool, i32(range(T)), i32([0, T]), i32([0] * T), table, T, heads, kv_heads, d, **common)
        check(out[ask], ask, "a whole prompt")
        a = ask[1]
        out = ops.paged_attention_mma(qm[a:].contiguous(), k_pool, v_pool, i32(range(a, T)), i32([0, T - a]), i32([0] * (T - a)), table, T - a, heads, kv_heads, d, **common)
        check(out[[p - a for p in ask if p >= a]], [p for p in ask if p >= a], "a portion")
        for splits in (1, 3, 7) if heads // kv_heads <= 16 else (1,):
            for p in ask:
                out = ops.paged_attention_mma(qm[p:p + 1].contiguous(), k_pool, v_pool, i32([p]), i32([0, 1]), i32([0]), table, 1, heads, kv_heads, d,
                                              n_splits=splits, **common)
                check(out, [p], f"decoded, {splits} splits")
    # the stars matter: without the window's edge or with the maps exchanged the result is another
    if W is not None and star1 + W < T and W > 2:
        p = star1 + W - 1
        fresh = plain_maps(q.double(), k.double(), v.double(), scale, W - 1, balance, diff, eps, [p])[0]
        assert float((fresh - want[ask.index(p)]).abs().max()) > 10 * tol * float(fresh.abs().max())
    swapped = plain_maps(q.double().flip(2), k.double().flip(2), v.double(), scale, W, balance, diff, eps, [star2 + 1])[0]
    if W is None or W > 2:
        assert float((swapped - want[ask.index(star2 + 1)]).abs().max()) > 5 * tol * float(swapped.abs().max())


@pytest.mark.parametrize("d, e, heads, kv_heads", [(32, 48, 4, 2), (64, 128, 6, 1), (16, 16, 20, 2)])
def test_unequal_requests_in_one_launch_each_as_alone(d, e, heads, kv_heads):
    """Equal bits: what else a launch holds leaves no trace, for portions and for single tokens with split keys."""
    from yalis_b200.ops import attention as ops
    g = torch.Generator().manual_seed(9)
    page, W = 16, 37
    lens, counts = [150, 61, 200, 5], [40, 61, 1, 2]
    width = max(-(-l // page) for l in lens)
    table = torch.full((4, width), -1, dtype=torch.int32)
    perm = iter(torch.randperm(60, generator=g).tolist())
    k_pool = torch.full((60, kv_heads, page, 2 * d), float("nan"), dtype=torch.bfloat16, device=DEV)
    v_pool = torch.full((60, kv_heads, page, e), float("nan"), dtype=torch.bfloat16, device=DEV)
    for r, l in enumerate(lens):
        for j in range(-(-l // page)):
            table[r, j] = pg = next(perm)
            rows = min(page, l - j * page)
            k_pool[pg, :, :rows] = torch.randn(kv_heads, rows, 2 * d, generator=g).to(torch.bfloat16).to(DEV)
            v_pool[pg, :, :rows] = torch.randn(kv_heads, rows, e, generator=g).to(torch.bfloat16).to(DEV)
    table = table.to(DEV)
    for counts, splits in (([40, 61, 1, 2], 1), ([1, 1, 1, 1], 4)):
        q = torch.randn(sum(counts), heads * 2 * d, generator=g).to(torch.bfloat16).to(DEV)
        pos = [p for l, c in zip(lens, counts) for p in range(l - c, l)]
        qs = [sum(counts[:i]) for i in range(5)]
        args = dict(window=W, v_head_dim=e, out_scale=0.6, difference=ops.MapDifference(0.4, 1e-5), n_splits=splits)
        together = ops.paged_attention_mma(q, k_pool, v_pool, i32(pos), i32(qs), i32([r for r, c in enumerate(counts) for _ in range(c)]), table, max(counts),
                                           heads, kv_heads, d, **args)
        assert not bool(together.isnan().any())
        for r, c in enumerate(counts):
            a, b = qs[r], qs[r + 1]
            alone = ops.paged_attention_mma(q[a:b].contiguous(), k_pool, v_pool, i32(pos[a:b]), i32([0, c]), i32([0] * c), table[r:r + 1].contiguous(), max(counts),
                                            heads, kv_heads, d, **args)
            assert torch.equal(alone, together[a:b]), (counts, r)


# ---- the router and the experts -----------------------------------------------------------------------------------------

@pytest.mark.parametrize("n, experts, top, groups, hidden", [(9, 6, 3, (3, 2), 40), (1100, 20, 4, (4, 2), 64), (50, 12, 5, None, 33), (70, 64, 8, (8, 3), 96),
                                                             (30, 200, 6, (10, 2), 64), (40, 1000, 32, (100, 9), 32), (12, 5, 5, (1, 1), 24), (20, 24, 1, (24, 1), 40)])
@pytest.mark.parametrize("low", [False, True])
def test_corrected_choice_among_the_best_groups(n, experts, top, groups, hidden, low):
    """``low``: corrections that make every choice score negative; a group that is masked with zero would then win."""
    from yalis_b200.ops.experts import route
    g = torch.Generator().manual_seed(n + experts)
    identity = experts // 4
    x = torch.randn(n, hidden, generator=g)
    w = torch.randn(experts, hidden, generator=g) * (2.0 / hidden ** 0.5)
    c = torch.randn(experts, generator=g) * 0.2 - (3.0 if low else 0.0)
    ids, weights, same = route(x.to(DEV), w.to(DEV), top, None, i32([0] * n), correction=c.to(DEV), groups=groups, identity=identity) if identity else \
        route(x.to(DEV), w.to(DEV), top, None, i32([0] * n), correction=c.to(DEV), groups=groups) + (torch.zeros(n),)
    rule = None if groups is None else {"count": groups[0], "keep": groups[1]}
    chosen, scores = plain.routing(x.double(), w.double(), c.double(), top, rule)
    ids, weights = ids.cpu().long(), weights.double().cpu()
    agree = (ids == chosen).all(dim=1)
    assert float(agree.float().mean()) > 0.97                        # a close call may fall the other way in float32
    torch.testing.assert_close(weights[agree], scores[agree], rtol=1e-4, atol=1e-7)
    want_same = (scores * (chosen >= experts - identity)).sum(dim=1)
    torch.testing.assert_close(same.double().cpu()[agree], want_same[agree], rtol=1e-4, atol=1e-7)
    # a correction decides: the same scores without it choose others
    if top < experts and groups is None:
        assert not torch.equal(plain.routing(x.double(), w.double(), torch.zeros(experts).double(), top, rule)[0], chosen)
    # rows of no request
    none = route(x[:2].to(DEV), w.to(DEV), top, None, i32([-1, 0]), correction=c.to(DEV), groups=groups, identity=identity)
    assert none[0][0].tolist() == [-1] * top and float(none[1][0].abs().max()) == 0.0
    assert not identity or float(none[2][0]) == 0.0


def test_ties_go_to_the_smaller_index_among_groups_and_outputs():
    from yalis_b200.ops.experts import route
    x, w = torch.zeros(1, 8), torch.zeros(8, 8)
    ids, weights = route(x.to(DEV), w.to(DEV), 2, None, i32([0]), correction=torch.zeros(8, device=DEV), groups=(4, 1))
    assert ids.tolist() == [[0, 1]] and weights.flatten().tolist() == pytest.approx([0.125, 0.125])
    c = torch.tensor([0.0, 0.0, 0.0, 1.0, 1.0, 0.0, 0.0, 0.0])
    ids, _ = route(x.to(DEV), w.to(DEV), 3, None, i32([0]), correction=c.to(DEV), groups=(4, 2))
    assert ids.tolist() == [[3, 4, 2]]
    ids, weights = route(x.to(DEV), w.to(DEV), 2, 1e-20, i32([0]), correction=c.to(DEV), score="sigmoid", factor=3.0)     # renormed, other scores
    assert ids.tolist() == [[3, 4]] and weights.flatten().tolist() == pytest.approx([1.5, 1.5])


def expert_tensors(hidden, experts, identity, inner, seed, dtype):
    g = torch.Generator().manual_seed(seed)
    t = {"router": (torch.randn(experts + identity, hidden, generator=g) * (3.0 / hidden ** 0.5)).to(dtype),
         "correction": (torch.randn(experts + identity, generator=g) * 0.2).to(dtype)}
    for e in range(experts):
        for name, shape in (("gate", (inner, hidden)), ("up", (inner, hidden)), ("down", (hidden, inner))):
            t[f"e{e}.{name}"] = (torch.randn(shape, generator=g) * (1.6 / shape[1] ** 0.5)).to(dtype)
    return t


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, hidden, experts, identity, top, inner, limit, groups", [
    (5, 64, 6, 2, 3, 24, 0.7, (4, 2)), (70, 36, 5, 0, 5, 18, 1.5, None), (900, 128, 10, 6, 2, 64, 3.0, (2, 1)), (300, 128, 16, 4, 4, 40, 1.0, (5, 3)),
    (1, 40, 1, 3, 2, 7, 2.0, (1, 1)), (40, 64, 3, 5, 8, 16, 1.0, None)])
def test_clamped_experts_beside_identity_experts(dtype, n, hidden, experts, identity, top, inner, limit, groups):
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import make_part
    t = expert_tensors(hidden, experts, identity, inner, n, dtype)
    rule = None if groups is None else {"count": groups[0], "keep": groups[1]}
    part = make_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": hidden, "experts": experts, "top": top, "expert_size": inner, "gated": True, "activation": "clamped", "limit": limit,
        "alpha": 1.702, "shift": 1.0, "shared_size": None, "renorm": False, "correction": True, "groups": rule, "identity": identity}))
    local = {"router": t["router"].float().to(DEV), "correction": t["correction"].float().to(DEV)}
    for e in range(experts):
        for name in ("gate", "up", "down"):
            local[f"expert_{e}_{name}"] = t[f"e{e}.{name}"].to(DEV)
    part.load(local)
    x = (torch.randn(n, hidden, generator=torch.Generator().manual_seed(1)) * 1.5).to(torch.bfloat16)
    got = part.forward(x.to(dtype).to(DEV), None).double().cpu()
    mlp = {"router": {"experts": experts, "identity": identity, "top": top, "groups": rule}, "expert": {"ff": inner, "limit": limit}}
    named = {"p." + k: v.double() for k, v in t.items()}
    want = plain.mixture_of_experts(x.double(), named, "p.", mlp)
    if dtype == torch.float32:
        err = (got - want).abs().max(dim=1).values / want.abs().max()
        assert float((err > 1e-4).float().mean()) <= 0.01, float(err.max())            # (a close call among hundreds of tokens)
    else:
        err = (got - want).abs().max(dim=1).values / want.abs().max()
        assert float(err.median()) < 2e-2 and float((err > 4e-2).float().mean()) <= 0.03, float(err.max())
    if identity and n > 4:
        chosen, _ = plain.routing(x.double(), named["p.router"], named["p.correction"], top, rule)
        assert bool((chosen >= experts).any()) and bool((chosen < experts).any())      # both kinds are chosen


# ---- whole models -----------------------------------------------------------------------------------------------------

TOL = {"float32": 1e-4, "bfloat16": 5e-2}       # relative to the largest |logit| of the request
LENGTHS = {"A": [1, 5, 33, 70, 21, 48], "B": [2, 40, 9, 64, 17, 90], "C": [3, 37, 18, 130, 12, 66], "D": [7, 1, 50, 19, 33, 4]}
PAGE = {"A": 16, "B": 8, "C": 64, "D": 16}
_oracle = {}


def requests_for(which):
    cfg, _ = plain.read_folder(lagulorn_dir(which))
    g = torch.Generator().manual_seed(ord(which) + 100)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[which])}


def oracle(which):
    if which not in _oracle:
        cfg, w = plain.read_folder(lagulorn_dir(which))
        _oracle[which] = {rid: plain.forward(cfg, w, t).numpy() for rid, t in requests_for(which).items()}
    return _oracle[which]


def replay(model_dir, page, dtype, steps, max_tokens, graphs=False):
    from yalis_b200.engine.replay import Replayer
    rep = Replayer(model_dir, dtype, max_tokens, page_size=page, graphs=graphs)
    out = {}
    for s in steps:
        r = rep.run_step(s)
        if r is not None:
            out[s["step"]] = r
    rep.engine.check_device_errors()
    rep.engine.manager.check()
    for grp in rep.engine.groups:
        assert rep.engine.manager.free_pages(grp.name) == grp.num_pages          # every page came back
    return out, rep


def compare(got, want, tol, what, outliers=0.0):
    assert set(got) == set(want), what
    total = bad = 0
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        err = np.abs(got[rid] - want[rid]).max(axis=1) / np.abs(want[rid]).max()
        assert np.isfinite(err).all(), (what, rid)
        total += len(err)
        bad += int((err > tol).sum())
        if err.max() > tol and not outliers:
            raise AssertionError(f"{what}: request {rid} differs by {err.max():.3e} (tolerance {tol}); first wrong "
                                 f"position {int(np.argmax(err > tol))} of {len(err)}")
    assert bad <= outliers * total, f"{what}: {bad} of {total} positions differ by more than {tol}"


# bfloat16: a token whose last chosen output and the first one left out (or the last group kept and the first one not)
# score nearly alike may run another expert than the float64 model
OUTLIERS = {"A": 0.06, "B": 0.06, "C": 0.06, "D": 0.06}


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_requests_cut_four_ways_agree_with_the_plain_model(which, dtype):
    reqs, want = requests_for(which), oracle(which)
    vocab = plain.read_folder(lagulorn_dir(which))[0]["vocab"]
    outliers = 0.0 if dtype == "float32" else OUTLIERS[which]
    results = {}
    for name, steps in (("whole", traces.whole(reqs)), ("tail", traces.tail_decoded(reqs, tail=12)),
                        ("portions", traces.portions(reqs, seed=3)), ("mixed", traces.mixed(reqs, seed=5, tail=6))):
        steps = traces.number(steps)
        out, _ = replay(lagulorn_dir(which), PAGE[which], dtype, steps, traces.peak_tokens(steps, max(64, PAGE[which])))
        results[name] = traces.collect(steps, out, vocab)
        compare(results[name], want, TOL[dtype], f"{which} {dtype} {name}", outliers=outliers)
    # how a request was cut, what ran beside it and which pages and slots it had leave (nearly) no trace
    for name in ("tail", "portions", "mixed"):
        for rid in want:
            diff = np.abs(results[name][rid] - results["whole"][rid]).max(axis=1) / np.abs(want[rid]).max()
            if dtype == "float32":
                assert diff.max() < 2e-5, (name, rid)
            else:
                assert np.mean(diff > 5e-2) <= outliers or len(diff) < 20, (name, rid)


@pytest.mark.parametrize("which", ["A", "C", "D"])
def test_steps_replayed_from_recordings_give_the_same(which):
    """Decoded tokens through recorded steps (CUDA graphs): routing, identity weights and states are read on the device."""
    reqs, want = requests_for(which), oracle(which)
    vocab = plain.read_folder(lagulorn_dir(which))[0]["vocab"]
    steps = traces.number(traces.tail_decoded(reqs, tail=12))
    peak = traces.peak_tokens(steps, max(64, PAGE[which]))
    launched, _ = replay(lagulorn_dir(which), PAGE[which], "float32", steps, peak)
    recorded, rep = replay(lagulorn_dir(which), PAGE[which], "float32", steps, peak, graphs=True)
    assert rep.steps_replayed > 40
    a, b = traces.collect(steps, launched, vocab), traces.collect(steps, recorded, vocab)
    compare(b, want, TOL["float32"], f"{which} recorded")
    for rid in a:
        assert np.abs(a[rid] - b[rid]).max() / np.abs(a[rid]).max() < 1e-6


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_the_sum_of_the_copies_after_every_layer(which):
    """A layer that runs another's tensors counts like any other."""
    from yalis_b200.engine.engine import Engine, StepEntry
    d = lagulorn_dir(which)
    cfg, w = plain.read_folder(d)
    tokens = requests_for(which)["r2"]
    want = []
    plain.forward(cfg, w, tokens, taps=want)
    eng = Engine(d, dtype="float32", page_size=16, num_pages=8, max_slots=2, max_context=128)
    eng.add_request("x")
    seen = []
    inner = eng.model.forward
    eng.model.forward = lambda ctx, caches: inner(ctx, caches, tap=lambda i, x: seen.append(x.double().cpu()))
    eng.run([StepEntry("x", tokens, [len(tokens) - 1])])
    assert len(seen) == len(want) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, want)):
        assert float((a - b).abs().max() / b.abs().max()) < 2e-5, f"layer {i}"


@pytest.mark.parametrize("which, dtype", [("A", "float32"), ("B", "float32"), ("C", "bfloat16"), ("D", "float32")])
def test_long_decoding_keeps_to_the_plain_model(which, dtype):
    """300 tokens one by one after a two-token prompt, through pages of eight that come back behind the windows and are
    used again; the states are carried 300 times."""
    from yalis_b200.engine.engine import Engine, StepEntry
    d = lagulorn_dir(which)
    cfg, w = plain.read_folder(d)
    tokens = torch.randint(0, cfg["vocab"], (302,), generator=torch.Generator().manual_seed(9)).tolist()
    want = plain.forward(cfg, w, tokens).numpy()
    eng = Engine(d, dtype=dtype, page_size=8, num_pages=14 if which != "D" else 40, max_slots=2, max_context=384)
    eng.add_request("x")
    rows = [eng.run([StepEntry("x", tokens[:2], [0, 1])]).logits.cpu().numpy()]
    for t in tokens[2:]:
        rows.append(eng.run([StepEntry("x", [t], [0])]).logits.cpu().numpy())
    got = np.concatenate(rows)
    eng.check_device_errors()
    err = np.abs(got - want).max(axis=1) / np.abs(want).max()
    if dtype == "float32":
        assert err.max() < 1e-4
    else:
        assert np.mean(err > 5e-2) <= OUTLIERS[which]


@pytest.mark.parametrize("which", ["A", "C"])
def test_a_slot_and_its_pages_used_again_start_clean(which):
    """The states and pages of a finished request must not show in the next one, for every run of shared tensors."""
    from yalis_b200.engine.engine import Engine, StepEntry
    d = lagulorn_dir(which)
    reqs = requests_for(which)
    eng = Engine(d, dtype="float32", page_size=64, num_pages=3, max_slots=1, max_context=192)
    first = None
    for rid in ("r3", "r2", "r3"):
        assert eng.add_request(rid) == 0                       # the only slot, every time
        cut = len(reqs[rid]) // 2                              # in two portions: the second starts from slot and pages
        eng.run([StepEntry(rid, reqs[rid][:cut], [])])
        out = eng.run([StepEntry(rid, reqs[rid][cut:], [len(reqs[rid]) - cut - 1])]).logits.cpu().numpy()
        eng.finish_request(rid)
        if rid == "r3":
            if first is None:
                first = out
            else:
                assert np.array_equal(first, out)


@pytest.mark.parametrize("which", ["A", "B", "D"])
def test_greedy_generation_through_the_entry_point(which):
    from yalis_b200 import InferenceConfig, LLMEngine, ModelConfig
    d = lagulorn_dir(which)
    cfg, w = plain.read_folder(d)
    g = torch.Generator().manual_seed(4)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (3, 19, 40, 7, 26)]
    engine = LLMEngine(ModelConfig(model_name=f"lagulorn-tiny-{which}", model_path=d, precision="fp32"),
                       InferenceConfig(max_batch_size=3, max_length_of_generated_sequences=64, temperature=0.0, top_p=0.0,
                                       page_size=PAGE[which]))
    tokens, metrics = engine.generate(prompts, tokens_to_generate=10)[:2]
    for p, row in zip(prompts, tokens.cpu().tolist()):
        assert row == plain.greedy(cfg, w, p, 10)


def test_the_replay_program_runs_a_lagulorn_folder(tmp_path):
    reqs = {k: v for k, v in requests_for("B").items() if k in ("r1", "r2")}
    steps = traces.number(traces.portions(reqs, seed=1))
    out_dir = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", lagulorn_dir("B"), "--dtype", "float32",
                           "--out", str(out_dir), "--max-tokens", str(traces.peak_tokens(steps))],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    vocab = plain.read_folder(lagulorn_dir("B"))[0]["vocab"]
    outputs = {s["step"]: np.fromfile(out_dir / f"{s['step']}.f32", dtype="<f4") for s in steps}
    compare(traces.collect(steps, outputs, vocab), {k: oracle("B")[k] for k in reqs}, TOL["float32"], "program")


# ---- configurations drawn at random -------------------------------------------------------------------------------------

def random_lagulorn(rng):
    from yalis_b200.config.presets import _lagulorn, _lg_attention, _lg_dense, _lg_lightning, _lg_moe

    def mlp():
        kind = rng.choice(["none", "dense", "moe", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return _lg_dense(rng.choice([24, 70, 128, 200]))
        count = rng.choice([1, 2, 3, 4])
        size = rng.choice([2, 3, 4, 5])
        outputs, keep = count * size, rng.randint(1, count)
        identity = rng.randint(0, outputs - 1)
        return _lg_moe(outputs - identity, rng.randint(1, min(6, keep * size)), rng.choice([9, 24, 40, 64]), rng.choice([0.3, 1.0, 2.5]), identity,
                       rng.choice([None, (count, keep)]))

    def layer():
        if rng.random() < 0.5:
            heads = rng.choice([1, 2, 3, 4])
            return _lg_lightning(heads, rng.choice([5, 8, 16, 24, 40, 64]), rng.choice([3, 8, 20, 32, 64]),
                                 [rng.choice([0.0, 0.5, 0.9, 0.99, 0.999, 1.0]) for _ in range(heads)], mlp())
        kv = rng.choice([1, 1, 2, 3])
        d = rng.choice([6, 8, 16, 24, 32, 48, 64])
        return _lg_attention(kv * rng.choice([1, 2, 3, 10]), kv, d, rng.choice([5, 8, 16, 40, 64, 96]), rng.choice([d ** -0.5, 0.3]), rng.choice([-0.2, 0.3, 0.8]),
                             rng.choice([1, 2, 7, 16, 33, 64, 500]), mlp())

    layers = []
    for i in range(rng.randint(2, 6)):
        layers.append(rng.randrange(i) if i and rng.random() < 0.25 else layer())
    return _lagulorn(rng.choice([48, 64, 90, 136, 192]), rng.choice([80, 300, 701]), rng.choice([None, 1, 2, 3, 4, 6]), layers,
                     embedding_scale=rng.choice([1.0, 4.0]), residual_mult=rng.choice([0.2, 0.6, 1.0]), eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", [41, 42, 43, 44, 45, 46, 47, 48, 49, 50])
def test_configurations_drawn_at_random(seed, tmp_path):
    rng = random.Random(seed)
    config = random_lagulorn(rng)
    d = write_model(config, str(tmp_path / "m"), seed)
    cfg, w = plain.read_folder(d)
    page = rng.choice([8, 16, 32, 64])
    g = torch.Generator().manual_seed(seed)
    reqs = {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
            for i, n in enumerate([rng.randint(1, 30), rng.randint(31, 90), rng.randint(40, 110), rng.randint(2, 9), rng.randint(10, 60)])}
    want = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for dtype, cuttings in (("float32", ("whole", "portions", "mixed")), ("bfloat16", ("mixed",))):
        for name in cuttings:
            steps = traces.number({"whole": traces.whole, "portions": lambda r: traces.portions(r, seed=seed),
                                   "mixed": lambda r: traces.mixed(r, seed=seed, tail=5)}[name](reqs))
            out, _ = replay(d, page, dtype, steps, traces.peak_tokens(steps, max(64, page)))
            got = traces.collect(steps, out, cfg["vocab"])
            what = f"seed {seed} {dtype} {name}: {config}"
            if dtype == "float32":
                compare(got, want, TOL[dtype], what)
            else:
                # close calls of the routers decide much, and a state carries them on: most positions keep to the plain model
                errs = np.concatenate([np.abs(got[r] - want[r]).max(axis=1) / np.abs(want[r]).max() for r in want])
                assert np.isfinite(errs).all() and np.median(errs) < 4e-2 and np.mean(errs > 0.08) < 0.15, (what, float(np.median(errs)), float(np.mean(errs > 0.08)))
