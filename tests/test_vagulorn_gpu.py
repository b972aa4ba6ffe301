"""Vagulorn on the GPU: every new kernel alone against its plain statement (tests/torch_ops.py, float64), with inputs made so that a
lost state, a kept token that is left out or a key that is one token off shows; then the engine in both precisions against the plain
whole-sequence implementation: prompts, token-by-token decoding, portions down to two tokens, unequal requests in one batch, slots
and pages that are used again, long decoding through captured graphs, greedy generation through the scheduler, the tools."""
import json
import os
import random

import pytest
import torch

from gpu_util import assert_close
from test_vafozen_gpu import _fill_pages, batch, rnd, to_cpu
from torch_ops import TorchOps
from vagulorn_util import (CFG_A, CFG_B, CFG_C, assert_within_32_bit, assert_within_rounding, chunked, lightning, mixed_schedule, model, pair,
                           plain_logits, random_config, softmax, ssm, tokens, write_model)

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
REF = TorchOps()


@pytest.fixture(scope="module")
def ops():
    from nanoinfer_b200.csrc.lib import load_kernels
    return load_kernels()


def cpu(x):
    return x.cpu() if torch.is_tensor(x) else x


# ------------------------------------------------------------------------------------------ layer norm
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,width", [(1, 64), (9, 36), (5, 100), (70, 258), (3, 512), (8, 516), (33, 1024), (2, 1280), (5, 2048), (3, 4096), (4, 4100), (2, 1)])
def test_layer_norm(ops, dtype, m, width):
    """Rows with a mean a thousand times their deviation (the variance is that of the deviations), and a choice of rows."""
    x, g, b = rnd(m, width, seed=1) + 1000.0 * rnd(m, 1, seed=2), rnd(width, seed=3), rnd(width, seed=4)
    x = x.to(torch.float32)
    x[0] = rnd(width, seed=5, scale=0.01)
    for rows in (None, torch.tensor([m - 1, 0, m // 2], dtype=torch.int32, device=DEV)):
        out = torch.empty(m if rows is None else 3, width, dtype=dtype, device=DEV)
        ref = torch.empty(out.shape, dtype=torch.float64)
        ops.layernorm(x, g, b, 1e-5, out, rows)
        REF.layernorm(x.cpu(), g.cpu(), b.cpu(), 1e-5, ref, cpu(rows))
        if dtype == torch.float32:      # (a sum of a thousand numbers near 1,000 is known to 1e-4 of their deviation)
            assert (out.cpu().double() - ref).abs().max().item() < 1e-3 * max(1.0, ref.abs().max().item())
            assert_close(out[out.shape[0] - m:][:1] if rows is None else out[1:2], ref[:1] if rows is None else ref[1:2], dtype)
        else:
            assert_close(out, ref, dtype)


# ------------------------------------------------------------------------------------------ the gelu-gated product
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,inter,k", [(1, 24, 40), (3, 72, 96), (7, 200, 128), (12, 130, 256), (30, 96, 64), (50, 300, 320), (90, 136, 200), (200, 256, 128), (300, 264, 192), (520, 384, 256)])
def test_gelu_gated_product(ops, dtype, m, inter, k):
    """Gates from far below zero to far above; every product kernel that the sizes reach."""
    a, w = rnd(m, k, seed=1).to(dtype), rnd(2 * inter, k, seed=2, scale=3.0 / k ** 0.5).to(dtype)
    w[:inter:7] *= 8.0
    ref = torch.empty(m, inter, dtype=torch.float64)
    REF.linear_swiglu(a.cpu(), w.cpu(), ref, act="gelu_tanh")
    routes = [None] + (["smallm", "tc", "tc_pair"] if dtype == torch.bfloat16 and k % 32 == 0 else [])
    for route in routes:
        if route == "smallm" and m > 64:
            continue
        out = torch.empty(m, inter, dtype=dtype, device=DEV)
        (ops if route is None else ops.with_options(gemm_route=route)).linear_swiglu(a, w, out, act="gelu_tanh")
        assert_close(out, ref, dtype, str(route))


# ------------------------------------------------------------------------------------------ operands of the attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,d,rot", [(4, 2, 64, 32), (6, 3, 32, 8), (2, 1, 128, 128), (3, 3, 16, 16), (4, 1, 24, 24), (2, 2, 10, 2), (3, 1, 40, 16)])
def test_interleaved_operands_whose_values_are_the_projected_keys(ops, dtype, heads, kv, d, rot):
    """A long step (eight elements a thread in bfloat16) and a short one; rows lie apart in a wider matrix."""
    freq = torch.pow(torch.tensor(500.0, dtype=torch.float64), -2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot).float().to(DEV)
    for q_lens, before in (([290, 1, 40], [3, 70, 0]), ([1, 5], [9, 30])):
        ctx, bt, num_pages = batch(q_lens, before, page_size=8)
        m, n = sum(q_lens), (heads + kv) * d
        wide = rnd(m, n + 12, seed=1)
        qk = wide[:, 4:4 + n]
        gains = (rnd(d, seed=2), rnd(d, seed=3))
        kp, vp = torch.zeros(num_pages, kv, 8, d, dtype=dtype, device=DEV), torch.zeros(num_pages, kv, 8, d, dtype=dtype, device=DEV)
        q = torch.empty(m, heads * d, dtype=dtype, device=DEV)
        args = (heads, kv, d, d)
        kw = dict(layout="interleaved", values_are_keys=True)
        ops.attention_prepare(qk, q, *args, *gains, 1e-5, freq, rot, ctx, bt, 8, kp, vp, True, **kw)
        rq, rk, rv = torch.empty(q.shape, dtype=torch.float64), torch.zeros(kp.shape, dtype=torch.float64), torch.zeros(vp.shape, dtype=torch.float64)
        REF.attention_prepare(qk.cpu(), rq, *args, *(g.cpu() for g in gains), 1e-5, freq.cpu(), rot, to_cpu(ctx), bt.cpu(), 8, rk, rv, True, **kw)
        tol = 5.0 if dtype == torch.float32 else 1.0        # (angles of a few hundred radians are 32-bit products)
        for got, ref, what in ((q, rq, "q"), (kp, rk, "k"), (vp, rv, "v")):
            if dtype == torch.float32:
                assert (got.cpu().double() - ref).abs().max().item() < tol * 2e-5 * max(1.0, ref.abs().max().item()), what
            else:
                assert_close(got, ref, dtype, what)


# ------------------------------------------------------------------------------------------ windows with kept first tokens, a gate per head
def paged_inputs(ops, dtype, q_lens, before, page, heads, kv, dk, dv, window, keep, seed=3):
    """A step's queries over filled pages of which only those that the window or the kept tokens need are still held."""
    full_ctx, full_bt, num_pages = batch([b + q for b, q in zip(before, q_lens)], [0] * len(q_lens), page_size=page)
    ctx, _, _ = batch(q_lens, before, page_size=page)
    qkv = rnd(sum(q_lens) + sum(before), heads * dk + kv * (dk + dv), seed=seed, scale=0.7)
    q_all, kp, vp = _fill_pages(ops, dtype, full_ctx, full_bt, page, num_pages, heads, kv, dk, dv, qkv)
    starts = full_ctx.q_start.cpu().tolist()
    rows = torch.cat([torch.arange(s + b, s + b + q) for s, b, q in zip(starts, before, q_lens)]).to(DEV)
    bt = full_bt.clone()
    for r, b in enumerate(before):
        bt[r, -(-keep // page):max(-(-keep // page), max(0, b - window + 1) // page)] = -1
    return q_all[rows].contiguous(), ctx, bt, kp, vp


KEPT = [(4, 70, 2), (1, 33, 0), (16, 16, 3), (20, 5, 40), (65, 64, 129), (130, 17, 200), (300, 9, 1), (3, 1, 0)]     # keep, window, seed of the gate


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("keep,window,seed", KEPT)
@pytest.mark.parametrize("heads,kv,dk,dv,page", [(4, 2, 64, 64, 16), (2, 1, 128, 128, 16), (3, 1, 12, 8, 4), (6, 3, 40, 40, 8), (2, 2, 96, 32, 16), (1, 1, 136, 20, 8)])
def test_kept_first_tokens_and_a_gate_per_head(ops, dtype, keep, window, seed, heads, kv, dk, dv, page):
    """Prompt portions far behind the kept tokens, over them and at the start; single tokens; a mix (leading single tokens)."""
    for q_lens, before in (([150, 90], [260, 0]), ([1, 1, 1], [400, 3, 66]), ([1, 40, 2], [333, 120, 18])):
        q, ctx, bt, kp, vp = paged_inputs(ops, dtype, q_lens, before, page, heads, kv, dk, dv, window, keep)
        m = sum(q_lens)
        gate = rnd(m, heads + 5, seed=seed)[:, 2:2 + heads]
        ref = torch.empty(m, heads * dv, dtype=torch.float64)
        rest = (heads, kv, dk, dv, 0.3, 0.0, None, window, 0, 1.7)
        REF.attention_flex(q.cpu(), ref, *rest, to_cpu(ctx), bt.cpu(), page, kp.cpu(), vp.cpu(), keep_first=keep, gate32=gate.cpu())
        for what, k in (("default", ops), ("mma.sync", ops.with_options(force_mma_prefill=True)), ("general", ops.with_options(force_general_attention=True)),
                        ("split keys", ops.with_options(fixed_decode_splits=5))):
            out = torch.empty(m, heads * dv, dtype=dtype, device=DEV)
            k.attention_flex(q, out, *rest, ctx, bt, page, kp, vp, keep_first=keep, gate32=gate)
            assert_close(out, ref, dtype, f"{what} {q_lens}")
            if dtype == torch.float32:
                break
    ops.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("d", [64, 40])
@pytest.mark.parametrize("keep,window,page", [(1, 4, 4), (4, 70, 16), (16, 33, 16), (17, 64, 16), (64, 30, 16), (65, 128, 8), (3, 1, 16)])
def test_edges_of_the_kept_tokens_and_of_the_window(ops, keep, window, page, d, decode, dtype):
    """Four marked keys whose scores stand out: the last kept token, the first that is not kept, the last behind the window, the
    first inside it. The query must return the mean of the visible marks, whatever its place in a portion."""
    n = keep + 3 * window + 150
    p = n - 2
    marks = {keep - 1: 1.0, keep: 10.0, p - window: 100.0, p - window + 1: 1000.0}
    qkv = torch.zeros(n, 3 * d, device=DEV)
    qkv[:, d] = 1.0
    for pos, mark in marks.items():
        qkv[pos, d + 1] = 9.0
        qkv[pos, 2 * d:] = mark
    qkv[:, 1] = 9.0
    full_ctx, bt, num_pages = batch([n], [0], page_size=page)
    q_all, kp, vp = _fill_pages(ops, dtype, full_ctx, bt, page, num_pages, 1, 1, d, d, qkv)
    for pos in (p - 1, p, p + 1):
        seen = [v for j, v in marks.items() if j <= pos and (pos - j < window or j < keep)]
        first = pos if decode else max(0, pos - 100)
        ctx, _, _ = batch([pos + 1 - first], [first], page_size=page)
        out = torch.empty(pos + 1 - first, d, dtype=dtype, device=DEV)
        ops.attention_flex(q_all[first:pos + 1].contiguous(), out, 1, 1, d, d, 1.0, 0.0, None, window, 0, 1.0, ctx, bt, page, kp, vp, keep_first=keep)
        want = sum(seen) / len(seen)
        assert abs(out[-1, 0].item() - want) < 0.01 * want, (pos, out[-1, 0].item(), want)
    ops.check_device_errors()


# ------------------------------------------------------------------------------------------ matrix states with one decay per head
def state_inputs(m, heads, kq, dk, dv, kind, seed=1, dtype=torch.float32):
    """q, k and v hold bfloat16 numbers (as floats, or stored as such), so that the chunks' operands lose nothing and only what has to
    be 32-bit can differ."""
    stored = lambda x: x.to(torch.bfloat16).to(dtype)
    g = {"q": stored(rnd(m, kq * dk, seed=seed)), "k": stored(rnd(m, kq * dk, seed=seed + 1)), "v": stored(rnd(m, heads * dv, seed=seed + 2))}
    if kind == "steps":
        kw = {"dt_bias32": rnd(heads, seed=5) - 2.0, "a_log32": rnd(heads, seed=6)}
        g["raw32"] = rnd(m, heads + 3, seed=seed + 3)[:, 1:1 + heads]
    else:
        kw = {"decay32": fixed_decays(torch.linspace(0.3, 0.999, heads))}
    return g, kw


def fixed_decays(d):
    d = d.double()
    return torch.stack([d, torch.log2(d)]).float().to(DEV)


def run_scan(k, g, kw, rows, state, off, ctx, heads, kq, dk, dv, dev=DEV, **more):
    pick = {n: t[rows] if dev == DEV else t[rows].cpu() for n, t in g.items()}
    kw = kw if dev == DEV else {n: cpu(t) for n, t in kw.items()}
    out = torch.empty(len(rows), heads * dv, device=dev)
    k.decay_state_scan(pick.pop("q"), pick.pop("k"), pick.pop("v"), state, off, ctx, out, heads, kq, dk, dv, **pick, **kw, **more)
    return out


def near(got, ref, what, rel=4e-5):
    """Well inside 16 bits of the largest value: a bfloat16 state or decay would be off by a hundred times as much."""
    err, top = (got.cpu().double() - ref.double()).abs().max().item(), ref.abs().max().item()
    assert err <= rel * max(1.0, top), f"{what}: {err:.3e} of {top:.3e}"


SIZES = [(1, 1, 8, 5), (3, 3, 20, 12), (4, 2, 48, 40), (2, 2, 64, 64), (6, 2, 33, 7), (2, 1, 100, 33), (2, 1, 128, 64), (4, 2, 64, 128), (2, 2, 128, 128),
         (6, 3, 1, 8), (1, 1, 32, 1), (2, 2, 130, 20), (1, 1, 256, 130)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["steps", "fixed"])
@pytest.mark.parametrize("heads,kq,dk,dv", SIZES)
def test_states_whole_and_cut_anywhere(ops, heads, kq, dk, dv, kind, dtype):
    """Whole (chunks, the last one partly filled), exactly, then in portions (single tokens, short steps, steps at and beyond a chunk's
    edge) beside another request's rows; the state sits between other columns of a wider state row and does not start from zero."""
    n, off = 300, 11
    size = heads * dv * dk
    g, kw = state_inputs(n + 60, heads, kq, dk, dv, kind, dtype=dtype)
    start = rnd(3, off + size + 4, seed=9, scale=0.3)
    rstate = start.cpu().clone()
    ctx, _, _ = batch([n], [0], slots=[1])
    ref = run_scan(REF, g, kw, list(range(n)), rstate, off, to_cpu(ctx), heads, kq, dk, dv, "cpu")
    for what, more in (("chunks", {}), ("exact", {"exact": True})):
        state = start.clone()
        near(run_scan(ops, g, kw, list(range(n)), state, off, ctx, heads, kq, dk, dv, **more), ref, what)
        near(state, rstate, what + ", state")
        assert torch.equal(state[[0, 2]], start[[0, 2]]) and torch.equal(state[1, :off], start[1, :off]) and torch.equal(state[1, off + size:], start[1, off + size:])
    state = start[[1, 0, 2]].clone()
    got, pos, opos = [], 0, n
    for c in [2, 1, 64, 17, 1, 65, 2, 16, 63, 69]:
        oc = min(1 if c > 3 else 5, n + 60 - opos)
        ctx, _, _ = batch([oc, c], [0, 0], slots=[2, 0])
        out = run_scan(ops, g, kw, list(range(opos, opos + oc)) + list(range(pos, pos + c)), state, off, ctx, heads, kq, dk, dv)
        got.append(out[oc:])
        pos, opos = pos + c, opos + oc
    assert pos == n
    near(torch.cat(got), ref, "in portions")
    near(state[0], rstate[1], "state after portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,heads,kq,dk,dv", [("steps", 4, 2, 64, 48), ("fixed", 3, 3, 64, 70), ("steps", 2, 1, 128, 64), ("fixed", 1, 1, 40, 8), ("steps", 2, 2, 96, 144)])
def test_unequal_requests_side_by_side(ops, kind, heads, kq, dk, dv, dtype):
    """Leading single tokens (token by token) beside portions of one to many chunks, twice from the states that are left."""
    q_lens, slots, off = [1, 1, 700, 3, 64, 65, 128], [5, 2, 0, 1, 4, 6, 3], 8
    g, kw = state_inputs(sum(q_lens), heads, kq, dk, dv, kind, seed=3, dtype=dtype)
    ctx, _, _ = batch(q_lens, [0] * 7, slots=slots)
    state = rnd(7, off + heads * dv * dk + 2, seed=9, scale=0.3)
    rstate = state.cpu().clone()
    rows = list(range(sum(q_lens)))
    for step in range(2):
        near(run_scan(ops, g, kw, rows, state, off, ctx, heads, kq, dk, dv), run_scan(REF, g, kw, rows, rstate, off, to_cpu(ctx), heads, kq, dk, dv, "cpu"), f"step {step}")
        near(state, rstate, f"state {step}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kq,dk,dv", [(32, 2, 24, 40), (12, 6, 72, 68), (10, 10, 128, 130), (16, 1, 64, 64)])
def test_many_heads_that_share_their_keys(ops, heads, kq, dk, dv, dtype):
    """Enough heads and tokens that a block takes two units (heads of one group, or the value channels of one head), beside sizes
    where it does not; a short request between two long ones."""
    q_lens, slots = [1000, 30, 800], [1, 0, 2]
    g, kw = state_inputs(sum(q_lens), heads, kq, dk, dv, "steps", seed=5, dtype=dtype)
    ctx, _, _ = batch(q_lens, [0] * 3, slots=slots)
    state = rnd(3, heads * dv * dk, seed=9, scale=0.3)
    rstate = state.cpu().clone()
    rows = list(range(sum(q_lens)))
    near(run_scan(ops, g, kw, rows, state, 0, ctx, heads, kq, dk, dv), run_scan(REF, g, kw, rows, rstate, 0, to_cpu(ctx), heads, kq, dk, dv, "cpu"), "outputs")
    near(state, rstate, "states")


@pytest.mark.parametrize("n", [3, 16, 17, 200])
def test_activations_stand_before_the_state(ops, n):
    heads, dk, dv = 3, 24, 20
    q, k, v = rnd(n, heads * dk, seed=1), rnd(n, heads * dk, seed=2), rnd(n, heads * dv, seed=3)
    ctx, _, _ = batch([n], [0])
    kw = dict(act="silu", decay32=fixed_decays(torch.tensor([0.5, 0.9, 0.99])))
    ref, rstate = torch.empty(n, heads * dv), torch.zeros(1, heads * dk * dv)
    REF.decay_state_scan(q.cpu(), k.cpu(), v.cpu(), rstate, 0, to_cpu(ctx), ref, heads, heads, dk, dv, **{a: cpu(b) for a, b in kw.items()})
    for exact in (False, True):
        out, state = torch.empty(n, heads * dv, device=DEV), torch.zeros(1, heads * dk * dv, device=DEV)
        ops.decay_state_scan(q, k, v, state, 0, ctx, out, heads, heads, dk, dv, exact=exact, **kw)
        dtype = torch.float32 if exact or n <= 16 else torch.bfloat16
        assert_close(out, ref, dtype)
        assert_close(state, rstate, dtype)


@pytest.mark.parametrize("exact", [False, True])
def test_a_far_key_is_found_through_slow_decays_and_lost_through_fast_ones(ops, exact):
    """One token writes a value under a key of its own; 2,000 tokens later a query finds it, scaled by the decays in between, in
    one head; in a head with a faster decay it is gone; a decay of one keeps it whole and a decay of zero not a token long."""
    n, dk, dv, where = 2100, 16, 8, 70
    decays = [0.9995, 0.9, 1.0, 0.0]
    q, k, v = torch.zeros(n, 4 * dk, device=DEV), rnd(n, 4 * dk, seed=1, scale=0.25).bfloat16().float(), rnd(n, 4 * dv, seed=2).bfloat16().float()
    for h in range(4):
        k[:, h * dk + 3] = 0.0
        k[where, h * dk:(h + 1) * dk] = 0.0
        k[where, h * dk + 3] = 1.0
        q[2070, h * dk + 3] = q[where, h * dk + 3] = q[where + 1, h * dk + 3] = 1.0
    ctx, _, _ = batch([n], [0])
    out = torch.empty(n, 4 * dv, device=DEV)
    ops.decay_state_scan(q, k, v, torch.zeros(1, 4 * dk * dv, device=DEV), 0, ctx, out, 4, 4, dk, dv, decay32=fixed_decays(torch.tensor(decays)), exact=exact)
    for at in (where, where + 1, 2070):
        for h, d in enumerate(decays):
            want = v[where, h * dv:(h + 1) * dv].double() * float(torch.tensor(d, dtype=torch.float64) ** (at - where))
            got = out[at, h * dv:(h + 1) * dv].double()
            assert (got - want).abs().max().item() <= 1e-4 * want.abs().max().item() + 1e-7, (at, d)     # (a decay is a 32-bit number)


def test_strong_decays_cost_the_tokens_behind_them_nothing(ops):
    """Step sizes of 10^4 now and then (everything before is wiped out) among tiny ones: what follows within the same chunk is as
    exact as without them, and nothing turns into NaN."""
    n, dk, dv = 400, 32, 16
    g, _ = state_inputs(n, 1, 1, dk, dv, "fixed")
    raw = torch.full((n, 1), -6.0, device=DEV)
    raw[3::67] = 1e4
    g["raw32"] = raw
    kw = {"dt_bias32": torch.zeros(1, device=DEV), "a_log32": torch.zeros(1, device=DEV)}
    g["v"][3::67] = (g["v"][3::67] * 1e-4).bfloat16().float()
    ctx, _, _ = batch([n], [0])
    state, rstate = torch.zeros(1, dk * dv, device=DEV), torch.zeros(1, dk * dv)
    ref = run_scan(REF, g, kw, list(range(n)), rstate, 0, to_cpu(ctx), 1, 1, dk, dv, "cpu")
    near(run_scan(ops, g, kw, list(range(n)), state, 0, ctx, 1, 1, dk, dv), ref, "outputs", rel=2e-5)
    near(state, rstate, "state", rel=2e-5)


def test_one_launch_for_a_short_step_and_three_for_chunks(ops):
    g, kw = state_inputs(101, 2, 2, 64, 64, "steps")
    state = torch.zeros(3, 2 * 64 * 64, device=DEV)
    for q_lens, launches in (([1, 1, 1], 1), ([16, 2, 9], 1), ([17, 1, 1], 3), ([1, 1, 99], 4)):
        ctx, _, _ = batch(q_lens, [0] * 3)
        before = ops.launches
        run_scan(ops, g, kw, list(range(sum(q_lens))), state, 0, ctx, 2, 2, 64, 64)
        assert ops.launches - before == launches, q_lens


# ------------------------------------------------------------------------------------------ around the states
@pytest.mark.parametrize("out,skip_type", [(a, b) for a in DTYPES for b in DTYPES])
@pytest.mark.parametrize("m,parts,width,heads", [(5, 2, 260, 4), (3, 1, 512, 8), (9, 3, 1024, 6), (2, 2, 2048, 32), (4, 1, 4096, 16), (2, 1, 4100, 4), (3, 2, 300, 8), (6, 4, 48, 4), (3, 2, 262, 4)])
def test_gate_skip_and_norm_of_wide_parts(ops, m, parts, width, heads, out, skip_type):
    """Rows that lie apart, on 16-byte boundaries or not; the gate before or behind the norm; no norm."""
    n = parts * width
    for off in (0, 1):
        wide = rnd(m, 2 * n + 8, seed=1, scale=1.5)
        o, gate = wide[:, off:off + n], wide[:, n + 4:2 * n + 4]
        skip = rnd(m, n + 8, seed=2).to(skip_type)[:, 4 * off:4 * off + n]
        for kw in (dict(groups=parts, gate_first=True, gain32=rnd(n, seed=3)), dict(groups=parts, gain32=rnd(width, seed=4)), dict(groups=0)):
            kw = dict(kw, eps=1e-5, gate32=gate, gate_kind="silu", skip32=skip, skip_coef32=rnd(heads, seed=5), out_scale=0.8)
            got, ref = torch.empty(m, n, dtype=out, device=DEV), torch.empty(m, n, dtype=torch.float64)
            ops.gated_norm(o, got, **kw)
            REF.gated_norm(o.cpu(), ref, **{k: cpu(v) for k, v in kw.items()})
            assert_close(got, ref, out, f"{off} {kw['groups']}")


@pytest.mark.parametrize("width,taps", [(12, 1), (48, 2), (64, 4), (130, 3), (40, 12)])
def test_convolution_stored_as_bfloat16_is_the_rounding_of_the_float_one(ops, width, taps):
    x, w, b = rnd(200, width, seed=1), rnd(width, taps, seed=2), rnd(width, seed=3)
    for q_lens in ([150, 1, 49], [1, 5, 16]):
        ctx, _, _ = batch(q_lens, [0] * 3)
        states, outs = [], []
        for dtype in DTYPES:
            state = rnd(3, max(1, (taps - 1) * width) + 3, seed=4)
            out = torch.empty(sum(q_lens), width, dtype=dtype, device=DEV)
            ops.conv_step(x[:sum(q_lens)], w, b, "silu", state, 1, ctx, out, taps)
            states.append(state)
            outs.append(out)
        assert torch.equal(outs[0].to(torch.bfloat16), outs[1]) and torch.equal(*states)


# ------------------------------------------------------------------------------------------ whole models through the engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(str(tmp_path_factory.mktemp("vag_" + name.lower())), cfg, seed)
            for name, cfg, seed in (("A", CFG_A, 11), ("B", CFG_B, 12), ("C", CFG_C, 13))}


def judge(folder, dtype):
    """32-bit: by the common tolerance, or by what 32-bit arithmetic alone does to this model. bfloat16: by a multiple of what rounding
    alone does to this model."""
    if dtype == "float32":
        return lambda got, ref, ids, what: assert_within_32_bit(folder, ids, got, ref, what)
    return lambda got, ref, ids, what: assert_within_rounding(got, ref, plain_logits(folder, ids, stored_as=torch.bfloat16)[:ref.shape[0]], what)


def gpu_engine(folder, dtype, page=4, pages=96, slots=4, graphs=True):
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine import Engine
    return Engine(folder, EngineConfig(dtype=dtype, page_size=page, num_pages=pages, max_batch=slots, cuda_graphs=graphs))


def run_cut(eng, name, ids, cuts):
    from nanoinfer_b200.engine import StepEntry
    rc = eng.open(name)
    out, pos = [], 0
    for n in cuts:
        out.append(eng.step([StepEntry(rc, ids[pos:pos + n], list(range(n)))]).clone())
        pos += n
    assert pos == len(ids)
    eng.close(rc)
    eng.check_device()
    return torch.cat(out)


def run_plan(eng, seqs, plan):
    """Steps of [(request, count)]; a request is closed behind its last token. Logits of every position of every request."""
    from nanoinfer_b200.engine import StepEntry
    got, at, live = {i: [] for i in range(len(seqs))}, {i: 0 for i in range(len(seqs))}, {}
    for step in plan:
        entries = []
        for r, c in step:
            if r not in live:
                live[r] = eng.open(f"r{r}")
            entries.append(StepEntry(live[r], seqs[r][at[r]:at[r] + c], list(range(c))))
        logits = eng.step(entries).clone()
        row = 0
        for r, c in step:
            got[r].append(logits[row:row + c])
            row += c
            at[r] += c
            if at[r] == len(seqs[r]):
                eng.close(live.pop(r))
        eng.cache.check()
    eng.check_device()
    return {r: torch.cat(x) for r, x in got.items()}


def vocab_of(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)["vocab"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,n,page", [("A", 45, 4), ("B", 141, 8), ("C", 300, 16)])
def test_engine_prompts_decoding_and_portions_equal_plain(folders, dtype, name, n, page):
    folder = folders[name]
    ids = tokens(n, vocab_of(folder), 5)
    ref = plain_logits(folder, ids)
    eng = gpu_engine(folder, dtype, page=page, pages=160)
    close = judge(folder, dtype)
    whole = run_cut(eng, "whole", ids, [n])
    close(whole, ref, ids, "whole prompt")
    tail = 40 if n > 100 else n - 1
    close(run_cut(eng, "decode", ids, [n - tail] + [1] * tail), ref, ids, "prompt, then token by token")
    cuts = [2, 7, 2, 13, 1, 1, 5, 2]
    cuts = cuts + [n - sum(cuts) - 2, 2]
    got = run_cut(eng, "cut", ids, cuts)
    close(got, ref, ids, "portions")
    if dtype == "float32":      # a cut moves a position by rounding only
        assert (got - whole).abs().max().item() <= 2e-5 * max(1.0, ref.abs().max().item())
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_engine_unequal_requests_and_reused_slots_and_pages(folders, dtype):
    folder = folders["A" if dtype == "float32" else "B"]       # (A's small heads move too far by bfloat16 rounding alone)
    eng = gpu_engine(folder, dtype, page=4, pages=14, slots=2)
    seqs = [tokens(n, 77, s) for n, s in ((23, 1), (9, 2), (17, 3), (12, 4))]
    plan = [[(0, 6), (1, 2)], [(0, 1), (1, 5)], [(0, 7), (1, 2)], [(0, 1), (2, 9)], [(2, 1), (0, 1)], [(0, 7), (2, 7)], [(3, 3)], [(3, 1)], [(3, 8)]]
    for r, got in run_plan(eng, seqs, plan).items():
        judge(folder, dtype)(got, plain_logits(folder, seqs[r]), seqs[r], f"request {r}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_mixed_schedule_with_heads_of_64_and_128(folders, dtype):
    lens = [211, 97, 160, 75, 130]
    seqs = [tokens(n, 300, 70 + i) for i, n in enumerate(lens)]
    eng = gpu_engine(folders["C"], dtype, page=16, pages=4 * (-(-max(lens) // 16) + 1) + 2, slots=4)
    for r, got in run_plan(eng, seqs, mixed_schedule(random.Random(5), lens)).items():
        judge(folders["C"], dtype)(got, plain_logits(folders["C"], seqs[r]), seqs[r], f"request {r}")


def test_long_decoding_through_captured_graphs(folders):
    """150 tokens one by one (two requests side by side, so the steps are replayed from a captured graph): windows and chunks are
    passed many times, the kept tokens' pages stay."""
    from nanoinfer_b200.engine import StepEntry
    eng = gpu_engine(folders["A"], "float32", page=4, pages=300, slots=2)
    seqs = [tokens(150, 131, 31), tokens(140, 131, 32)]
    rcs = [eng.open("a"), eng.open("b")]
    got = [[], []]
    for t in range(150):
        live = [i for i in range(2) if t < len(seqs[i])]
        logits = eng.step([StepEntry(rcs[i], [seqs[i][t]], [0]) for i in live]).clone()
        for j, i in enumerate(live):
            got[i].append(logits[j])
    assert eng.graph_launches > 0
    for i in range(2):
        assert_within_32_bit(folders["A"], seqs[i], torch.stack(got[i]), plain_logits(folders["A"], seqs[i]), f"request {i}")


def test_prompt_portions_replayed_from_a_captured_graph(folders):
    """Portions of one shape, often enough that they are replayed, on requests whose states differ; in bfloat16 the chunks."""
    for dtype in ("float32", "bfloat16"):
        eng = gpu_engine(folders["C"], dtype, page=16, pages=100, slots=2)
        eng._portion_graphs.min_tokens, eng._portion_graphs.sightings = 16, 2
        for seed in (1, 2):
            ids = tokens(256, 300, seed)
            judge(folders["C"], dtype)(run_cut(eng, "p", ids, [32] * 8), plain_logits(folders["C"], ids), ids, dtype)
        assert eng._portion_graphs.captured


def test_greedy_generation_through_the_scheduler(folders):
    from nanoinfer_b200.api import Model
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine.scheduler import Request, Scheduler
    m = Model(folders["B"], EngineConfig(dtype="float32", page_size=8, num_pages=64, max_batch=3, max_tokens_per_step=8))
    sched = Scheduler(m)
    prompts = [tokens(13, 77, 21), tokens(5, 77, 22), tokens(29, 77, 23), tokens(3, 77, 24)]
    for i, p in enumerate(prompts):
        sched.add(Request(f"g{i}", p, max_tokens=8))
    done = sched.run()
    for i, p in enumerate(prompts):
        ids = list(p)
        for _ in range(8):
            row = plain_logits(folders["B"], ids)[-1]
            top = row.topk(2).values
            assert top[0] - top[1] > 1e-3, "the test's model has a tie here; pick another seed"
            ids.append(int(row.argmax()))
        assert done[f"g{i}"] == ids[len(p):], i
    m.engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["kept", "lightning", "steps"])
def test_the_first_token_reaches_the_last_and_only_through_its_memory(tmp_path, kind, dtype):
    """Changing the FIRST token of a 300-token prompt moves the last position's logits through a kept token, a slow fixed decay or
    small steps, decoded and in portions, although windows and chunks ended long ago; without that memory it must not."""
    def fast(t):
        for name in t:
            if name.endswith("dt_bias"):
                t[name].fill_(9.0)
            if name.endswith("A_log"):
                t[name].fill_(4.0)

    def slow(t):
        for name in t:
            if name.endswith("dt_bias"):
                t[name].fill_(-6.0)
            if name.endswith("A_log"):
                t[name].fill_(-2.0)
            if name.endswith(".in"):
                t[name].mul_(0.5)
    half = lambda keep: softmax(2, 1, 16, 20, 8, keep_first=keep)
    layers = {"kept": lambda on: [pair(half(2 if on else 0), lightning(1, 4, 4, [0.0]), ff=32)],
              "lightning": lambda on: [pair(half(0), lightning(2, 32, 16, [0.999, 0.998] if on else [0.5, 0.0]), ff=32)],
              "steps": lambda on: [chunked(2, 1, 16, 9, 8, ff=32), ssm(2, 16, 32, 1, 2, 2)]}[kind]
    ids = tokens(300, 64, 3)
    other = [(ids[0] + 1) % 64] + ids[1:]
    for on in (True, False):
        d = write_model(str(tmp_path / str(on)), model(64, 48, layers(on)), 5, weights=(slow if on else fast) if kind == "steps" else None)
        eng = gpu_engine(d, dtype, page=16, pages=64, slots=2)
        refs = []
        for seq in (ids, other):
            ref = plain_logits(d, seq)
            judge(d, dtype)(run_cut(eng, "x", seq, [70, 2, 180] + [1] * 48), ref, seq, kind)
            refs.append(ref)
        moved = (refs[0][-1] - refs[1][-1]).abs().max().item()
        assert moved > 1e-3 if on else moved < 1e-6, (on, moved)


@pytest.mark.parametrize("seed,dtype", [(900 + i, "float32") for i in range(10)] + [(900 + i, "bfloat16") for i in range(6)])
def test_random_configurations(seed, dtype, tmp_path):
    """Layer orders, sizes and constants drawn at random (one head, one channel, a window of 1, kept tokens beyond the window, one
    tap): a prompt in portions with a decoded tail beside a second request."""
    rng = random.Random(seed)
    cfg = random_config(rng)
    d = write_model(str(tmp_path), cfg, seed)
    seqs = [tokens(70, cfg["vocab"], seed), tokens(33, cfg["vocab"], seed + 1)]
    plan, left = [], 33
    for c in [17, 2, 1, 30, 3, 11] + [1] * 6:
        m = min(left, max(1, c // 2))
        plan.append(([(1, m)] if m else []) + [(0, c)])
        left -= m
    seqs[1] = seqs[1][:33 - left]
    eng = gpu_engine(d, dtype, page=rng.choice([4, 16]), pages=400, slots=2)
    for r, got in run_plan(eng, seqs, plan).items():
        judge(d, dtype)(got, plain_logits(d, seqs[r]), seqs[r], f"request {r}")


@pytest.mark.parametrize("seed,dtype", [(21, "float32"), (21, "bfloat16"), (34, "float32"), (34, "bfloat16"), (48, "bfloat16"), (55, "bfloat16")])
def test_larger_configurations_under_a_mixed_schedule(seed, dtype, tmp_path):
    """Six requests of 60 to 230 tokens, at most four live: portions of 2 to 100 tokens beside single tokens, requests left out of
    a step, slots and pages given back and used again; sizes of a small real model."""
    rng = random.Random(seed)
    cfg = random_config(rng, small=False)
    lens = [rng.randint(60, 230) for _ in range(6)]
    seqs = [tokens(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate(lens)]
    plan = mixed_schedule(rng, lens)
    page = rng.choice([16, 64])
    d = write_model(str(tmp_path), cfg, seed)
    eng = gpu_engine(d, dtype, page=page, pages=4 * (-(-max(lens) // page) + 1) + 2, slots=4)
    for r, got in run_plan(eng, seqs, plan).items():
        judge(d, dtype)(got, plain_logits(d, seqs[r]), seqs[r], f"request {r}")


def test_trace_replay_as_a_child_process(folders, tmp_path):
    """``bin/trace_run`` as a child process on a model of this design."""
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ids = tokens(40, 77, 9)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:21], "want": [10]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[21:], "want": [0, 18]}], "end": ["a"]}]
    rows = [10, 21, 39]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["B"], "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [line for line in r.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
        got = torch.cat([torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(n, -1)) for i, n in ((0, 1), (1, 2))])
        if dtype == "float32":
            assert_close(got, plain_logits(folders["B"], ids)[rows], torch.float32)
        else:
            assert_within_rounding(got, plain_logits(folders["B"], ids)[rows], plain_logits(folders["B"], ids, stored_as=torch.bfloat16)[rows])


def test_command_line_tools_generate_and_serve(folders):
    """bin/generate (with the cache and recomputing every token) and bin/serve as child processes, in 32-bit: the plain
    implementation's greedy tokens."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

    def tool(name, argv):
        done = subprocess.run([sys.executable, os.path.join(root, "bin", name)] + argv, capture_output=True, text=True, timeout=600)
        assert done.returncode == 0, done.stderr[-2000:]
        return [[int(t) for t in line.split("Completion: ", 1)[1].split()] for line in done.stdout.splitlines()
                if line.startswith("Completion: ")]

    def greedy(prompt, n):
        ids = list(prompt)
        for _ in range(n):
            ids.append(int(plain_logits(folders["B"], ids)[-1].argmax()))
        return ids[len(prompt):]

    prompts = [tokens(9, 77, 41), tokens(26, 77, 42)]
    common = ["--model-dir", folders["B"], "--dtype", "float32", "--block-size", "8", "--num-blocks", "64", "--max-tokens", "6"]
    for extra in ([], ["--no-cache"]):
        (got,) = tool("generate", common + ["--prompt", " ".join(map(str, prompts[0]))] + extra)
        assert got == greedy(prompts[0], 6), extra
    argv = common + ["--max-batch", "2", "--max-tokens-per-step", "16"]
    for p in prompts:
        argv += ["--prompt", " ".join(map(str, p))]
    assert tool("serve", argv) == [greedy(p, 6) for p in prompts]
