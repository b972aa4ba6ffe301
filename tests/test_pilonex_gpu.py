"""Pilonex on the GPU: every new kernel alone against its plain statement (tests/torch_ops.py, float64), with inputs made so that a
lost state, a swapped stream, a limit that does not cut or a key that is one token off shows; then the engine in both
precisions against the plain whole-sequence implementation: prompts, token-by-token decoding, portions down to two tokens,
unequal requests in one batch, slots and pages that are used again, long decoding through captured graphs, greedy generation
through the scheduler, the tools."""
import json
import os
import random

import pytest
import torch

from gpu_util import assert_close
from pilonex_util import (CFG_A, CFG_B, CFG_C, CFG_D, assert_within_32_bit, assert_within_rounding, dense, left, memory, mixed_schedule, model, moe, pair,
                          pin_routing, plain_logits, random_config, right, tokens, write_model)
from test_vafozen_gpu import _fill_pages, batch, rnd, to_cpu
from torch_ops import TorchOps

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


# ------------------------------------------------------------------------------------------ several streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,width", [(5, 2, 64), (70, 3, 100), (3, 1, 1024), (130, 4, 36), (2, 2, 2050), (9, 6, 52), (4, 16, 24), (8, 2, 1), (65, 2, 1280)])
def test_streams_between_sublayers(ops, dtype, m, n, width):
    """Three sublayers in a row: the first reads streams that all equal one tensor, the second and third take the result before
    them into the streams (out of the one tensor, then in place), and the last sum ends in one stream."""
    x = rnd(m, width, seed=1)
    factors = [{"in32": rnd(n, seed=10 + i), "gain32": rnd(width, seed=20 + i), "mix32": rnd(n, n, seed=30 + i), "out32": rnd(n, seed=40 + i)} for i in range(3)]
    host = [{k: v.cpu() for k, v in f.items()} for f in factors]
    h, rh = torch.empty(m, width, dtype=dtype, device=DEV), torch.empty(m, width, dtype=torch.float64)
    buf, rbuf = torch.empty(m, n, width, device=DEV), torch.empty(m, n, width)
    ops.stream_mix(x, n, in32=factors[0]["in32"], gain32=factors[0]["gain32"], eps=1e-5, h_out=h)
    REF.stream_mix(x.cpu(), n, in32=host[0]["in32"], gain32=host[0]["gain32"], eps=1e-5, h_out=rh)
    assert_close(h, rh, dtype, "first")
    cur, rcur = x, x.cpu()
    for i in (1, 2):
        y = rnd(m, width, seed=50 + i)
        ry = y.cpu().clone()
        ops.stream_mix(cur, n, y32=y, mix32=factors[i - 1]["mix32"], out32=factors[i - 1]["out32"], dst32=buf, in32=factors[i]["in32"],
                       gain32=factors[i]["gain32"], eps=1e-5, h_out=h, clear=True)
        REF.stream_mix(rcur, n, y32=ry, mix32=host[i - 1]["mix32"], out32=host[i - 1]["out32"], dst32=rbuf, in32=host[i]["in32"],
                       gain32=host[i]["gain32"], eps=1e-5, h_out=rh, clear=True)
        assert_close(buf, rbuf, torch.float32, f"streams {i}")
        assert_close(h, rh, dtype, f"normed {i}")
        assert (y == 0).all()
        cur, rcur = buf, rbuf
    y = rnd(m, width, seed=60)
    total, rtotal = torch.empty(m, width, device=DEV), torch.empty(m, width)
    ops.stream_mix(cur, n, y32=y, mix32=factors[2]["mix32"], out32=factors[2]["out32"], sum_out32=total)
    REF.stream_mix(rcur, n, y32=y.cpu(), mix32=host[2]["mix32"], out32=host[2]["out32"], sum_out32=rtotal)
    assert_close(total, rtotal, torch.float32, "sum")


# ------------------------------------------------------------------------------------------ the gated form with limits
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,inter,k", [(1, 24, 40), (3, 72, 96), (7, 200, 128), (12, 130, 256), (30, 96, 64), (50, 300, 320), (90, 136, 200), (200, 256, 128), (300, 264, 192), (520, 384, 256)])
def test_gated_product_cuts_where_it_should(ops, dtype, m, inter, k):
    """Sums far beyond the limit on every side (the gate has none below); every product kernel that the sizes reach."""
    a, w = rnd(m, k, seed=1).to(dtype), rnd(2 * inter, k, seed=2, scale=3.0 / k ** 0.5).to(dtype)
    for glu in ((1.702, 1.25, 1.0), (1.0, 0.4, 0.0), (0.7, 100.0, -0.5)):
        out = torch.empty(m, inter, dtype=dtype, device=DEV)
        ops.linear_swiglu(a, w, out, glu)
        ref = torch.empty(m, inter, dtype=torch.float64)
        REF.linear_swiglu(a.cpu(), w.cpu(), ref, glu)
        assert_close(out, ref, dtype, f"{glu}")
    for route in ("smallm", "tc", "tc_pair") if dtype == torch.bfloat16 and k % 32 == 0 else ():
        if route == "smallm" and m > 64:
            continue
        out = torch.empty(m, inter, dtype=dtype, device=DEV)
        ops.with_options(gemm_route=route).linear_swiglu(a, w, out, (1.702, 1.25, 1.0))
        ref = torch.empty(m, inter, dtype=torch.float64)
        REF.linear_swiglu(a.cpu(), w.cpu(), ref, (1.702, 1.25, 1.0))
        assert_close(out, ref, dtype, route)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,hidden,ff,experts,top", [(5, 64, 24, 4, 2), (3, 40, 18, 3, 3), (140, 128, 136, 5, 2), (600, 64, 64, 2, 1), (8, 72, 40, 9, 3)])
def test_experts_with_limits_and_softmax_over_the_chosen(ops, dtype, m, hidden, ff, experts, top):
    h = rnd(m, hidden, seed=1).to(dtype)
    w1 = rnd(experts, 2 * ff, hidden, seed=2, scale=2.0 / hidden ** 0.5).to(dtype)
    w2 = rnd(experts, hidden, ff, seed=3, scale=1.0 / ff ** 0.5).to(dtype)
    z = rnd(m, experts, seed=4, scale=2.0)
    e, wt = torch.empty(m, top, dtype=torch.int32, device=DEV), torch.empty(m, top, device=DEV)
    ops.moe_route(z.clone(), top, e, wt, score="softmax", renormalize=True)
    order = torch.sort(z.cpu().double(), dim=-1, descending=True).indices[:, :top]
    assert (e.cpu().long() == order).all()
    assert_close(wt, torch.softmax(torch.gather(z.cpu().double(), 1, order), -1), torch.float32, "weights")
    out = rnd(m, hidden, seed=5)
    ref = out.cpu().double()
    ops.moe_experts(h, e, wt, w1, w2, out, weight_on="output", glu=(1.702, 0.9, 1.0))
    REF.moe_experts(h.cpu(), e.cpu(), wt.cpu(), w1.cpu(), w2.cpu(), ref, weight_on="output", glu=(1.702, 0.9, 1.0))
    assert_close(out, ref, dtype, "experts")


# ------------------------------------------------------------------------------------------ gates of the matrix memory
@pytest.mark.parametrize("heads,cap", [(1, 4.0), (3, 12.0), (8, 15.0)])
def test_gates_keep_a_running_maximum_across_steps(ops, heads, cap):
    """Unequal requests in three steps (one longer than a block of 1,024 threads), a slot handed on zeroed; gates that pull the
    maximum up, let it decay for hundreds of tokens, and start below zero."""
    off = 3
    state = torch.zeros(4, off + heads + 2, device=DEV)
    state[:, :off], state[:, off + heads:] = 5.0, -5.0
    rstate = state.cpu().clone()
    bi, bf = rnd(heads, seed=1), rnd(heads, seed=2) + 3.0
    for step, (q_lens, slots) in enumerate([([2300, 1, 40], [2, 0, 1]), ([1, 1, 33], [2, 0, 1]), ([700, 5], [3, 2])]):
        m = sum(q_lens)
        ctx, _, _ = batch(q_lens, [0] * len(q_lens), slots=slots)
        wide = rnd(m, 2 * heads + 3, seed=10 + step, scale=4.0)
        wide[:, 1:1 + heads] -= 6.0
        wide[::97, 1:1 + heads] += 14.0
        zi, zf = wide[:, 1:1 + heads], wide[:, 2 + heads:2 + 2 * heads]
        got, ref = torch.empty(3, m, heads, device=DEV), torch.empty(3, m, heads)
        ops.memory_gates(zi, zf, bi, bf, cap, state, off, ctx, *got.unbind(0))
        REF.memory_gates(zi.cpu(), zf.cpu(), bi.cpu(), bf.cpu(), cap, rstate, off, to_cpu(ctx), *ref.unbind(0))
        assert torch.allclose(state.cpu(), rstate, rtol=0, atol=3e-5), step
        for i, what in enumerate(("decay", "write", "floor")):
            assert torch.allclose(got[i].cpu(), ref[i], rtol=4e-5, atol=1e-9), (step, what, (got[i].cpu() - ref[i]).abs().max())
    assert (state[:, :off] == 5.0).all() and (state[:, off + heads:] == -5.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,heads,d", [(5, 3, 20), (3, 2, 300), (40, 1, 7), (9, 4, 64), (33, 2, 128), (7, 5, 16), (6, 3, 256), (5, 1, 32)])
def test_norm_of_a_part_behind_its_divisor(ops, dtype, m, heads, d):
    """A part's number behind the channels divides it (its size, or the floor where that is larger, plus a small constant)."""
    o, gate = rnd(m, heads * (d + 1), seed=1), rnd(m, heads * d, seed=2)
    o[:, heads * d] = 1e-7
    floor = torch.rand(m, heads, generator=torch.Generator().manual_seed(3)).to(DEV) * 1.5
    kw = dict(groups=heads, eps=1e-5, gain32=rnd(heads * d, seed=4), gate32=gate, gate_kind="sigmoid", out_scale=0.7, floor32=floor, den_eps=1e-6)
    out, ref = torch.empty(m, heads * d, dtype=dtype, device=DEV), torch.empty(m, heads * d, dtype=torch.float64)
    ops.gated_norm(o, out, **kw)
    REF.gated_norm(o.cpu(), ref, **{k: cpu(v) for k, v in kw.items()})
    assert_close(out, ref, dtype)


# ------------------------------------------------------------------------------------------ walks, eight tokens at a time
def walk_inputs(m, heads, kq, dk, dv, seed, kind):
    g = {"q32": rnd(m, kq * dk, seed=seed), "k32": rnd(m, kq * dk, seed=seed + 1), "v32": rnd(m, heads * dv, seed=seed + 2)}
    if kind == "delta":             # step sizes per channel, beta, unit vectors
        kw = {"z32": rnd(m, heads * dk, seed=seed + 3), "beta32": rnd(m, heads, seed=seed + 4, scale=2.0)}
    elif kind == "delta_decays":    # decays as they are
        kw = {"z32": torch.sigmoid(rnd(m, heads * dk, seed=seed + 3) + 2.0), "beta32": rnd(m, heads, seed=seed + 4)}
    elif kind == "channel":
        kw = {"z32": torch.sigmoid(rnd(m, heads * dk, seed=seed + 3) + 2.0)}
    else:                           # one decay per head, a factor on the keys, a column of ones
        kw = {"z32": torch.sigmoid(rnd(m, heads, seed=seed + 3) + 2.0), "k_scale32": torch.rand(m, heads, generator=torch.Generator().manual_seed(seed)).to(DEV)}
    g.update(kw)
    return g


def walk_constants(heads, dk, kind):
    kw = {"q_scale": dk ** -0.5}
    if kind == "delta":
        kw.update(rate32=torch.exp(rnd(heads, seed=70)), dt_bias32=rnd(heads * dk, seed=71) - 3.0)
    if kind.startswith("delta"):
        kw.update(unit_eps=1e-6)
    if kind == "head":
        kw.update(ones=True)
    return kw


def run_walk(k, g, rows, state, off, ctx, heads, kq, dk, dv, const, dev=DEV):
    """``rows``: which rows of the inputs the step brings."""
    pick = {n: (t[rows].contiguous() if dev == DEV else t[rows].cpu().contiguous()) for n, t in g.items()}
    const = const if dev == DEV else {n: cpu(t) for n, t in const.items()}
    out = torch.empty(len(rows), heads * (dv + (1 if const.get("ones") else 0)), device=dev)
    k.grouped_state_scan(pick.pop("q32"), pick.pop("k32"), pick.pop("v32"), pick.pop("z32"), state, off, ctx, out, heads, kq, dk, dv, **pick, **const)
    return out


WALKS = [(1, 1, 8, 5), (3, 3, 20, 12), (4, 2, 48, 40), (2, 2, 64, 64), (6, 2, 33, 7), (2, 1, 100, 33), (1, 1, 130, 70), (6, 3, 1, 8), (2, 2, 256, 9), (1, 1, 32, 1)]


@pytest.mark.parametrize("heads,kq,dk,dv", WALKS)
@pytest.mark.parametrize("kind", ["delta", "delta_decays", "channel", "head"])
def test_walk_against_plain_and_cut_anywhere(ops, heads, kq, dk, dv, kind):
    """Whole, then in portions (two tokens, one token, across the groups of eight) beside another request's rows; the state sits
    behind other columns of a wider state row."""
    n, off = 61, 11
    const = walk_constants(heads, dk, kind)
    size = heads * (dv + (1 if const.get("ones") else 0)) * dk
    g = walk_inputs(n + 40, heads, kq, dk, dv, 1, kind)
    state, rstate = torch.zeros(3, off + size + 4, device=DEV), torch.zeros(3, off + size + 4)
    ctx, _, _ = batch([n], [0], slots=[1])
    whole = run_walk(ops, g, list(range(n)), state, off, ctx, heads, kq, dk, dv, const)
    ref = run_walk(REF, g, list(range(n)), rstate, off, to_cpu(ctx), heads, kq, dk, dv, const, "cpu")
    assert_close(whole, ref, torch.float32, "whole")
    assert_close(state, rstate, torch.float32, "state")
    assert (state[[0, 2]] == 0).all() and (state[1, :off] == 0).all() and (state[1, off + size:] == 0).all()
    state2 = torch.zeros(3, off + size + 4, device=DEV)
    got, pos, opos = [], 0, n
    for c in [2, 1, 9, 17, 1, 2, 8, 5, 16]:
        oc = min(3, n + 40 - opos)
        ctx, _, _ = batch([oc, c], [0, 0], slots=[2, 0])
        out = run_walk(ops, g, list(range(opos, opos + oc)) + list(range(pos, pos + c)), state2, off, ctx, heads, kq, dk, dv, const)
        got.append(out[oc:])
        pos, opos = pos + c, opos + oc
    assert pos == n
    assert_close(torch.cat(got), ref, torch.float32, "in portions")
    assert_close(state2[0], rstate[1], torch.float32, "state after portions")
    ops.check_device_errors()


@pytest.mark.parametrize("heads,kq,dk,dv", [(4, 2, 64, 64), (2, 2, 20, 33), (3, 1, 129, 6), (1, 1, 1, 1)])
@pytest.mark.parametrize("kind", ["delta", "delta_decays", "channel", "head"])
def test_short_steps_go_on_where_long_ones_stopped(ops, heads, kq, dk, dv, kind):
    """A portion of 30 tokens, then steps of one to four tokens (one launch each), then one of 12, beside a request that is at
    another place; slots that no request owns stay as they are."""
    off = 3
    const = walk_constants(heads, dk, kind)
    size = heads * (dv + (1 if const.get("ones") else 0)) * dk
    cuts = [30, 1, 1, 4, 1, 3, 2, 1, 12, 1]
    n = sum(cuts)
    g = walk_inputs(2 * n, heads, kq, dk, dv, 5, kind)
    state = rnd(4, off + size + 1, seed=4, scale=0.3)
    rstate = state.cpu().clone()
    ctx, _, _ = batch([n, n], [0, 0], slots=[3, 1])
    ref = run_walk(REF, g, list(range(2 * n)), rstate, off, to_cpu(ctx), heads, kq, dk, dv, const, "cpu")
    got, pos, launches = ([], []), 0, []
    for c in cuts:
        ctx, _, _ = batch([c, c], [0, 0], slots=[3, 1])
        before = ops.launches
        out = run_walk(ops, g, list(range(pos, pos + c)) + list(range(n + pos, n + pos + c)), state, off, ctx, heads, kq, dk, dv, const)
        launches.append(ops.launches - before)
        got[0].append(out[:c])
        got[1].append(out[c:])
        pos += c
    assert launches == [1 if c <= 4 else 2 for c in cuts]
    assert_close(torch.cat(got[0] + got[1]), ref, torch.float32, "outputs")
    assert_close(state, rstate, torch.float32, "states")
    ops.check_device_errors()


@pytest.mark.parametrize("kind,heads,kq,dk,dv", [("delta", 4, 2, 64, 48), ("head", 3, 3, 64, 70), ("delta", 2, 2, 128, 128), ("channel", 1, 1, 40, 8)])
def test_unequal_requests_a_long_prompt_and_states_that_go_on(ops, kind, heads, kq, dk, dv):
    q_lens, slots, off = [700, 3, 1, 8, 64], [2, 0, 1, 4, 3], 7
    const = walk_constants(heads, dk, kind)
    size = heads * (dv + (1 if const.get("ones") else 0)) * dk
    g = walk_inputs(sum(q_lens), heads, kq, dk, dv, 3, kind)
    ctx, _, _ = batch(q_lens, [0] * 5, slots=slots)
    state = rnd(5, off + size + 2, seed=9, scale=0.3)          # the requests do not start from zero
    rstate = state.cpu().clone()
    for step in range(2):
        out = run_walk(ops, g, list(range(sum(q_lens))), state, off, ctx, heads, kq, dk, dv, const)
        ref = run_walk(REF, g, list(range(sum(q_lens))), rstate, off, to_cpu(ctx), heads, kq, dk, dv, const, "cpu")
        assert_close(out, ref, torch.float32, f"step {step}")
        assert_close(state, rstate, torch.float32, f"state {step}")


def test_strong_decays_underflow_to_zero_and_weak_ones_last(ops):
    """Channels whose decay is zero, tiny, one, and close to one over 3,000 tokens: nothing turns into NaN, and the slow
    channel stays within rounding of a 64-bit recurrence."""
    n, dk, dv = 3000, 8, 4
    z = torch.zeros(n, dk, device=DEV)
    z[:, 0], z[:, 1], z[:, 2], z[:, 3] = 80.0, 12.0, -200.0, -7.5
    z[:, 4:] = rnd(n, 4, seed=5)
    g = {"q32": rnd(n, dk, seed=1), "k32": rnd(n, dk, seed=2), "v32": rnd(n, dv, seed=3), "z32": z, "beta32": rnd(n, 1, seed=4) - 1.0}
    const = dict(rate32=torch.tensor([1.5], device=DEV), dt_bias32=torch.zeros(dk, device=DEV), unit_eps=1e-6)
    state, rstate = torch.zeros(1, dk * dv, device=DEV), torch.zeros(1, dk * dv)
    ctx, _, _ = batch([n], [0])
    out = run_walk(ops, g, list(range(n)), state, 0, ctx, 1, 1, dk, dv, const)
    ref = run_walk(REF, g, list(range(n)), rstate, 0, to_cpu(ctx), 1, 1, dk, dv, const, "cpu")
    assert_close(out, ref, torch.float32)
    assert_close(state, rstate, torch.float32, "state")


@pytest.mark.parametrize("where", [13, 16, 23])
def test_delta_walk_remembers_a_far_key_and_overwrites_it(ops, where):
    """One token writes a value under a key of its own; 600 tokens later a query finds it, scaled by the decays in between. A
    second write under the same key with beta = 1 replaces the value, where a sum would give both."""
    n, dk, dv = 640, 16, 8
    q, k, v = torch.zeros(n, dk, device=DEV), rnd(n, dk, seed=1, scale=0.3), rnd(n, dv, seed=2)
    k[:, 3] = 0.0
    k[where] = 0.0
    k[where, 3] = 1.0
    q[630, 3] = 1.0
    const = dict(unit_eps=0.0)
    g = {"q32": q, "k32": k, "v32": v, "z32": torch.full((n, dk), 0.999, device=DEV), "beta32": torch.full((n, 1), 30.0, device=DEV)}
    q[q.abs().sum(-1) == 0, 5] = 1.0            # (unit vectors need a length)
    ctx, _, _ = batch([n], [0])
    out = run_walk(ops, g, list(range(n)), torch.zeros(1, dk * dv, device=DEV), 0, ctx, 1, 1, dk, dv, const)
    want = v[where].double() * 0.999 ** (630 - where)
    assert (out[630].double() - want).abs().max().item() <= 2e-5 * want.abs().max().item() + 1e-7
    k[where + 3] = 0.0
    k[where + 3, 3] = 1.0
    out = run_walk(ops, g, list(range(n)), torch.zeros(1, dk * dv, device=DEV), 0, ctx, 1, 1, dk, dv, const)
    want = v[where + 3].double() * 0.999 ** (630 - where - 3)
    assert (out[630].double() - want).abs().max().item() <= 2e-5 * want.abs().max().item() + 1e-7


# ------------------------------------------------------------------------------------------ the softmax half
@pytest.mark.parametrize("dim,heads,kv", [(64, 4, 2), (128, 2, 1)])
def test_prompt_attention_on_tensor_memory_carries_the_output_factor(ops, dim, heads, kv):
    q_lens, before, page = [150, 90], [20, 0], 16
    full_ctx, full_bt, num_pages = batch([b + q for b, q in zip(before, q_lens)], [0, 0], page_size=page)
    ctx, _, _ = batch(q_lens, before, page_size=page)
    qkv = rnd(sum(q_lens) + sum(before), (heads + 2 * kv) * dim, seed=3, scale=0.7)
    q_all, kp, vp = _fill_pages(ops, torch.bfloat16, full_ctx, full_bt, page, num_pages, heads, kv, dim, dim, qkv)
    rows = torch.cat([torch.arange(s + b, s + b + q) for s, b, q in zip(full_ctx.q_start.cpu().tolist(), before, q_lens)]).to(DEV)
    q = q_all[rows].contiguous()
    outs = []
    for k in (ops, ops.with_options(force_mma_prefill=True)):
        out = torch.empty(sum(q_lens), heads * dim, dtype=torch.bfloat16, device=DEV)
        k.attention_flex(q, out, heads, kv, dim, dim, 0.2, 0.0, None, 70, 0, 1.7, ctx, full_bt, page, kp, vp)
        outs.append(out)
    ref = torch.empty(sum(q_lens), heads * dim, dtype=torch.float64)
    REF.attention_flex(q.cpu(), ref, heads, kv, dim, dim, 0.2, 0.0, None, 70, 0, 1.7, to_cpu(ctx), full_bt.cpu(), page, kp.cpu(), vp.cpu())
    for out, what in zip(outs, ("tensor memory", "mma.sync")):
        assert_close(out, ref, torch.bfloat16, what)
    ops.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window,page", [(1, 4), (2, 16), (33, 8), (64, 16), (70, 16), (128, 16), (257, 16)])
def test_a_key_just_inside_the_window_is_seen_and_the_one_before_is_not(ops, window, page, decode, dtype):
    """Values narrower than keys. Two marked keys next to each other stand out: the first that the query's window holds and the
    last that it does not; the query must return the former's value alone, one position on neither's mark of the latter."""
    dk, dv, n = 64, 32, 3 * window + 9
    p = n - 2
    inside, outside = p - window + 1, p - window
    qkv = torch.zeros(n, 2 * dk + dv, device=DEV)
    qkv[:, dk] = 1.0
    for pos, mark in ((inside, 1.0), (outside, 2.0)):
        qkv[pos, dk + 1] = 9.0
        qkv[pos, 2 * dk:] = mark
    qkv[:, 1] = 9.0
    full_ctx, bt, num_pages = batch([n], [0], page_size=page)
    q_all, kp, vp = _fill_pages(ops, dtype, full_ctx, bt, page, num_pages, 1, 1, dk, dv, qkv)
    for pos, want in ((p - 1, 2.0 if window > 1 else None), (p, 1.0), (p + 1, 0.0)):
        first = pos if decode else max(0, pos - 5)
        ctx, _, _ = batch([pos + 1 - first], [first], page_size=page)
        out = torch.empty(pos + 1 - first, dv, device=DEV)
        ops.attention_flex(q_all[first:pos + 1].contiguous(), out, 1, 1, dk, dv, 1.0, 0.0, None, window, 0, 1.0, ctx, bt, page, kp, vp)
        got = out[-1, 0].item()
        if pos == p:
            assert abs(got - 1.0) < 1e-3, (pos, got)
        elif pos == p - 1 and want is not None:     # both marked keys are visible with equal scores
            assert abs(got - 1.5) < 1e-2, (pos, got)
        elif pos == p + 1:
            assert abs(got) < 1e-3, (pos, got)


# ------------------------------------------------------------------------------------------ whole models through the engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Four models, each twice: with random routers (the 32-bit tests) and, under ``<name>/pinned``, with a routing that
    rounding cannot change (the bfloat16 tests)."""
    out = {}
    for name, cfg, seed in (("A", CFG_A, 11), ("B", CFG_B, 12), ("C", CFG_C, 13), ("D", CFG_D, 14)):
        out[name] = write_model(str(tmp_path_factory.mktemp("pil_" + name.lower())), cfg, seed, strip_ranks=True)
        out[name + "/pinned"] = write_model(str(tmp_path_factory.mktemp("pil_pin_" + name.lower())), cfg, seed, weights=pin_routing(cfg))
    return out


def folder_for(folders, name, dtype):
    return folders[name if dtype == "float32" else name + "/pinned"]


def judge(folder, dtype):
    """32-bit: by the common tolerance, or by what 32-bit arithmetic alone does to this model. bfloat16: by a multiple of what rounding alone does to this model."""
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
@pytest.mark.parametrize("name,n,page", [("A", 45, 4), ("B", 141, 8), ("C", 300, 16), ("D", 330, 16)])
def test_engine_prompts_decoding_and_portions_equal_plain(folders, dtype, name, n, page):
    folder = folder_for(folders, name, dtype)
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
    folder = folder_for(folders, "A", dtype)
    eng = gpu_engine(folder, dtype, page=4, pages=34, slots=2)
    seqs = [tokens(n, 131, s) for n, s in ((23, 1), (9, 2), (17, 3), (12, 4))]
    plan = [[(0, 6), (1, 2)], [(0, 1), (1, 5)], [(0, 7), (1, 2)], [(0, 1), (2, 9)], [(2, 1), (0, 1)], [(0, 7), (2, 7)], [(3, 3)], [(3, 1)], [(3, 8)]]
    for r, got in run_plan(eng, seqs, plan).items():
        judge(folder, dtype)(got, plain_logits(folder, seqs[r]), seqs[r], f"request {r}")


def test_long_decoding_through_captured_graphs(folders):
    """150 tokens one by one (two requests side by side, so the steps are replayed from a captured graph), every pass of the
    looped layers with a state of its own; windows are passed many times."""
    from nanoinfer_b200.engine import StepEntry
    eng = gpu_engine(folders["A"], "float32", page=4, pages=300, slots=2)
    seqs = [tokens(150, 131, 31), tokens(140, 131, 32)]
    rcs = [eng.open("a"), eng.open("b")]
    got = [[], []]
    for t in range(150):
        entries = [StepEntry(rcs[i], [seqs[i][t]], [0]) for i in range(2) if t < len(seqs[i])]
        logits = eng.step(entries).clone()
        for j, i in enumerate(i for i in range(2) if t < len(seqs[i])):
            got[i].append(logits[j])
    assert eng.graph_launches > 0
    for i in range(2):
        assert_within_32_bit(folders["A"], seqs[i], torch.stack(got[i]), plain_logits(folders["A"], seqs[i]), f"request {i}")


def test_prompt_portions_replayed_from_a_captured_graph(folders):
    """Portions of one shape, often enough that they are replayed, on requests whose states differ."""
    eng = gpu_engine(folders["C"], "float32", page=16, pages=100, slots=2)
    eng._portion_graphs.min_tokens, eng._portion_graphs.sightings = 16, 2
    for seed in (1, 2):
        ids = tokens(256, 300, seed)
        assert_close(run_cut(eng, "p", ids, [32] * 8), plain_logits(folders["C"], ids), torch.float32)
    assert eng._portion_graphs.captured


def test_greedy_generation_through_the_scheduler(folders):
    from nanoinfer_b200.api import Model
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine.scheduler import Request, Scheduler
    m = Model(folders["B"], EngineConfig(dtype="float32", page_size=8, num_pages=64, max_batch=3, max_tokens_per_step=8))
    sched = Scheduler(m)
    prompts = [tokens(13, 77, 21), tokens(5, 77, 22), tokens(19, 77, 23), tokens(3, 77, 24)]
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


@pytest.mark.parametrize("kind", ["delta", "memory"])
def test_the_first_token_reaches_the_logits_through_a_state_and_not_through_a_window(tmp_path, kind):
    """Changing the FIRST token of a 300-token prompt moves the last position's logits through a slowly decaying state, decoded
    and in portions, although every window ended long ago; without such a state (one tap, decays of zero) it must not."""
    def slow(t):
        for name in t:
            if name.endswith("A_log"):
                t[name].fill_(-9.0)
            if name.endswith(".b") and t[name].dim() == 2:
                t[name].mul_(0.1)               # beta near one half
            if name.endswith(".f.b"):
                t[name].fill_(9.0)

    def none(t):
        for name in t:
            if name.endswith("A_log"):
                t[name].fill_(9.0)
            if name.endswith(".dt_bias"):
                t[name].fill_(9.0)
            if name.endswith(".f.b"):
                t[name].fill_(-300.0)
    lt, rt = left(2, 1, 16, 8, 20, 8), right(2, 1, 64, 8, 1)
    layer = pair(lt, rt, mlp=None) if kind == "delta" else memory(2, 64, 8, 12.0, mlp=dense(16))
    cfg = model(64, 48, [pair(lt, right(1, 1, 2, 2, 1), 1.0, 0.0, mlp=dense(32)), layer])
    ids = tokens(300, 64, 3)
    other = [(ids[0] + 1) % 64] + ids[1:]
    for name, change in (("slow", slow), ("none", none)):
        d = write_model(str(tmp_path / name), cfg, 5, weights=change)
        eng = gpu_engine(d, "float32", page=16, pages=64, slots=2)
        refs = []
        for seq in (ids, other):
            ref = plain_logits(d, seq)
            assert_close(run_cut(eng, "x", seq, [70, 2, 180] + [1] * 48), ref, torch.float32, name)
            refs.append(ref)
        moved = (refs[0][-1] - refs[1][-1]).abs().max().item()
        assert moved > 1e-3 if name == "slow" else moved < 1e-4, (name, moved)


@pytest.mark.parametrize("seed,dtype", [(700 + i, "float32") for i in range(9)] + [(700, "bfloat16"), (702, "bfloat16"), (705, "bfloat16"), (707, "bfloat16")])
def test_random_configurations(seed, dtype, tmp_path):
    """Layer orders, sizes and constants drawn at random (one head, one channel, a window of 1, one expert, one tap, one or six
    streams, loops over any stretch): a prompt in portions with a decoded tail beside a second request."""
    rng = random.Random(seed)
    cfg = random_config(rng)
    d = write_model(str(tmp_path), cfg, seed, weights=None if dtype == "float32" else pin_routing(cfg), strip_ranks=True)
    seqs = [tokens(70, cfg["vocab"], seed), tokens(33, cfg["vocab"], seed + 1)]
    plan, left_ = [], 33
    for c in [17, 2, 1, 30, 3, 11] + [1] * 6:
        m = min(left_, max(1, c // 2))
        plan.append(([(1, m)] if m else []) + [(0, c)])
        left_ -= m
    seqs[1] = seqs[1][:33 - left_]
    eng = gpu_engine(d, dtype, page=rng.choice([4, 16]), pages=400, slots=2)
    for r, got in run_plan(eng, seqs, plan).items():
        judge(d, dtype)(got, plain_logits(d, seqs[r]), seqs[r], f"request {r}")


@pytest.mark.parametrize("seed,dtype", [(21, "float32"), (21, "bfloat16"), (34, "float32"), (34, "bfloat16"), (48, "bfloat16")])
def test_larger_configurations_under_a_mixed_schedule(seed, dtype, tmp_path):
    """Six requests of 60 to 230 tokens, at most four live: portions of 2 to 100 tokens beside single tokens, requests left out of
    a step, slots and pages given back and used again; sizes of a small real model."""
    rng = random.Random(seed)
    cfg = random_config(rng, small=False)
    lens = [rng.randint(60, 230) for _ in range(6)]
    seqs = [tokens(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate(lens)]
    plan = mixed_schedule(rng, lens)
    page = rng.choice([16, 64])
    d = write_model(str(tmp_path), cfg, seed, weights=None if dtype == "float32" else pin_routing(cfg))
    eng = gpu_engine(d, dtype, page=page, pages=4 * (-(-max(lens) // page) + 1) + 2, slots=4)
    for r, got in run_plan(eng, seqs, plan).items():
        judge(d, dtype)(got, plain_logits(d, seqs[r]), seqs[r], f"request {r}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_mixed_schedule_with_heads_of_64_and_128(folders, dtype):
    folder = folder_for(folders, "D", dtype)
    lens = [211, 97, 160, 75, 130]
    seqs = [tokens(n, 200, 70 + i) for i, n in enumerate(lens)]
    eng = gpu_engine(folder, dtype, page=16, pages=4 * (-(-max(lens) // 16) + 1) + 2, slots=4)
    for r, got in run_plan(eng, seqs, mixed_schedule(random.Random(5), lens)).items():
        judge(folder, dtype)(got, plain_logits(folder, seqs[r]), seqs[r], f"request {r}")


def test_trace_replay_as_a_child_process(folders, tmp_path):
    """``bin/trace_run`` as a child process on a model of this design."""
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ids = tokens(20, 77, 9)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:11], "want": [10]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[11:], "want": [0, 8]}], "end": ["a"]}]
    for dtype in ("float32", "bfloat16"):
        folder = folder_for(folders, "B", dtype)
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [line for line in r.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
        got = torch.cat([torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(n, -1)) for i, n in ((0, 1), (1, 2))])
        rows = [10, 11, 19]
        if dtype == "float32":
            assert_close(got, plain_logits(folder, ids)[rows], torch.float32)
        else:
            assert_within_rounding(got, plain_logits(folder, ids)[rows], plain_logits(folder, ids, stored_as=torch.bfloat16)[rows])


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
