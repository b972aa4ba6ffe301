"""Pilonex on the host backend: configuration, plan and weights; the engine's cache, state, pages and batching with the design's
mixers, streams and feed-forwards against the plain whole-sequence implementation (no GPU: the kernels' plain statements of
tests/torch_ops.py stand in for them)."""
import json
import math
import os
import random

import pytest
import torch

from pilonex_util import (CFG_A, CFG_B, dense, left, memory, model, moe, pair, plain_logits, random_config, read_model, right, tokens,
                          write_model)
from torch_ops import TorchOps


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {"A": write_model(str(tmp_path_factory.mktemp("pil_a")), CFG_A, 11, strip_ranks=True),
            "B": write_model(str(tmp_path_factory.mktemp("pil_b")), CFG_B, 12)}


def host_engine(folder, page=4, pages=96, slots=4):
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine import Engine
    return Engine(folder, EngineConfig(dtype="float32", page_size=page, num_pages=pages, max_batch=slots, device="cpu",
                                       cuda_graphs=False), ops=TorchOps())


def run_cut(eng, name, ids, cuts):
    """The request fed in portions of the given sizes; logits of every position."""
    from nanoinfer_b200.engine import StepEntry
    rc = eng.open(name)
    out, pos = [], 0
    for n in cuts:
        out.append(eng.step([StepEntry(rc, ids[pos:pos + n], list(range(n)))]))
        pos += n
    assert pos == len(ids)
    eng.close(rc)
    return torch.cat(out).double()


def close(a, b, tol=2e-4):
    assert a.shape == b.shape
    assert (a - b).abs().max().item() <= tol * max(1.0, b.abs().max().item()), (a - b).abs().max().item()


def test_config_reads_every_key_and_round_trips(folders):
    from nanoinfer_b200.config.model_config import read_config_json
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    from nanoinfer_b200.weights.loader import tensor_shapes
    cfg = config_from_json_dict(read_config_json(folders["A"]))
    assert cfg.architecture == "Pilonex" and cfg.vocab_size == 131 and cfg.hidden_size == 64
    assert cfg.norm_eps == 1e-6 and cfg.streams == 3 and cfg.loop == (1, 4, 2)
    cfg = cfg.with_tensor_shapes(tensor_shapes(folders["A"]))      # the inner widths come from the tensors
    plan = plan_for(cfg)
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 3, 1, 2, 3, 4] and all(e.reads_cache_of is None for e in plan.schedule)
    assert all(layer.arrangement == "multi_stream" for layer in plan.layers)
    lt, rt = plan.layers[0].parts["mixer"].params["left"], plan.layers[0].parts["mixer"].params["right"]
    assert lt.kind == "flex_attention" and lt.params["window"] == 5 and lt.params["rot"] == (8, 500.0) and lt.params["out_scale"] == 1.1
    assert lt.params["rot_scaling"] == {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40} and lt.params["qk_norm"] is True
    assert (lt.params["heads"], lt.params["kv_heads"], lt.params["dim"], lt.params["vdim"]) == (4, 2, 12, 6) and not lt.params["bias"]
    assert rt.kind == "gated_delta" and rt.params["conv"] == 3 and rt.params["decay_rank"] == 5 and rt.params["gate_rank"] == 3
    assert (rt.params["heads"], rt.params["kv_heads"], rt.params["dim"], rt.params["vdim"], rt.params["out_scale"]) == (4, 2, 8, 10, 0.8)
    mem = plan.layers[1].parts["mixer"]
    assert mem.kind == "matrix_memory" and mem.params["gate_cap"] == 6.0 and mem.params["vdim"] == 5
    assert plan.layers[2].parts["mixer"].params["left"].params["window"] == 0 and plan.layers[2].parts["mixer"].params["left"].params["rot_scaling"] is None
    assert plan.layers[0].parts["ffn"].params["glu"] == (1.702, 1.0, 1.0)
    assert plan.layers[1].parts["ffn"].params == {"hidden": 64, "ff": 24, "experts": 5, "top": 2, "score": "softmax", "renormalize": True,
                                                  "weight_on": "output", "glu": (1.702, 0.7, 1.0)}
    assert "ffn" not in plan.layers[2].parts and {"l2.norm2", "l2.hc2.mix", "l3.hc2.in"} <= set(plan.ignored_tensors)
    assert plan.layers[0].parts["ffn_streams"].tensors["mix"].shape == (3, 3) and plan.final_norm.params["gain_offset"] == 1.0
    again = config_from_json_dict(json.loads(json.dumps(cfg.to_json_dict())))
    assert again == cfg


def test_config_refuses_what_it_cannot_run():
    from nanoinfer_b200.config.model_config import ConfigError
    from nanoinfer_b200.registry import config_from_json_dict, plan_for

    def changed(fn):
        bad = json.loads(json.dumps(CFG_A))
        fn(bad)
        return bad

    for fn in (lambda c: c["layers"][0]["mixer"]["left"].update(heads=3),                 # no multiple of its two kv heads
               lambda c: c["layers"][0]["mixer"]["right"].update(heads=5),
               lambda c: c["layers"][1].update(type="lstm"),
               lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14),          # wider than the head
               lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("high"),
               lambda c: c["layers"][0]["mixer"].pop("right_scale"),
               lambda c: c["layers"][1]["mixer"].pop("gate_cap"),
               lambda c: c["layers"][1]["mlp"]["router"].update(top=6),
               lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"),
               lambda c: c["loop"].update(stop=6),
               lambda c: c["loop"].update(start=4, stop=2),
               lambda c: c.update(streams=0),
               lambda c: c.pop("norm")):
        with pytest.raises(ConfigError):
            config_from_json_dict(changed(fn))
    with pytest.raises(ConfigError, match="a1"):        # an inner width that neither the file nor a tensor gives
        plan_for(config_from_json_dict(changed(lambda c: c["layers"][0]["mixer"]["right"].pop("decay_rank"))))


def test_loader_names_missing_tensors_and_takes_the_unused_ones(folders, tmp_path):
    from nanoinfer_b200.weights.loader import WeightError
    from nanoinfer_b200.weights.safetensors_io import save_safetensors
    cfg, w = read_model(folders["A"])
    with open(os.path.join(tmp_path, "config.json"), "w") as f:
        json.dump(cfg, f)
    w["l2.norm2"] = torch.zeros(64, dtype=torch.bfloat16)       # of a layer without a feed-forward
    w["l2.hc2.mix"] = torch.zeros(3, 3, dtype=torch.bfloat16)
    save_safetensors(os.path.join(tmp_path, "model.safetensors"), w)
    ids = tokens(9, 131, 1)
    close(run_cut(host_engine(str(tmp_path)), "x", ids, [9]), plain_logits(folders["A"], ids))
    del w["l0.hc1.mix"]
    w["l0.mix.right.q.conv"] = torch.zeros(5, 5, dtype=torch.bfloat16)
    save_safetensors(os.path.join(tmp_path, "model.safetensors"), w)
    with pytest.raises(WeightError) as e:
        host_engine(str(tmp_path))
    assert "l0.hc1.mix" in str(e.value) and "l0.mix.right.q.conv" in str(e.value)


def test_pages_and_state_the_model_asks_for_every_pass_its_own(folders):
    eng = host_engine(folders["A"])
    needs = eng.model.cache_needs()
    assert len(needs) == 8
    assert [(t.heads, t.width) for t in needs[0][0].tensors] == [(2, 12), (2, 6)] and needs[0][0].window == 5
    assert needs[0][1].shape == (2 * (2 * 16 + 40) + 4 * 10 * 8,)           # convolution history, then S
    assert needs[1][0] is None and needs[1][1].shape == (4 + 3 * 6 * 8,)    # maxima (filled up to four), then S with the keys' sum
    assert needs[2][0].window == 0 and needs[2][1].shape == (2 * 4 * 20,)   # one tap: no history
    for e in (1, 2, 3):                                                      # the second pass of the looped layers
        assert needs[e][1] == needs[e + 3][1] and needs[e][0] == needs[e + 3][0]
        assert eng.storage.state[e].data_ptr() != eng.storage.state[e + 3].data_ptr()
    assert eng.storage.pages[2]["k"].data_ptr() != eng.storage.pages[5]["k"].data_ptr()


def test_blended_frequencies_follow_the_wavelength():
    """Every pair's frequency by hand: kept below original / high, divided above original / low, blended between, at bounds that
    fall inside, below and above all pairs."""
    from nanoinfer_b200.parts.position import scaled_frequencies
    import plain_pilonex as plain
    for dims, base, sc in ((64, 5e4, (8.0, 1.0, 4.0, 512)), (16, 100.0, (3.0, 0.25, 2.0, 20)), (8, 10.0, (2.0, 1.0, 4.0, 10 ** 6)),
                           (8, 10.0, (2.0, 1.0, 4.0, 2)), (2, 1e4, (5.0, 1.0, 4.0, 8))):
        scaling = dict(zip(("factor", "low", "high", "original"), sc))
        got, mag = scaled_frequencies(dims, base, scaling)
        assert mag == 1.0
        assert (got - plain.pair_frequencies({"dims": dims, "base": base, "scaling": scaling})).abs().max().item() < 1e-15
        raw = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        for f, g in zip(raw, got.tolist()):
            lam = 2.0 * math.pi / f
            if lam > sc[3] / sc[1]:
                assert abs(g - f / sc[0]) < 1e-15
            elif lam < sc[3] / sc[2]:
                assert g == f
            else:
                assert f / sc[0] - 1e-12 <= g <= f + 1e-12


@pytest.mark.parametrize("name,n", [("A", 37), ("B", 41)])
def test_whole_prompt_equals_plain(folders, name, n):
    ids = tokens(n, 77, 5)
    close(run_cut(host_engine(folders[name]), "r", ids, [n]), plain_logits(folders[name], ids))


@pytest.mark.parametrize("name", ["A", "B"])
def test_token_by_token_and_portions_down_to_two(folders, name):
    ids = tokens(31, 77, 6)
    ref = plain_logits(folders[name], ids)
    eng = host_engine(folders[name])
    close(run_cut(eng, "one", ids, [1] * 31), ref)
    close(run_cut(eng, "cut", ids, [2, 5, 2, 9, 1, 1, 7, 2, 2]), ref)
    close(run_cut(eng, "tail", ids, [20] + [1] * 11), ref)
    eng.cache.check()


def test_unequal_requests_in_one_batch_and_reused_slots_and_pages(folders):
    """Requests of different lengths advance together in portions and single tokens; when one ends, another takes its
    slot and pages (two slots only, a pool that forces reuse)."""
    from nanoinfer_b200.engine import StepEntry
    eng = host_engine(folders["A"], page=4, pages=34, slots=2)
    seqs = {k: tokens(n, 131, s) for k, n, s in (("p", 23, 1), ("q", 9, 2), ("r", 17, 3), ("s", 12, 4))}
    ref = {k: plain_logits(folders["A"], v) for k, v in seqs.items()}
    got, at, live, slots_used = {k: [] for k in seqs}, {k: 0 for k in seqs}, {}, {}
    plan = [[("p", 6), ("q", 2)], [("p", 1), ("q", 5)], [("p", 7), ("q", 2)], [("p", 1), ("r", 9)], [("r", 1), ("p", 1)],
            [("p", 7), ("r", 7)], [("s", 3)], [("s", 1)], [("s", 8)]]
    for step in plan:
        entries = []
        for k, n in step:
            if k not in live:
                live[k] = eng.open(k)
                slots_used[k] = live[k].slot
            entries.append(StepEntry(live[k], seqs[k][at[k]:at[k] + n], list(range(n))))
        logits = eng.step(entries).double()
        row = 0
        for k, n in step:
            got[k].append(logits[row:row + n])
            row += n
            at[k] += n
            if at[k] == len(seqs[k]):
                eng.close(live.pop(k))
        eng.cache.check()
    assert slots_used["r"] == slots_used["q"] and slots_used["s"] in (slots_used["p"], slots_used["r"])
    for k in seqs:
        close(torch.cat(got[k]), ref[k])


def test_pages_behind_a_window_go_back_to_the_pool(tmp_path):
    """A looped windowed layer: a long request holds no more pages than its window needs, twice."""
    cfg = model(50, 32, [pair(left(2, 1, 8, 4, 6, 8, 100.0), right(1, 1, 4, 4, 2), mlp=moe(3, 1, 16))], loop=(0, 1, 2))
    d = write_model(str(tmp_path), cfg, 3)
    eng = host_engine(d, page=2, pages=10, slots=1)
    ids = tokens(60, 50, 9)
    close(run_cut(eng, "long", ids, [3, 2] + [1] * 30 + [7, 11, 2, 5]), plain_logits(d, ids))
    eng.cache.check()


def variants(tmp_path, cfgs, changes=None, n=13, seed=4):
    """Plain logits of several models, each equal to the engine's; no two may be alike."""
    ids = tokens(n, 40, 2)
    refs = []
    for i, cfg in enumerate(cfgs):
        d = write_model(str(tmp_path / f"v{i}"), cfg, seed, weights=None if changes is None else changes[i])
        ref = plain_logits(d, ids)
        close(run_cut(host_engine(d), "x", ids, [5, 1, 2, n - 8]), ref)
        refs.append(ref)
    for i in range(len(refs)):
        for j in range(i):
            assert (refs[i] - refs[j]).abs().max().item() > 1e-3, (i, j)


def test_streams_are_mixed_from_row_to_column_and_in_every_number(tmp_path):
    """The mixing matrix is indexed [from, to]: its transpose gives another model; so do other numbers of streams, and each
    of the three kinds of factors moves the result."""
    layers = [memory(2, 4, 6, mlp=dense(16)), memory(1, 5, 4, mlp=None)]

    def transposed(t):
        for name in t:
            if name.endswith(".mix"):
                t[name].copy_(t[name].t().clone())

    def shares(t):
        t["l0.hc2.out"].copy_(torch.tensor([0.0, 2.0]).to(torch.bfloat16))

    def reads(t):
        t["l1.hc1.in"].copy_(torch.tensor([-1.0, 1.0]).to(torch.bfloat16))

    two = model(40, 24, layers, streams=2)
    variants(tmp_path, [two] * 4, [None, transposed, shares, reads])
    variants(tmp_path / "n", [model(40, 24, layers, streams=n) for n in (1, 3, 6)])


def test_the_loop_runs_with_the_same_weights_and_a_state_per_pass(tmp_path):
    layers = [memory(2, 4, 6, mlp=None), pair(left(2, 1, 8, 4, 3, 4, 100.0), right(2, 1, 4, 3, 3), mlp=dense(8)), memory(1, 3, 3, mlp=None)]
    variants(tmp_path, [model(40, 24, layers, loop=lp) for lp in (None, (0, 1, 2), (1, 2, 2), (1, 3, 2), (0, 3, 3))])


def test_scales_caps_and_limits_each_move_the_result(tmp_path):
    def one(scales=(1.0, 1.0), cap=8.0, limit=1.0, elimit=1.0, scaling=None, window=4):
        return model(40, 24, [pair(left(2, 1, 8, 4, window, 8, 20.0, scaling), right(2, 2, 4, 3, 3), *scales, mlp=dense(16, limit)),
                              memory(2, 4, 6, cap, mlp=moe(3, 2, 16, elimit))])
    variants(tmp_path, [one(), one(scales=(0.5, 1.0)), one(scales=(1.0, -0.5)), one(cap=1.5), one(limit=0.3), one(elimit=0.2),
                        one(scaling=(4.0, 1.0, 3.0, 12)), one(window=3), one(window=None)])


def test_limits_cut_the_gate_above_only_and_the_other_side_twice():
    ops, x = TorchOps(), torch.tensor([[1.0]])
    w = lambda g, u: torch.tensor([[g], [u]])
    for g, u in ((5.0, 5.0), (-5.0, -5.0), (0.3, -0.2), (5.0, -5.0)):
        out = torch.empty(1, 1)
        ops.linear_swiglu(x, w(g, u), out, (1.702, 2.0, 1.0))
        gc, uc = min(g, 2.0), max(-2.0, min(2.0, u))
        assert abs(out.item() - gc / (1.0 + math.exp(-1.702 * gc)) * (uc + 1.0)) < 1e-6


@pytest.mark.parametrize("seed", [600, 601, 602, 603, 604, 605, 606])
def test_random_configurations(seed, tmp_path):
    rng = random.Random(seed)
    cfg = random_config(rng)
    d = write_model(str(tmp_path), cfg, seed, strip_ranks=True)
    ids = tokens(rng.choice([19, 41, 60]), cfg["vocab"], seed)
    ref = plain_logits(d, ids)
    eng = host_engine(d, page=rng.choice([2, 4, 8]), pages=400)
    close(run_cut(eng, "w", ids, [len(ids)]), ref)
    cuts, left_ = [], len(ids)
    while left_:
        cuts.append(min(left_, rng.choice([1, 1, 2, 3, 7, 16])))
        left_ -= cuts[-1]
    close(run_cut(eng, "c", ids, cuts), ref)
    eng.cache.check()


def test_greedy_generation_through_the_scheduler(folders):
    """The framework's own entry point: a Model, its Scheduler with a small token budget (prompts go in portions,
    requests join and leave), three slots."""
    from nanoinfer_b200.api import Model
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine.scheduler import Request, Scheduler
    m = Model(folders["B"], EngineConfig(dtype="float32", page_size=4, num_pages=120, max_batch=3, max_tokens_per_step=8,
                                         device="cpu", cuda_graphs=False), ops=TorchOps())
    sched = Scheduler(m)
    prompts = [tokens(13, 77, 21), tokens(5, 77, 22), tokens(19, 77, 23), tokens(3, 77, 24)]
    for i, p in enumerate(prompts):
        sched.add(Request(f"g{i}", p, max_tokens=6))
    done = sched.run()
    for i, p in enumerate(prompts):
        ids = list(p)
        for _ in range(6):
            ids.append(int(plain_logits(folders["B"], ids)[-1].argmax()))
        assert done[f"g{i}"] == ids[len(p):], i
    m.engine.cache.check()
