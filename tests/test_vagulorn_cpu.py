"""Vagulorn on the host backend: configuration, plan and weights; the engine's cache (kept first tokens included), state and
batching with the design's mixers, norm and feed-forward against the plain whole-sequence implementation (no GPU: the kernels' plain
statements of tests/torch_ops.py stand in for them)."""
import json
import math
import os
import random

import pytest
import torch

import plain_vagulorn as plain
from torch_ops import TorchOps
from vagulorn_util import (CFG_A, CFG_B, chunked, lightning, model, pair, plain_logits, random_config, read_model, softmax, ssm, tokens,
                           write_model)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {"A": write_model(str(tmp_path_factory.mktemp("vag_a")), CFG_A, 11), "B": write_model(str(tmp_path_factory.mktemp("vag_b")), CFG_B, 12)}


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


# ------------------------------------------------------------------------------------------ the plain mechanisms, by hand
def test_plain_norm_activation_and_rotation_by_hand():
    x = torch.tensor([[1.0, 2.0, 6.0]], dtype=torch.float64)
    s = math.sqrt((4.0 + 1.0 + 9.0) / 3 + 0.5)
    got = plain.layer_norm(x, torch.tensor([1.0, 2.0, 3.0]).double(), torch.tensor([0.5, 0.0, -1.0]).double(), 0.5)
    assert torch.allclose(got, torch.tensor([[-2.0 / s + 0.5, -2.0 / s, 9.0 / s - 1.0]]).double())
    z = torch.tensor(0.7, dtype=torch.float64)
    assert abs(plain.gelu_tanh(z).item() - 0.35 * (1 + math.tanh(math.sqrt(2 / math.pi) * (0.7 + 0.044715 * 0.343)))) < 1e-15
    x = torch.arange(1.0, 13.0, dtype=torch.float64).view(2, 1, 6)
    for interleaved, (m, n) in ((True, (2, 3)), (False, (1, 3))):       # the second pair of four rotated elements
        y = plain.rotate(x, 4, 100.0, interleaved)
        a = 1 * 100.0 ** (-2.0 / 4)
        assert torch.equal(y[0], x[0]) and torch.equal(y[1, 0, 4:], x[1, 0, 4:])
        u, v = x[1, 0, m].item(), x[1, 0, n].item()
        assert abs(y[1, 0, m].item() - (u * math.cos(a) - v * math.sin(a))) < 1e-12 and abs(y[1, 0, n].item() - (v * math.cos(a) + u * math.sin(a))) < 1e-12


def test_plain_masks_by_hand():
    w = plain.visible_window(7, 2, 1)
    assert w[5].tolist() == [True, False, False, False, True, True, False] and w[0].tolist() == [True] + [False] * 6
    assert plain.visible_window(4, 2, 9)[3].tolist() == [True] * 4          # more kept tokens than there are
    assert plain.visible_window(4, 2, 0)[3].tolist() == [False, False, True, True]
    c = plain.visible_chunk(7, 3)
    assert c[5].tolist() == [False, False, False, True, True, True, False] and c[6].tolist() == [False] * 6 + [True]


# ------------------------------------------------------------------------------------------ configuration and weights
def test_config_reads_every_key_and_round_trips(folders):
    from nanoinfer_b200.config.model_config import read_config_json
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    cfg = config_from_json_dict(read_config_json(folders["A"]))
    assert cfg.architecture == "Vagulorn" and cfg.vocab_size == 131 and cfg.hidden_size == 64 and cfg.norm_eps == 1e-6 and cfg.embedding_scale == 3.0
    plan = plan_for(cfg)
    assert [e.layer for e in plan.schedule] == list(range(7)) and all(layer.arrangement == "parallel" for layer in plan.layers)
    norm = plan.layers[0].parts["mixer_norm"]
    assert norm.kind == "layernorm" and norm.params["eps"] == 1e-6 and [t.name for t in norm.tensors.values()] == ["l0.norm1", "l0.norm1.b"]
    ssm_ = plan.layers[0].parts["mixer"]
    assert ssm_.kind == "mamba2" and (ssm_.params["heads"], ssm_.params["vdim"], ssm_.params["state"], ssm_.params["groups"],
                                      ssm_.params["norm_groups"], ssm_.params["conv"]) == (3, 8, 6, 1, 3, 3)
    lt, rt = plan.layers[1].parts["mixer"].params["left"], plan.layers[1].parts["mixer"].params["right"]
    p = lt.params
    assert lt.kind == "flex_attention" and (p["heads"], p["kv_heads"], p["dim"], p["vdim"]) == (4, 2, 12, 12)
    assert (p["window"], p["keep_first"], p["chunk"], p["rot"], p["rot_layout"], p["out_scale"]) == (5, 5, 0, (8, 500.0), "interleaved", 1.1)
    assert p["values_from_keys"] and p["qk_norm"] is True and p["out_gate"] == "head" and "v" not in lt.tensors
    assert lt.tensors["g"].shape == (4, 64) and lt.tensors["g"].name == "l1.mix.left.g"
    assert rt.kind == "lightning_attention" and rt.params["decay"] == tuple(CFG_A["layers"][1]["mixer"]["right"]["decay"])
    assert (rt.params["heads"], rt.params["dim"], rt.params["vdim"], rt.params["out_scale"]) == (3, 8, 5, 0.8)
    p = plan.layers[2].parts["mixer"].params
    assert (p["chunk"], p["window"], p["rot_layout"], p["vdim"], p["out_gate"], p["values_from_keys"]) == (7, 0, "half", 8, False, False)
    assert plan.layers[0].parts["ffn"].params["act"] == "gelu_tanh" and "ffn" not in plan.layers[3].parts
    assert plan.lm_head.tensors["weight"].name == plan.embedding.tensors["table"].name == "embed"
    assert plan.final_norm.kind == "layernorm" and plan.final_norm.tensors["bias"].name == "final.norm.b"
    assert config_from_json_dict(json.loads(json.dumps(cfg.to_json_dict()))) == cfg


def test_config_refuses_what_it_cannot_run():
    from nanoinfer_b200.config.model_config import ConfigError
    from nanoinfer_b200.registry import config_from_json_dict
    for fn in (lambda c: c["layers"][1]["mixer"]["left"].update(heads=3),                 # no multiple of its two kv heads
               lambda c: c["layers"][1]["mixer"]["left"].update(vdim=6),                   # the values are the keys
               lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1),
               lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5]),        # three heads
               lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 1.5, 0.5]),
               lambda c: c["layers"][1]["mixer"].pop("right_scale"),
               lambda c: c["layers"][2]["mixer"].pop("rot"),
               lambda c: c["layers"][2]["mixer"]["rot"].update(dims=14),                   # wider than the head
               lambda c: c["layers"][0]["mixer"].update(norm_groups=5),
               lambda c: c["layers"][0].update(type="lstm"),
               lambda c: c["layers"][0]["mlp"].update(kind="moe"),
               lambda c: c.pop("norm")):
        bad = json.loads(json.dumps(CFG_A))
        fn(bad)
        with pytest.raises(ConfigError):
            config_from_json_dict(bad)


def test_loader_names_missing_and_wrong_tensors(folders, tmp_path):
    from nanoinfer_b200.weights.loader import WeightError
    from nanoinfer_b200.weights.safetensors_io import save_safetensors
    cfg, w = read_model(folders["A"])
    with open(os.path.join(tmp_path, "config.json"), "w") as f:
        json.dump(cfg, f)
    del w["l0.norm1.b"]
    w["l1.mix.left.g"] = torch.zeros(48, 64, dtype=torch.bfloat16)
    save_safetensors(os.path.join(tmp_path, "model.safetensors"), w)
    with pytest.raises(WeightError) as e:
        host_engine(str(tmp_path))
    assert "l0.norm1.b" in str(e.value) and "l1.mix.left.g" in str(e.value)


def test_random_weights_mode_makes_a_model_that_loads(tmp_path):
    from nanoinfer_b200.registry import config_from_json_dict
    from nanoinfer_b200.weights.random_init import write_random_model
    write_random_model(config_from_json_dict(CFG_B), str(tmp_path), seed=3)
    ids = tokens(9, 77, 1)
    close(run_cut(host_engine(str(tmp_path)), "x", ids, [9]), plain_logits(str(tmp_path), ids))


# ------------------------------------------------------------------------------------------ cache and state
def test_pages_and_state_the_model_asks_for(folders):
    eng = host_engine(folders["A"])
    needs = eng.model.cache_needs()
    assert needs[0][0] is None and needs[0][1].shape == (2 * (24 + 12) + 3 * 8 * 6,)         # convolution history, then S
    assert [(t.heads, t.width) for t in needs[1][0].tensors] == [(2, 12), (2, 12)]
    assert (needs[1][0].window, needs[1][0].keep_first) == (5, 5) and needs[1][1].shape == (3 * 8 * 5,)
    assert (needs[2][0].window, needs[2][0].keep_first) == (7, 0) and needs[2][1] is None
    assert needs[3][1].shape == (4 * 6 * 5,)                                                  # one tap: no history


def test_pages_between_kept_tokens_and_the_window_go_back_to_the_pool():
    """A group of its own; the pages that hold the first six positions stay, those behind the window go, in any portions."""
    from nanoinfer_b200.cache.pages import CacheManager, GroupSpec
    mgr = CacheManager([GroupSpec(5, (0,), (), 6), GroupSpec(5, (1,), ())], 8, 4, 2)
    rc = mgr.open("a")
    length = 0
    for n in (3, 9, 1, 1, 7, 1, 11):
        mgr.extend(rc, n)
        mgr.commit(rc, n)
        length += n
        first = max(0, length - 5 + 1) // 4
        pages = -(-length // 4)
        assert [p >= 0 for p in rc.tables[0]] == [lp < 2 or lp >= first for lp in range(pages)]
        assert [p >= 0 for p in rc.tables[1]] == [lp >= first for lp in range(pages)]
        mgr.check()
    with pytest.raises(ValueError):
        mgr.truncate(rc, 12)
    mgr.close(rc)
    assert mgr.num_free(0) == mgr.num_free(1) == 8
    mgr.check()


def test_needs_that_differ_in_kept_tokens_do_not_share_a_group():
    from nanoinfer_b200.cache.storage import plan_groups
    from nanoinfer_b200.parts.base import CacheNeed, PagedTensor
    t = (PagedTensor("k", 2, 8), PagedTensor("v", 2, 8))
    groups, of = plan_groups([(CacheNeed(t, 16, 2), None, None), (CacheNeed(t, 16), None, None), (CacheNeed(t, 16, 2), None, None)])
    assert of == [0, 1, 0] and [(g.window, g.keep_first) for g in groups] == [(16, 2), (16, 0)]


def test_a_long_request_holds_no_more_pages_than_its_window_and_kept_tokens(tmp_path):
    cfg = model(50, 32, [pair(softmax(2, 1, 8, 4, 4, 100.0, keep_first=3), lightning(1, 4, 4), ff=16), chunked(2, 1, 8, 6, 8, 50.0)])
    d = write_model(str(tmp_path), cfg, 3)
    eng = host_engine(d, page=2, pages=11, slots=1)
    ids = tokens(70, 50, 9)
    close(run_cut(eng, "long", ids, [3, 2] + [1] * 30 + [9, 11, 2, 13]), plain_logits(d, ids))
    eng.cache.check()


# ------------------------------------------------------------------------------------------ the engine against plain
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
    """Requests of different lengths advance together in portions and single tokens; when one ends, another takes its slot and
    pages (two slots only, a pool that forces reuse)."""
    from nanoinfer_b200.engine import StepEntry
    eng = host_engine(folders["A"], page=4, pages=14, slots=2)
    seqs = {k: tokens(n, 131, s) for k, n, s in (("p", 23, 1), ("q", 9, 2), ("r", 17, 3), ("s", 12, 4))}
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
        close(torch.cat(got[k]), plain_logits(folders["A"], seqs[k]))


def variants(tmp_path, cfgs, n=19, seed=4):
    """Plain logits of several models with the same weights, each equal to the engine's; no two may be alike."""
    ids = tokens(n, 40, 2)
    refs = []
    for i, cfg in enumerate(cfgs):
        d = write_model(str(tmp_path / f"v{i}"), cfg, seed)
        ref = plain_logits(d, ids)
        close(run_cut(host_engine(d), "x", ids, [5, 1, 2, n - 8]), ref)
        refs.append(ref)
    for i in range(len(refs)):
        for j in range(i):
            assert (refs[i] - refs[j]).abs().max().item() > 1e-3, (i, j)


def test_every_constant_of_config_moves_the_result(tmp_path):
    def one(scales=(1.0, 0.7), window=4, keep=2, decay=(0.5, 0.9), base=20.0, dims=4, scale=0.5, chunk=5, cdims=8, cbase=10.0, cscale=0.4, emb=2.0, eps=1e-3):
        return model(40, 24, [pair(softmax(2, 1, 8, window, dims, base, keep_first=keep, scale=scale), lightning(2, 4, 6, list(decay)), *scales, ff=16),
                              chunked(2, 2, 8, chunk, cdims, cbase, scale=cscale, ff=16), ssm(2, 4, 6, 2, 2, 3)], scale=emb, eps=eps)
    variants(tmp_path, [one(), one(scales=(0.5, 0.7)), one(scales=(1.0, -0.5)), one(window=5), one(keep=1), one(keep=None), one(decay=(0.5, 0.8)),
                        one(base=30.0), one(dims=8), one(scale=1.0), one(chunk=6), one(cdims=4), one(cbase=15.0), one(cscale=0.8), one(emb=0.5), one(eps=0.1)])


def test_without_a_mask_every_earlier_position_is_seen(tmp_path):
    wide = model(40, 24, [chunked(2, 1, 8, 1000, 4, 50.0, ff=16), pair(softmax(2, 1, 8, 1000, 8, 20.0), lightning(1, 4, 4), ff=16)])
    bare = json.loads(json.dumps(wide))
    bare["layers"][0]["mixer"].pop("mask")
    bare["layers"][1]["mixer"]["left"].pop("mask")
    ids = tokens(23, 40, 3)
    ref = plain_logits(write_model(str(tmp_path / "wide"), wide, 4), ids)
    close(run_cut(host_engine(write_model(str(tmp_path / "bare"), bare, 4)), "x", ids, [9, 1, 13]), ref)


@pytest.mark.parametrize("groups,parts", [(1, 1), (2, 4), (4, 2)])
def test_groups_and_norm_parts_of_the_state_space_mixer(tmp_path, groups, parts):
    d = write_model(str(tmp_path), model(40, 24, [ssm(4, 6, 5, groups, parts, 4, ff=16), ssm(4, 6, 5, groups, parts, 1)]), 7)
    ids = tokens(21, 40, 3)
    close(run_cut(host_engine(d), "x", ids, [2, 9, 1, 1, 8]), plain_logits(d, ids))


@pytest.mark.parametrize("seed", [800, 801, 802, 803, 804, 805, 806, 807])
def test_random_configurations(seed, tmp_path):
    rng = random.Random(seed)
    cfg = random_config(rng)
    d = write_model(str(tmp_path), cfg, seed)
    ids = tokens(rng.choice([19, 41, 60]), cfg["vocab"], seed)
    ref = plain_logits(d, ids)
    eng = host_engine(d, page=rng.choice([2, 4, 8]), pages=400)
    close(run_cut(eng, "w", ids, [len(ids)]), ref)
    cuts, left = [], len(ids)
    while left:
        cuts.append(min(left, rng.choice([1, 1, 2, 3, 7, 16])))
        left -= cuts[-1]
    close(run_cut(eng, "c", ids, cuts), ref)
    eng.cache.check()


def test_greedy_generation_through_the_scheduler(folders):
    """The framework's own entry point: a Model, its Scheduler with a small token budget (prompts go in portions, requests join
    and leave), three slots."""
    from nanoinfer_b200.api import Model
    from nanoinfer_b200.config import EngineConfig
    from nanoinfer_b200.engine.scheduler import Request, Scheduler
    m = Model(folders["B"], EngineConfig(dtype="float32", page_size=4, num_pages=120, max_batch=3, max_tokens_per_step=8,
                                         device="cpu", cuda_graphs=False), ops=TorchOps())
    sched = Scheduler(m)
    prompts = [tokens(13, 77, 21), tokens(5, 77, 22), tokens(25, 77, 23), tokens(3, 77, 24)]
    for i, p in enumerate(prompts):
        sched.add(Request(f"g{i}", p, max_tokens=6))
    done = sched.run()
    for i, p in enumerate(prompts):
        ids = list(p)
        for _ in range(6):
            ids.append(int(plain_logits(folders["B"], ids)[-1].argmax()))
        assert done[f"g{i}"] == ids[len(p):], i
    m.engine.cache.check()
