"""The arithmetic behind the bench record (bytes a decode step reads, FLOPs of a prefill, peaks), and what
the bench says when asked for more than one GPU. No GPU is needed."""
import json
import os
import subprocess
import sys

import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
import bench  # noqa: E402


@pytest.fixture()
def shape():
    saved = dict(bench.MODEL)
    yield lambda name: bench.MODEL.update(bench.SHAPES[name])
    bench.MODEL.clear()
    bench.MODEL.update(saved)


def test_step_bytes_and_prefill_flops_of_the_three_shapes(shape):
    # per layer: (q + 2 kv heads) * hd * hidden + hidden * q * hd + 3 * hidden * intermediate matrix parameters
    n = bench.model_numbers(24)                                  # 0.5B: 357.83 M in the layers + 136.13 M head
    assert n["per_layer_params"] == (14 + 4) * 64 * 896 + 896 * 14 * 64 + 3 * 896 * 4864
    assert round(n["weight_bytes"] / 1e6) == 988
    assert n["kv_bytes_per_token"] == 12 * 1024
    assert abs(n["prefill_flops"](2048) / 1e12 - 1.65) < 0.01
    shape("1.5b")
    n = bench.model_numbers(28)
    assert round(n["weight_bytes"] / 1e6) == 3087 and n["kv_bytes_per_token"] == 28 * 1024
    assert abs(n["prefill_flops"](2048) / 1e12 - 5.73) < 0.01
    shape("7b")
    n = bench.model_numbers(28)
    assert round(n["weight_bytes"] / 1e9, 2) == 14.14 and n["kv_bytes_per_token"] == 56 * 1024
    assert abs(n["prefill_flops"](2048) / 1e12 - 27.57) < 0.02
    assert bench.model_numbers(4)["weight_bytes"] < n["weight_bytes"]      # fewer layers: fewer bytes, named in config


def test_peaks_come_from_the_measured_file_when_it_is_there(tmp_path, monkeypatch):
    monkeypatch.setattr(bench, "ROOT", str(tmp_path))
    assert bench.peaks() == bench.FALLBACK_PEAKS and bench.peaks()["source"] == "fallback"
    (tmp_path / "MEASURED_PEAKS.json").write_text(json.dumps(
        {"hbm_gbs": 6900.5, "bf16_tflops": 1610, "bf16_tflops_sustained": {"value": 1405.0}, "clocks": {"sm": 1900}}))
    p = bench.peaks()
    assert (p["hbm_gbs"], p["bf16_tflops"], p["bf16_tflops_sustained"], p["source"]) == (6900.5, 1610.0, 1405.0, "measured")
    (tmp_path / "MEASURED_PEAKS.json").write_text(json.dumps({"hbm_gbs": 7000}))
    p = bench.peaks()
    assert p["hbm_gbs"] == 7000.0 and p["bf16_tflops"] == 1590.0 and "partly" in p["source"]
    (tmp_path / "MEASURED_PEAKS.json").write_text("not json")
    assert bench.peaks()["source"] == "fallback"


def test_more_than_one_gpu_is_refused_with_one_line():
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bench.py"), "--gpus", "2"], capture_output=True, text=True,
                       timeout=120)
    assert r.returncode == 2
    lines = [line for line in r.stdout.splitlines() if line.strip()]
    assert len(lines) == 1 and json.loads(lines[0])["n_gpus"] == 2


def test_launches_are_sorted_into_the_parts_of_a_layer():
    """The breakdown names a launch by its kernel, its epilogue and its place in the layer's order."""
    epi = {"qkv": "qkv", "o": "add", "gate_up": "swiglu", "down": "add", "head": "f32"}
    order = [("embed", None), ("gemm_smallm", "qkv"), ("attention_decode", None), ("gemm_smallm", "o"), ("rmsnorm", None),
             ("gemm_smallm", "gate_up"), ("gemm_tc", "down"), ("rmsnorm", None), ("gemm_tc", "qkv"), ("rope_store", None),
             ("attention_decode", None), ("gemm_tc", "o"), ("rmsnorm", None), ("gemm_tc", "gate_up"), ("gemm_tc", "down"),
             ("rmsnorm", None), ("gemm_tc", "head"), ("argmax", None)]
    state, kinds = {}, []
    for kernel, what in order:
        state["tag"] = epi.get(what)
        kinds.append(bench._kind_of(kernel, "", state))
    assert kinds == ["embed", "qkv", "attention", "o_proj", "rmsnorm", "gate_up", "down", "rmsnorm", "qkv", "rope_store",
                     "attention", "o_proj", "rmsnorm", "gate_up", "down", "rmsnorm", "lm_head", "argmax"]
    n = bench.model_numbers(24)
    assert n["kinds"]["qkv"] == 1152 * 896 and n["kinds"]["gate_up"] == 2 * 896 * 4864
    assert sum(n["kinds"][k] for k in ("qkv", "o_proj", "gate_up", "down")) == n["per_layer_params"]
    assert n["kv_bytes_per_token_layer"] * 24 == n["kv_bytes_per_token"]


def test_the_designs_bench_sizes_are_configurations_the_registry_takes():
    """``--design darotar``: both models of a size are valid configurations of equal width, depth and vocabulary, and a
    token passes through as many feed-forward parameters in both (``top`` experts, each ``1 / top`` of the dense one)."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    for size in bench.DAROTAR_SIZES.values():
        dar, dense = bench.darotar_configs(size)
        plan, dense_plan = plan_for(config_from_json_dict(dar)), plan_for(config_from_json_dict(dense))
        assert len(plan.layers) == len(dense_plan.layers) == size["layers"]
        assert plan.hidden_size == dense_plan.hidden_size == size["width"] and plan.vocab_size == dense_plan.vocab_size
        kinds = [layer["type"] for layer in dar["layers"]]
        assert kinds.count("attention") == kinds.count("latent_attention") == size["layers"] // 2
        readers = [i for i, layer in enumerate(dar["layers"]) if layer["mixer"].get("kv_from") is not None]
        assert readers and all(dar["layers"][dar["layers"][i]["mixer"]["kv_from"]]["type"] == "latent_attention" for i in readers)
        mlp = dar["layers"][0]["mlp"]
        assert mlp["router"]["top"] * mlp["expert"]["ff"] == size["ff_swiglu"]


def test_the_fifth_designs_bench_sizes_are_configurations_the_registry_takes():
    """``--design dusilorn``: both models of a size are valid configurations of equal width, depth and vocabulary; windowed and
    chunked layers by turns; a token passes through as many feed-forward parameters in both (two experts and the shared one,
    two matrices each and half as wide, against three matrices)."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    for size in bench.DUSILORN_SIZES.values():
        dus, dense = bench.dusilorn_configs(size)
        plan, dense_plan = plan_for(config_from_json_dict(dus)), plan_for(config_from_json_dict(dense))
        assert len(plan.layers) == len(dense_plan.layers) == size["layers"]
        assert plan.hidden_size == dense_plan.hidden_size == size["width"] and plan.vocab_size == dense_plan.vocab_size
        kinds = [layer["type"] for layer in dus["layers"]]
        assert kinds.count("attention") == kinds.count("attention_2") == size["layers"] // 2
        mlp = dus["layers"][1]["mlp"]
        assert 2 * (mlp["router"]["top"] * mlp["expert"]["ff"] + mlp["shared"]["ff"]) == 3 * size["ff_swiglu"]
        assert dus["layers"][0]["mlp"]["kind"] == "dense" and plan.layers[1].parts["mixer"].params["v_mix"] == "blend"


def test_the_sixth_designs_bench_sizes_are_configurations_the_registry_takes():
    """``--design pilonex``: both models of a size are valid configurations of equal width and vocabulary, with as many layer
    runs (two layers run twice) as the dense decoder has layers; a token passes through as many feed-forward parameters."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    for size in bench.PILONEX_SIZES.values():
        pil, dense = bench.pilonex_configs(size)
        plan, dense_plan = plan_for(config_from_json_dict(pil)), plan_for(config_from_json_dict(dense))
        assert len(plan.schedule) == len(dense_plan.layers) == size["layers"] and len(plan.layers) == size["layers"] - 2
        assert [e.layer for e in plan.schedule] == [0, 1, 0, 1, 2, 3, 4, 5]
        assert plan.hidden_size == dense_plan.hidden_size == size["width"] and plan.vocab_size == dense_plan.vocab_size
        kinds = [layer["type"] for layer in pil["layers"]]
        assert kinds.count("parallel") == 4 and kinds.count("mlstm") == 2
        moe = pil["layers"][1]["mlp"]
        assert moe["router"]["top"] * moe["expert"]["ff"] == size["ff_swiglu"] == pil["layers"][0]["mlp"]["ff"]


def test_the_seventh_designs_bench_sizes_are_configurations_the_registry_takes():
    """``--design vagulorn``: all three models of a size are valid configurations of equal width, depth and vocabulary; the two designs
    agree layer by layer in feed-forwards, head counts and state-space mixers."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    for size in bench.VAGULORN_SIZES.values():
        vag, vaf, dense = bench.vagulorn_configs(size)
        plans = [plan_for(config_from_json_dict(c)) for c in (vag, vaf, dense)]
        assert [len(p.layers) for p in plans] == [size["layers"]] * 3
        assert len({p.hidden_size for p in plans}) == len({p.vocab_size for p in plans}) == 1
        kinds = [layer["type"] for layer in vag["layers"]]
        assert (kinds.count("parallel"), kinds.count("mamba2"), kinds.count("attention")) == (2, 4, 2)
        for a, b in zip(vag["layers"], vaf["layers"]):
            assert a["mlp"] == b["mlp"]
            if a["type"] == "mamba2":
                assert a["mixer"] == b["mixer"]
            else:
                lt = a["mixer"].get("left", a["mixer"])
                assert all(lt[k] == b["mixer"]["left"][k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
