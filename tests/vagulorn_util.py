"""Small Vagulorn configurations and weights for the tests: sizes that differ from layer to layer, include 1 and values that are
no powers of two, and weights large enough that every mechanism moves the logits."""
import json
import os

import torch

from darotar_util import assert_within_rounding, mixed_schedule, tokens  # noqa: F401  (helpers that know no design)


def softmax(heads, kv_heads, dim, size, rot_dims, base=1e4, vdim=None, keep_first=None, scale=None):
    mask = {"size": size}
    if keep_first is not None:
        mask["keep_first"] = keep_first
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "mask": mask,
            "rot": {"dims": rot_dims, "base": base}, "scale": scale if scale is not None else 1.5 / dim ** 0.5}


def chunked(*args, ff=None, **kw):
    return {"type": "attention", "mixer": softmax(*args, **kw), "mlp": mlp(ff)}


def lightning(heads, dim, vdim, decay=None):
    if decay is None:       # from fast to slow
        decay = [1.0 - 0.5 ** (1 + 7 * i / max(1, heads - 1)) for i in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def pair(left, right, left_scale=1.1, right_scale=0.8, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp(ff)}


def ssm(heads, vdim, state, groups, norm_groups, conv, ff=None):
    return {"type": "mamba2", "mlp": mlp(ff),
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def model(vocab, width, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Vagulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


# Chunks of 7 and windows of 5 and 9 (no multiples of a page of four), one and five kept tokens (more than a page), a window without
# kept tokens, one decay, values narrower and wider than keys, one tap, a layer without a feed-forward.
CFG_A = model(131, 64, [
    ssm(3, 8, 6, 1, 3, 3, ff=80),
    pair(softmax(4, 2, 12, 5, 8, 500.0, keep_first=5), lightning(3, 8, 5), ff=40),
    chunked(3, 1, 12, 7, 12, 100.0, vdim=8),
    ssm(4, 6, 5, 2, 2, 1),
    pair(softmax(3, 3, 10, 9, 2, 1e4, keep_first=1), lightning(1, 20, 12, [0.97]), 0.6, -1.3, ff=24),
    pair(softmax(2, 1, 8, 6, 8, 1e4, keep_first=0), lightning(2, 3, 7, [0.0, 1.0]), ff=None),
    chunked(4, 2, 8, 33, 4, 1e5, vdim=20, ff=56),
], eps=1e-6)
# Sizes that the tensor-core kernels take; a chunk of 30; a window of 17 with 18 kept tokens; four taps.
CFG_B = model(77, 96, [
    chunked(4, 2, 32, 30, 16, 3e4, ff=112),
    pair(softmax(6, 3, 16, 17, 16, 1e3, keep_first=18), lightning(2, 32, 48), 0.9, 0.7, ff=64),
    ssm(4, 16, 16, 2, 4, 4, ff=72),
], scale=1.0)
# Larger: heads of 64 and 128, pages of 16; prompts of a few hundred tokens cross many pages, chunks and windows.
CFG_C = model(300, 128, [
    ssm(4, 64, 128, 2, 2, 4, ff=192),
    pair(softmax(8, 2, 64, 70, 32, 1e6, keep_first=3), lightning(4, 64, 32), 0.7, 0.9, ff=128),
    chunked(4, 2, 64, 100, 48, 1e4, ff=160),
    pair(softmax(2, 1, 128, 129, 128, 1e5, keep_first=20), lightning(2, 128, 100), ff=96),
    ssm(6, 32, 40, 3, 1, 2),
    chunked(4, 4, 96, 65, 32, 1e4, vdim=48),
], scale=7.0)


def make_weights(plan, seed):
    """bfloat16 tensors for every tensor of ``plan``: matrices N(0, 1.2^2 / fan_in), so activations stay of order one;
    step sizes small enough that dozens of tokens are remembered."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for ts in plan.tensor_specs():
        x = torch.randn(ts.shape, generator=g, dtype=torch.float32)
        if ts.init == "matrix":
            x = x * (1.2 / ts.shape[-1] ** 0.5)
        elif ts.init == "gain":
            x = 1.0 + 0.2 * x
        elif ts.init == "bias":
            x = 0.2 * x
        elif ts.init == "unit":
            x = 0.7 * x - (2.0 if ts.name.endswith(".dt_bias") else 0.0)
        elif ts.init != "embedding":
            raise ValueError(ts.init)
        out[ts.name] = x.to(torch.bfloat16)
    return out


def write_model(folder, cfg, seed, weights=None):
    """A model folder of ``cfg``. ``weights``: a function that changes the random tensors in place before they are written."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    from nanoinfer_b200.weights.safetensors_io import save_safetensors
    plan = plan_for(config_from_json_dict(cfg))
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = make_weights(plan, seed)
    if weights is not None:
        weights(tensors)
    save_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def read_model(folder):
    from nanoinfer_b200.weights.safetensors_io import SafetensorsFile
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    sf = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return cfg, {n: sf.tensor(n) for n in sf.names()}


def plain_logits(folder, ids, stored_as=None):
    """Float64 logits [len(ids), vocab] of the plain implementation; with ``stored_as`` every tensor that an engine keeps
    between two operations is rounded to that type on the way."""
    import plain_vagulorn as plain
    cfg, w = read_model(folder)
    if stored_as is None:
        return plain.logits(cfg, w, list(ids))
    with plain.stored_as(stored_as):
        return plain.logits(cfg, w, list(ids))


def assert_within_32_bit(folder, ids, got, ref, what=""):
    """``got`` (an engine in 32-bit) against ``ref`` (the plain implementation in float64): the common 32-bit tolerance, or three
    times what the plain implementation in 32-bit is off by where this model's own arithmetic is worse conditioned."""
    import plain_vagulorn as plain
    from gpu_util import F32_REL
    cfg, w = read_model(folder)
    got = got.detach().double().cpu()
    assert got.shape == ref.shape and torch.isfinite(got).all(), (what, got.shape, ref.shape)
    err, bound = (got - ref).abs().max().item(), F32_REL * max(1.0, ref.abs().max().item())
    if err > bound:
        with plain.computed_in(torch.float32):
            own = plain.logits(cfg, w, list(ids))
        bound = max(bound, 3.0 * (own.double()[:ref.shape[0]] - ref).abs().max().item())
    assert err <= bound < 0.01 * ref.abs().max().item(), f"{what}: max err {err:.3e}, bound {bound:.3e}"


def random_config(rng, small=True):
    """A configuration with random layer order, sizes and constants. ``small``: odd sizes, ones, sizes no kernel's fast path
    takes; else sizes of a small real model."""
    layers = []
    for _ in range(rng.randint(2, 6)):
        ff = rng.choice([None, 8, 24, 50] if small else [None, 64, 128, 256])
        kind = rng.choice(["mamba2", "attention", "parallel"])
        if kind == "mamba2":
            groups = rng.choice([1, 2, 3])
            heads = groups * rng.choice([1, 2, 4])
            vdim = rng.choice([1, 4, 8, 12, 33] if small else [32, 48, 64, 128])
            parts = rng.choice([g for g in (1, 2, 3, 4, heads) if (heads * vdim) % g == 0])
            layers.append(ssm(heads, vdim, rng.choice([1, 5, 16, 48, 70] if small else [32, 48, 96, 128]), groups, parts, rng.choice([1, 2, 3, 4, 6]), ff=ff))
            continue
        kv = rng.choice([1, 2, 3])
        dim = rng.choice([4, 8, 12, 16, 24, 40, 136] if small else [32, 64, 96, 128])
        args = (kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([1, 2, 5, 16, 17, 31, 32, 33, 64, 100] if small else [16, 48, 64, 96, 100, 130]),
                rng.choice([d for d in (2, 4, 8, 16, 32, dim) if d <= dim]), rng.choice([100.0, 1e4, 1e6]))
        scale = rng.choice([None, 0.2])
        if kind == "attention":
            layers.append(chunked(*args, vdim=rng.choice([None, 3, 8, 24] if small else [None, None, 32, 64, 128]), scale=scale, ff=ff))
            continue
        lt = softmax(*args, keep_first=rng.choice([None, 0, 1, 2, 5, 17, 40]), scale=scale)
        heads = rng.choice([1, 2, 3, 5])
        rt = lightning(heads, rng.choice([1, 4, 6, 20, 36, 140] if small else [32, 48, 64, 128]), rng.choice([1, 5, 8, 18] if small else [32, 48, 64, 128]),
                       [rng.choice([0.3, 0.9, 0.98, 0.999, 1.0]) for _ in range(heads)])
        layers.append(pair(lt, rt, rng.choice([1.0, 0.5, 1.4]), rng.choice([1.0, 0.7, -0.9]), ff=ff))
    return model(rng.choice([50, 131, 257, 1000]), rng.choice([40, 64, 72, 100, 136] if small else [128, 192, 256, 320]), layers,
                 eps=rng.choice([1e-6, 1e-5, 1e-4]), scale=rng.choice([1.0, 4.0, 11.0]))
