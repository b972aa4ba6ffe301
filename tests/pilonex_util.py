"""Small Pilonex configurations and weights for the tests: sizes that differ from layer to layer, include 1 and values that are
no powers of two, and weights large enough that every mechanism moves the logits."""
import json
import os

import torch

from darotar_util import assert_within_rounding, mixed_schedule, tokens  # noqa: F401  (helpers that know no design)


def dense(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def left(heads, kv_heads, dim, vdim, window, rot_dims, base=1e4, scaling=None, scale=None):
    """Softmax half of a pair. ``scaling``: (factor, low, high, original) or None."""
    rot = {"dims": rot_dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale if scale is not None else 1.5 / dim ** 0.5}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def right(heads, kv_heads, dim, vdim, conv, decay_rank=8, gate_rank=8):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank, "gate_rank": gate_rank}


def pair(lt, rt, left_scale=1.1, right_scale=0.8, mlp=None):
    return {"type": "parallel", "mixer": {"left": lt, "right": rt, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def memory(heads, dim, vdim, cap=10.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def model(vocab, width, layers, streams=2, loop=None, eps=1e-5):
    return {"architecture": "Pilonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": layers}


# Three streams; a loop in the middle; grouped heads on both halves, values narrower and wider than keys; windows of 5 and 9; all
# experts chosen in one layer; layers without a feed-forward; convolutions of 1, 3 and 5 taps; ranks that are no multiples of 8.
CFG_A = model(131, 64, [
    pair(left(4, 2, 12, 6, 5, 8, 500.0, (4.0, 1.0, 3.0, 40)), right(4, 2, 8, 10, 3, 5, 3), mlp=dense(40, 1.0)),
    memory(3, 8, 5, 6.0, mlp=moe(5, 2, 24, 0.7)),
    pair(left(3, 1, 8, 10, None, 4, 100.0), right(2, 1, 20, 4, 1, 11, 6), 0.6, -1.3, mlp=None),
    memory(1, 20, 12, 3.0, mlp=None),
    pair(left(2, 2, 6, 3, 9, 6, 1e4, (8.0, 0.5, 2.0, 16)), right(3, 3, 4, 7, 5, 1, 9), mlp=moe(3, 3, 16)),
], streams=3, loop=(1, 4, 2), eps=1e-6)
# Sizes that the tensor-core kernels take, windows of 17 and 33, two streams, the loop over the first layers.
CFG_B = model(77, 96, [
    pair(left(4, 2, 32, 24, 17, 32, 30000.0, (2.0, 1.0, 4.0, 64)), right(4, 4, 16, 24, 4, 16, 16), mlp=moe(7, 2, 40, 2.0)),
    memory(4, 24, 32, 8.0, mlp=dense(64)),
    pair(left(6, 3, 16, 32, 33, 8, 1000.0), right(6, 2, 32, 16, 2, 24, 8), 1.0, 1.0, mlp=dense(72, 0.9)),
], streams=2, loop=(0, 2, 3))
# Larger: pages of 16 and prompts of a few hundred tokens cross many pages and windows; one stream; no loop.
CFG_C = model(300, 128, [
    pair(left(8, 2, 64, 32, 70, 64, 1e6, (8.0, 1.0, 4.0, 256)), right(4, 2, 48, 64, 4, 16, 24), mlp=moe(8, 2, 48)),
    memory(4, 64, 48, 14.0, mlp=dense(192)),
    pair(left(4, 4, 96, 16, 129, 48, 1e4), right(2, 2, 64, 32, 3, 32, 32), mlp=moe(6, 3, 32, 0.8)),
    memory(2, 100, 64, 12.0, mlp=None),
], streams=1)
# Heads of 64 and 128 with values as wide as keys: in bfloat16 prompt portions take the attention kernel with scores in tensor
# memory. Five streams.
CFG_D = model(200, 128, [
    pair(left(4, 2, 64, 64, 70, 32, 1e6, (4.0, 1.0, 4.0, 128)), right(2, 2, 64, 128, 4, 16, 16), 0.7, 1.2, mlp=dense(96)),
    pair(left(2, 1, 128, 128, 129, 128, 1e4), right(2, 1, 128, 64, 4, 16, 16), mlp=moe(6, 2, 32)),
    memory(2, 128, 128, 15.0, mlp=dense(64)),
], streams=5, loop=(1, 3, 2))


def make_weights(plan, seed):
    """bfloat16 tensors for every tensor of ``plan``: matrices N(0, 1.2^2 / fan_in), so activations stay of order one;
    decays slow enough that dozens of tokens are remembered."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for ts in plan.tensor_specs():
        x = torch.randn(ts.shape, generator=g, dtype=torch.float32)
        if ts.init == "matrix":
            x = x * (1.2 / ts.shape[-1] ** 0.5)
        elif ts.init == "embedding":
            x = x * (1.0 if ts.name == "embed" else 1.2 / ts.shape[-1] ** 0.5)
        elif ts.init == "gain":
            x = 1.0 + 0.1 * x
        elif ts.init == "bias":             # gains stored around zero, the gates' biases
            x = 0.1 * x + (3.0 if ts.name.endswith(".f.b") else 0.0)
        elif ts.init == "unit":             # taps, rates and step sizes of the decays
            x = 0.7 * x - (3.0 if ts.name.endswith(".dt_bias") else 0.0)
        elif ts.init == "mix":
            x = (1.0 + 0.4 * x) / max(1, x.numel())
        elif ts.init == "near_identity":
            x = 0.9 * torch.eye(ts.shape[0]) + 0.15 * x
        else:
            raise ValueError(ts.init)
        out[ts.name] = x.to(torch.bfloat16)
    return out


def write_model(folder, cfg, seed, weights=None, strip_ranks=False):
    """A model folder of ``cfg``. ``weights``: a function that changes the random tensors in place before they are written.
    ``strip_ranks``: config.json does not state the inner widths that the tensors' shapes give."""
    from nanoinfer_b200.registry import config_from_json_dict, plan_for
    from nanoinfer_b200.weights.safetensors_io import save_safetensors
    plan = plan_for(config_from_json_dict(cfg))
    os.makedirs(folder, exist_ok=True)
    stated = json.loads(json.dumps(cfg))
    if strip_ranks:
        for layer in stated["layers"]:
            for key in ("decay_rank", "gate_rank"):
                layer["mixer"].get("right", {}).pop(key, None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(stated, f)
    tensors = make_weights(plan, seed)
    if weights is not None:
        weights(tensors)
    save_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def pin_routing(cfg, classes=8):
    """A change of the random tensors after which rounding cannot change the routing: the first ``classes`` channels of the
    streams hold a one-hot class of the token (token id modulo ``classes``), no sublayer ever writes them (those rows of the
    output matrices are zero) and the routers read nothing else. All logits of a token are then one number of a table times
    one common positive factor, in any precision, and no two numbers of a class are equal."""
    def change(t):
        emb = t["embed"]
        emb[:, :classes] = 0
        emb[torch.arange(emb.shape[0]), torch.arange(emb.shape[0]) % classes] = 2.0
        for name in t:
            if name.endswith((".o", ".down")):
                t[name][:classes] = 0
            if name.endswith(".in"):
                t[name].copy_(t[name].abs())
            if name.endswith(".mix"):       # the class channels keep their sign through every mix
                t[name].copy_(t[name].abs())
        for i, layer in enumerate(cfg["layers"]):
            if (layer.get("mlp") or {}).get("kind") != "moe":
                continue
            r = t[f"l{i}.mlp.router"]
            r[:, classes:] = 0
            g = torch.Generator().manual_seed(100 + i)
            for c in range(classes):
                order = torch.randperm(r.shape[0], generator=g).float()
                r[:, c] = ((order - (r.shape[0] - 1) / 2) / 4).to(r.dtype)
    return change


def read_model(folder):
    from nanoinfer_b200.weights.safetensors_io import SafetensorsFile
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    sf = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return cfg, {n: sf.tensor(n) for n in sf.names()}


def plain_logits(folder, ids, stored_as=None):
    """Float64 logits [len(ids), vocab] of the plain implementation; with ``stored_as`` every tensor that an engine keeps
    between two operations is rounded to that type on the way."""
    import plain_pilonex as plain
    cfg, w = read_model(folder)
    if stored_as is None:
        return plain.logits(cfg, w, list(ids))
    with plain.stored_as(stored_as):
        return plain.logits(cfg, w, list(ids))


def assert_within_32_bit(folder, ids, got, ref, what=""):
    """``got`` (an engine in 32-bit) against ``ref`` (the plain implementation in float64): the common 32-bit tolerance, or three
    times what the plain implementation in 32-bit is off by where this model's own arithmetic is worse conditioned."""
    import plain_pilonex as plain
    from gpu_util import F32_REL
    cfg, w = read_model(folder)
    with plain.computed_in(torch.float32):
        own = plain.logits(cfg, w, list(ids))
    got = got.detach().double().cpu()
    assert got.shape == ref.shape and torch.isfinite(got).all(), (what, got.shape, ref.shape)
    bound = max(F32_REL * max(1.0, ref.abs().max().item()), 3.0 * (own.double()[:ref.shape[0]] - ref).abs().max().item())
    err = (got - ref).abs().max().item()
    assert err <= bound < 0.01 * ref.abs().max().item(), f"{what}: max err {err:.3e}, bound {bound:.3e}"


def random_config(rng, small=True):
    """A configuration with random layer order, sizes and constants. ``small``: odd sizes, ones, sizes no kernel's fast path
    takes; else sizes of a small real model."""
    width = rng.choice([40, 64, 72, 100, 136] if small else [128, 192, 256, 320])
    layers = []
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice([None, "dense", "dense", "moe", "moe"])
        limit = rng.choice([0.4, 1.0, 3.0, 7.0])
        if kind == "dense":
            mlp = dense(rng.choice([8, 24, 50] if small else [64, 128, 256]), limit)
        elif kind == "moe":
            experts = rng.choice([1, 2, 3, 5, 8, 33] if small else [4, 8, 10, 16])
            mlp = moe(experts, rng.choice([t for t in (1, 2, 3, 4) if t <= experts]), rng.choice([8, 24, 40, 66] if small else [32, 64, 128]), limit)
        else:
            mlp = None
        if rng.random() < 0.4:
            layers.append(memory(rng.choice([1, 2, 3, 5]), rng.choice([1, 3, 8, 20, 40] if small else [32, 48, 64, 128]),
                                 rng.choice([1, 3, 5, 16, 24] if small else [32, 48, 64, 128]), rng.choice([1.0, 4.0, 10.0, 15.0]), mlp=mlp))
            continue
        kv = rng.choice([1, 2, 3])
        dim = rng.choice([4, 8, 12, 16, 24, 40, 136] if small else [32, 64, 96, 128])
        rot = rng.choice([d for d in (2, 4, 8, 16, 32, dim) if d <= dim])
        window = rng.choice([None, 1, 2, 5, 16, 17, 31, 32, 33, 64, 100] if small else [None, 16, 48, 64, 96, 100, 130])
        scaling = rng.choice([None, (2.0, 1.0, 4.0, 64), (8.0, 1.0, 2.0, 512), (32.0, 0.5, 8.0, 100)])
        lt = left(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([3, 4, 10, 24] if small else [16, 32, 64, 128]), window, rot,
                  rng.choice([100.0, 1e4, 1e6]), scaling, rng.choice([None, 0.2]))
        g = rng.choice([1, 2, 3])
        rt = right(g * rng.choice([1, 2, 3]), g, rng.choice([1, 4, 6, 20, 36] if small else [32, 48, 64, 128]),
                   rng.choice([1, 5, 8, 18] if small else [32, 48, 64, 128]), rng.choice([1, 2, 3, 4, 6]), rng.choice([1, 5, 8, 24]), rng.choice([2, 7, 16]))
        layers.append(pair(lt, rt, rng.choice([1.0, 0.5, 1.4]), rng.choice([1.0, 0.7, -0.9]), mlp=mlp))
    loop = None
    if rng.random() < 0.6:
        start = rng.randint(0, len(layers) - 1)
        loop = (start, rng.randint(start + 1, len(layers)), rng.choice([1, 2, 3]))
    return model(rng.choice([50, 131, 257, 1000]), width, layers, streams=rng.choice([1, 2, 3, 4, 6]), loop=loop, eps=rng.choice([1e-6, 1e-5, 1e-4]))
