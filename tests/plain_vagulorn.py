"""Vagulorn, slowly and plainly: whole sequences in float64, one function per mechanism, loops over tokens where the
design is a recurrence. Shares no code with the package; the tests compare the engine with it.

A model is ``(config dict, {tensor name: tensor})``. ``logits(cfg, w, ids)`` returns ``[len(ids), vocab]``;
``forward(cfg, w, ids)`` also returns the residual stream after every layer. Inside ``stored_as(torch.bfloat16)`` the
matrix products' inputs and activations are rounded to that type, which gives the error that storage alone causes;
inside ``computed_in(torch.float32)`` everything is computed in that type.
"""
import math
from contextlib import contextmanager

import torch

F = torch.float64
_STORE = [None]


@contextmanager
def computed_in(dtype):
    global F
    before, F = F, dtype
    try:
        yield
    finally:
        F = before


@contextmanager
def stored_as(dtype):
    _STORE[0] = dtype
    try:
        yield
    finally:
        _STORE[0] = None


def stored(x):
    """x as it is kept between two kernels: rounded to the storage type, if one is set."""
    return x if _STORE[0] is None else x.to(_STORE[0]).to(F)


def product(h, w):
    return stored(h) @ w.t()


def layer_norm(x, w, b, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(u, w, bias):
    """u [T, C], w [C, taps]: y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    t_len, taps = u.shape[0], w.shape[1]
    y = bias.expand(t_len, -1).clone()
    for t in range(t_len):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def rotate(x, dims, base, interleaved):
    """x [T, heads, d]: the first ``dims`` of every head turned by position; pairs (2i, 2i + 1) or (i, i + dims/2)."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(x.shape[0], dtype=F) * base ** (-2.0 * i / dims)
        c, s = a.cos()[:, None], a.sin()[:, None]
        m, n = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        out[..., m] = x[..., m] * c - x[..., n] * s
        out[..., n] = x[..., n] * c + x[..., m] * s
    return out


def visible_chunk(t_len, size):
    """[T, T] bool: earlier positions of the own block of ``size``, counted from the sequence's start."""
    i, j = torch.arange(t_len)[:, None], torch.arange(t_len)[None, :]
    return (j <= i) & (i // size == j // size)


def visible_window(t_len, size, keep_first):
    """[T, T] bool: the last ``size`` positions and the first ``keep_first`` of the sequence."""
    i, j = torch.arange(t_len)[:, None], torch.arange(t_len)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_attention(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    rep = q.shape[1] // k.shape[1]
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=F)
    for h in range(q.shape[1]):
        s = (q[:, h] @ k[:, h // rep].t()) * scale
        out[:, h] = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v[:, h // rep]
    return out


def matrix_state(q, k, v, decay):
    """S_t = decay_t S_(t-1) + k_t v_t^T per head, o_t = S_t^T q_t. q, k [T, H, dk]; v [T, H, dv]; decay [T, H]."""
    t_len, heads, dk = k.shape
    s = torch.zeros(heads, dk, v.shape[2], dtype=F)
    out = torch.zeros(t_len, heads, v.shape[2], dtype=F)
    for t in range(t_len):
        s = decay[t][:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out


def chunked_attention(h, w, p, m, eps):
    t_len = h.shape[0]
    q = rms_norm(product(h, w[p + ".q"]).view(t_len, m["heads"], m["dim"]), w[p + ".q.norm"], eps)
    k = rms_norm(product(h, w[p + ".k"]).view(t_len, m["kv_heads"], m["dim"]), w[p + ".k.norm"], eps)
    v = product(h, w[p + ".v"]).view(t_len, m["kv_heads"], m["vdim"])
    q, k = (rotate(x, m["rot"]["dims"], m["rot"]["base"], False) for x in (q, k))
    o = softmax_attention(stored(q), stored(k), stored(v), m["scale"], visible_chunk(t_len, m["mask"]["size"]))
    return product(o.reshape(t_len, -1), w[p + ".o"])


def windowed_attention(h, w, p, m, eps):
    """Values are the projected keys; the first tokens stay visible; one gate per head."""
    t_len = h.shape[0]
    q = rms_norm(product(h, w[p + ".q"]).view(t_len, m["heads"], m["dim"]), w[p + ".q.norm"], eps)
    v = product(h, w[p + ".k"]).view(t_len, m["kv_heads"], m["dim"])
    k = rms_norm(v, w[p + ".k.norm"], eps)
    q, k = (rotate(x, m["rot"]["dims"], m["rot"]["base"], True) for x in (q, k))
    o = softmax_attention(stored(q), stored(k), stored(v), m["scale"], visible_window(t_len, m["mask"]["size"], m["mask"].get("keep_first") or 0))
    o = o * torch.sigmoid(product(h, w[p + ".g"]))[:, :, None]
    return product(o.reshape(t_len, -1), w[p + ".o"])


def lightning_attention(h, w, p, m, eps):
    t_len, heads = h.shape[0], m["heads"]
    q, k = (silu(product(h, w[f"{p}.{n}"])).view(t_len, heads, m["dim"]) for n in "qk")
    v = silu(product(h, w[p + ".v"])).view(t_len, heads, m["vdim"])
    o = matrix_state(q, k, v, torch.tensor(m["decay"], dtype=F).expand(t_len, heads)).reshape(t_len, -1)
    return product(rms_norm(o, w[p + ".norm"], eps) * torch.sigmoid(product(h, w[p + ".g"])), w[p + ".o"])


def pair_mixer(h, w, p, m, eps):
    return m["left_scale"] * windowed_attention(h, w, p + ".left", m["left"], eps) \
        + m["right_scale"] * lightning_attention(h, w, p + ".right", m["right"], eps)


def mamba2_mixer(h, w, p, m, eps):
    t_len = h.shape[0]
    heads, dv, n, groups = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = heads * dv, groups * n
    z, xbc, dt = torch.split(product(h, w[p + ".in"]), [inner, inner + 2 * gn, heads], dim=1)
    xbc = silu(short_conv(xbc, w[p + ".conv"], w[p + ".conv.b"]))
    x, b, c = torch.split(xbc, [inner, gn, gn], dim=1)
    x, b, c = x.reshape(t_len, heads, dv), b.reshape(t_len, groups, n), c.reshape(t_len, groups, n)
    dt = torch.logaddexp(dt + w[p + ".dt_bias"], torch.zeros((), dtype=F))
    rep = heads // groups
    y = matrix_state(c.repeat_interleave(rep, 1), b.repeat_interleave(rep, 1), x * dt[:, :, None], torch.exp(-torch.exp(w[p + ".A_log"]) * dt))
    y = (y + w[p + ".D"][:, None] * x).reshape(t_len, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms_norm(y.view(t_len, parts, -1), w[p + ".norm"].view(parts, -1), eps).reshape(t_len, inner)
    return product(y, w[p + ".o"])


def feed_forward(h, w, p):
    return product(gelu_tanh(product(h, w[p + ".gate"])) * product(h, w[p + ".up"]), w[p + ".down"])


MIXERS = {"attention": chunked_attention, "parallel": pair_mixer, "mamba2": mamba2_mixer}


def forward(cfg, weights, ids):
    w = {k: v.to(F) for k, v in weights.items() if v.is_floating_point()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)] * cfg["embedding"]["scale"]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        h = layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
        y = MIXERS[layer["type"]](h, w, f"l{i}.mix", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, f"l{i}.mlp")
        x = x + y
        streams.append(x)
    return product(layer_norm(x, w["final.norm"], w["final.norm.b"], eps), w["embed"]), streams


def logits(cfg, weights, ids):
    return forward(cfg, weights, ids)[0]
