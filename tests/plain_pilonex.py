"""Pilonex, slowly and plainly: whole sequences in float64, one function per mechanism. Shares no code with the package;
the tests compare the engine with it.

A model is ``(config dict, {tensor name: tensor})``. ``logits(cfg, w, ids)`` returns ``[len(ids), vocab]``;
``forward(cfg, w, ids)`` also returns the sum of the streams after every layer run (a looped layer counts every time).

Computed in float64; ``with computed_in(torch.float32):`` the same statements in 32-bit, whose distance to the 64-bit result is what
32-bit arithmetic alone does to a model (a head of one channel, normed, turns a small number into a sign).

With a storage type set (``with stored_as(torch.bfloat16):``) every tensor that an engine keeps in that type between two
operations is rounded to it; the distance to the unrounded result is what rounding alone does to the model's logits.
"""
import math

import torch

F = torch.float64
_STORED = None


class stored_as:
    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        global _STORED
        self.before, _STORED = _STORED, self.dtype

    def __exit__(self, *exc):
        global _STORED
        _STORED = self.before


class computed_in:
    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        global F
        self.before, F = F, self.dtype

    def __exit__(self, *exc):
        global F
        F = self.before


def kept(x):
    return x if _STORED is None else x.to(_STORED).to(F)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    """The layer norm of the design: the gain is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


# ---- softmax half of a pair -------------------------------------------------------------------------------------------
def pair_frequencies(rot):
    """One frequency per rotated pair; with ``scaling`` the slow ones are divided by its factor, the fast ones stay, and
    those whose wavelength lies between the two bounds are blended."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wavelength = 2.0 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif not wavelength < original / high:
                share = (original / wavelength - low) / (high - low)
                f = (1.0 - share) * f / factor + share * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate_half_pairs(x, rot, first=0):
    """x [T, heads, d]: element i of the first rot.dims elements of a head is paired with element i + dims/2."""
    dims = int(rot["dims"])
    half = dims // 2
    a = (first + torch.arange(x.shape[0], dtype=F))[:, None] * pair_frequencies(rot)[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def mask_window(t_len, size):
    i, j = torch.arange(t_len)[:, None], torch.arange(t_len)[None, :]
    return (j <= i) & (i - j < size)


def window_attention(m, w, p, h, eps):
    t_len = h.shape[0]
    heads, groups, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = unit_rms((h @ w[p + ".q"].t()).view(t_len, heads, dim), eps) * w[p + ".q.norm"]
    k = unit_rms((h @ w[p + ".k"].t()).view(t_len, groups, dim), eps) * w[p + ".k.norm"]
    q, k = kept(rotate_half_pairs(q, m["rot"])), kept(rotate_half_pairs(k, m["rot"]))
    v = kept(h @ w[p + ".v"].t()).view(t_len, groups, vdim)
    mask = mask_window(t_len, int(m["mask"]["size"]) if m.get("mask") else t_len)
    out = torch.zeros(t_len, heads, vdim, dtype=F)
    for n in range(heads):
        g = n // (heads // groups)
        s = ((q[:, n] @ k[:, g].t()) * float(m["scale"])).masked_fill(~mask, -math.inf)
        out[:, n] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(t_len, -1)


# ---- delta-rule half of a pair ----------------------------------------------------------------------------------------
def short_convolution(x, taps):
    """x [T, channels], taps [channels, n]: the last column meets the current token; zeros before the start; then silu."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F), x], 0)
    y = sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n))
    return y * torch.sigmoid(y)


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_decays(w, p, h, heads, dim):
    z = kept(h @ w[p + ".a1"].t()) @ w[p + ".a2"].t() + w[p + ".dt_bias"]
    step = torch.nn.functional.softplus(z, threshold=1e9).view(h.shape[0], heads, dim)
    return torch.exp(-torch.exp(w[p + ".A_log"])[None, :, None] * step)


def delta_walk(q, k, v, g, beta):
    """q, k, g [T, heads, dim], v [T, heads, vdim], beta [T, heads]: the state decays by rows, the part of v that the
    state already answers to k is taken off, the rest is written (times beta), then the state is read."""
    t_len, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=F)
    out = torch.zeros(t_len, heads, v.shape[-1], dtype=F)
    for t in range(t_len):
        s = g[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", s, q[t])
    return out


def gated_delta(m, w, p, h, eps):
    t_len = h.shape[0]
    heads, groups, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = short_convolution(h @ w[p + ".q"].t(), w[p + ".q.conv"]).view(t_len, groups, dim)
    k = short_convolution(h @ w[p + ".k"].t(), w[p + ".k.conv"]).view(t_len, groups, dim)
    v = short_convolution(h @ w[p + ".v"].t(), w[p + ".v.conv"]).view(t_len, heads, vdim)
    rep = heads // groups
    q = (unit_vectors(q) * dim ** -0.5).repeat_interleave(rep, 1)
    k = unit_vectors(k).repeat_interleave(rep, 1)
    beta = torch.sigmoid(h @ w[p + ".b"].t())
    o = delta_walk(q, k, v, delta_decays(w, p, h, heads, dim), beta)
    gate = torch.sigmoid(kept(h @ w[p + ".g1"].t()) @ w[p + ".g2"].t())
    return (unit_rms(o, eps) * w[p + ".norm"]).reshape(t_len, -1) * gate


def pair(m, w, p, h, eps):
    """The scales go on what enters the output projections, where an engine rounds (they are linear)."""
    left = kept(float(m["left_scale"]) * window_attention(m["left"], w, p + ".left", h, eps)) @ w[p + ".left.o"].t()
    right = kept(float(m["right_scale"]) * gated_delta(m["right"], w, p + ".right", h, eps)) @ w[p + ".right.o"].t()
    return left + right


# ---- matrix memory ----------------------------------------------------------------------------------------------------
def log_gates(m, w, p, h):
    cap = float(m["gate_cap"])
    i = cap * torch.tanh((h @ w[p + ".i"].t() + w[p + ".i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + ".f"].t() + w[p + ".f.b"]) / cap))
    return i, f


def memory_walk(q, k, v, i, f):
    """q, k [T, heads, dim], v [T, heads, vdim], i, f [T, heads]: the stabilized matrix memory, its maximum from zero."""
    t_len, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=F)
    n = torch.zeros(heads, dim, dtype=F)
    top = torch.zeros(heads, dtype=F)
    out = torch.zeros(t_len, heads, v.shape[-1], dtype=F)
    for t in range(t_len):
        new = torch.maximum(f[t] + top, i[t])
        keep, write = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        s = keep[:, None, None] * s + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out[t] = torch.einsum("hkv,hk->hv", s, q[t]) / den[:, None]
    return out


def matrix_memory(m, w, p, h, eps):
    t_len = h.shape[0]
    heads, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + ".q"].t()).view(t_len, heads, dim) * dim ** -0.5
    k = (h @ w[p + ".k"].t()).view(t_len, heads, dim)
    v = (h @ w[p + ".v"].t()).view(t_len, heads, vdim)
    o = unit_rms(memory_walk(q, k, v, *log_gates(m, w, p, h)), eps).reshape(t_len, -1)
    return kept(o * w[p + ".norm"] * torch.sigmoid(h @ w[p + ".g"].t())) @ w[p + ".o"].t()


# ---- feed-forwards ----------------------------------------------------------------------------------------------------
def clamped_glu(w, p, h, limit):
    g = torch.clamp(h @ w[p + ".gate"].t(), max=limit)
    u = torch.clamp(h @ w[p + ".up"].t(), -limit, limit)
    return kept(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].t()


def route(mlp, w, p, h):
    """Per token: the experts with the largest logits (the first of equal ones) and the softmax over theirs alone."""
    z = h @ w[p + ".router"].t()
    chosen, weights = [], []
    for t in range(h.shape[0]):
        order = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:int(mlp["router"]["top"])]
        chosen.append(order)
        weights.append(torch.softmax(z[t, order], -1))
    return chosen, weights


def mixture(mlp, w, p, h):
    out = torch.zeros_like(h)
    for t, (chosen, weights) in enumerate(zip(*route(mlp, w, p, h))):
        for e, wt in zip(chosen, weights):
            out[t] += wt * clamped_glu(w, f"{p}.e{e}", h[t:t + 1], float(mlp["expert"]["limit"]))[0]
    return out


# ---- streams, layers, model -------------------------------------------------------------------------------------------
def through_streams(xs, w, p, sublayer):
    """xs [streams, T, width]: what the sublayer reads is a sum of the streams; every new stream is a mix of the old ones
    (from, to) plus its share of the sublayer's result."""
    y = sublayer(torch.einsum("s,std->td", w[p + ".in"], xs))
    return torch.einsum("st,sxd->txd", w[p + ".mix"], xs) + w[p + ".out"][:, None, None] * y


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(cfg, w, ids):
    w = {k: v.to(F) for k, v in w.items() if v.is_floating_point()}
    eps = float(cfg["norm"]["eps"])
    xs = w["embed"][torch.as_tensor(ids, dtype=torch.long)].expand(int(cfg["streams"]), -1, -1)
    sums = []
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        mixer = pair if layer["type"] == "parallel" else matrix_memory

        def mix(u):
            return mixer(layer["mixer"], w, p + ".mix", kept(norm_one_plus(u, w[p + ".norm1"], eps)), eps)

        xs = through_streams(xs, w, p + ".hc1", mix)
        mlp = layer.get("mlp")
        if mlp is not None:
            def feed(u):
                h = kept(norm_one_plus(u, w[p + ".norm2"], eps))
                return clamped_glu(w, p + ".mlp", h, float(mlp["limit"])) if mlp["kind"] == "dense" else mixture(mlp, w, p + ".mlp", h)

            xs = through_streams(xs, w, p + ".hc2", feed)
        sums.append(xs.sum(0))
    return kept(norm_one_plus(xs.sum(0), w["final.norm"], eps)) @ w["head"].t(), sums


def logits(cfg, w, ids):
    return forward(cfg, w, ids)[0]
