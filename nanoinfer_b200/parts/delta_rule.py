"""Delta rules: recurrent mixers with a matrix state per head that take what the state already answers off before they write.

``GeneralizedDeltaRule``: with ``r, k, v`` the head's projections of the token (``d`` elements each), a decay per key channel
``w = exp(-exp(-1/2) * sigmoid(W_w2 tanh(W_w1 h) + w0))``, a removal rate per key channel ``a = sigmoid(W_a h + b_a)``
and the unit key ``u = k / sqrt(sum(k^2) + 1e-6)``, the state ``S`` (key channel x value channel, zero at the start of
a request, 32-bit) moves as

    S <- diag(w) S - (a * u)(u^T S) + k v^T        (both products read the old S),        o = S^T r.

Each head's ``o`` is divided by its root mean square, multiplied by a gain (all heads' size) and by
``sigmoid(W_g h)``; then ``W_o``, added to the residual stream. Everything that enters the recurrence is 32-bit: the
projections leave the matrix kernels as floats.

``GatedDeltaRule``: q and k (``kv_heads`` heads, shared by groups of heads) and v pass a short causal convolution per channel
(``conv`` taps, zeros before a request's start) and silu; q and k become unit vectors per head
(``x / sqrt(sum(x^2) + 1e-6)``), q times ``dim^(-1/2)``; ``beta = sigmoid(W_b h)`` per head; the decay per head and key channel
is ``w = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias))``. Per head

    S <- diag(w) S,        u = beta (v - S^T k),        S <- S + k u^T,        o = S^T q,

then ``o`` is divided by its root mean square, times a gain of ``vdim`` shared by the heads, times ``sigmoid(W_g2 W_g1 h)``,
then ``W_o``; ``out_scale`` times the result is added to the residual stream. The state of a request is S and the
convolution's last ``conv - 1`` inputs, 32-bit.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..registry import register_part
from .base import LayerCache, Mixer, ProjectedMixer, Runtime, StateNeed, StepContext
from .spec import PartSpec, TensorSpec


class GeneralizedDeltaRule(Mixer):
    """params: ``hidden``, ``heads``, ``dim``, ``decay_rank`` (inner width of the decay's two-layer map), ``eps``
    (of the per-head norm). tensors: ``r k v g a [heads*dim, hidden]``, ``a_b``, ``w1 [decay_rank, hidden]``,
    ``w2 [heads*dim, decay_rank]``, ``w0``, ``norm [heads*dim]``, ``o [hidden, heads*dim]``."""

    graph_safe = True   # launches do not depend on which requests are in the batch

    @staticmethod
    def spec(prefix: str, hidden: int, heads: int, dim: int, decay_rank: int, eps: float) -> PartSpec:
        n = heads * dim
        t = {name: TensorSpec(f"{prefix}.{name}", (n, hidden)) for name in ("r", "k", "v", "g", "a")}
        t["a_b"] = TensorSpec(f"{prefix}.a.b", (n,), "bias")
        t["w1"] = TensorSpec(f"{prefix}.w1", (decay_rank, hidden))
        t["w2"] = TensorSpec(f"{prefix}.w2", (n, decay_rank))
        t["w0"] = TensorSpec(f"{prefix}.w0", (n,), "unit")
        t["norm"] = TensorSpec(f"{prefix}.norm", (n,), "gain")
        t["o"] = TensorSpec(f"{prefix}.o", (hidden, n))
        return PartSpec("general_delta", {"hidden": hidden, "heads": heads, "dim": dim, "decay_rank": decay_rank, "eps": eps}, t)

    def __init__(self, spec: PartSpec, tensors: Dict[str, torch.Tensor], rt: Runtime):
        super().__init__(spec, tensors, rt)
        p = spec.params
        self.hidden, self.heads, self.dim = int(p["hidden"]), int(p["heads"]), int(p["dim"])
        self.decay_rank, self.eps = int(p["decay_rank"]), float(p["eps"])
        n = self.n = self.heads * self.dim
        # One product for everything that reads h: rows [r | k | v | a | g | w1]; only a has a bias.
        self.w_in = rt.matrix(torch.cat([tensors[x] for x in ("r", "k", "v", "a", "g", "w1")], dim=0))
        bias = torch.zeros(5 * n + self.decay_rank, dtype=torch.float32)
        bias[3 * n:4 * n] = tensors["a_b"].to(torch.float32)
        self.b_in = rt.vector32(bias)
        self.w_2, self.w_0 = rt.matrix(tensors["w2"]), rt.vector32(tensors["w0"])
        self.gain = rt.vector32(tensors["norm"])
        self.w_o = rt.matrix(tensors["o"])

    def state_need(self) -> StateNeed:
        # per head [value channel, key channel]: a value column's key channels lie together
        return StateNeed((self.heads, self.dim, self.dim), torch.float32)

    def forward(self, h: torch.Tensor, residual32: torch.Tensor, ctx: StepContext, cache: LayerCache) -> None:
        m, dev, n, ops = h.shape[0], h.device, self.n, self.ops
        p32 = torch.empty((m, 5 * n + self.decay_rank), dtype=torch.float32, device=dev)
        ops.linear(h, self.w_in, self.b_in, p32, "f32")
        inner = torch.empty((m, self.decay_rank), dtype=self.rt.dtype, device=dev)
        ops.unary(p32[:, 5 * n:], inner, "tanh")
        w_logit = torch.empty((m, n), dtype=torch.float32, device=dev)
        ops.linear(inner, self.w_2, self.w_0, w_logit, "f32")
        o32 = torch.empty((m, n), dtype=torch.float32, device=dev)
        ops.delta_rule_scan(p32[:, :n], p32[:, n:2 * n], p32[:, 2 * n:3 * n], p32[:, 3 * n:4 * n], w_logit, cache.state,
                            ctx, o32, self.heads, self.dim)
        gated = torch.empty((m, n), dtype=self.rt.dtype, device=dev)
        ops.head_norm_gate(o32, p32[:, 4 * n:5 * n], self.gain, self.eps, self.heads, self.dim, gated)
        ops.linear(gated, self.w_o, None, residual32, "add")


class GatedDeltaRule(ProjectedMixer):
    """params: ``hidden heads kv_heads dim vdim conv decay_rank gate_rank eps out_scale``, optionally ``joint_input``.
    tensors: ``q k [kv_heads*dim, hidden]``,
    ``v [heads*vdim, hidden]``, ``q_conv k_conv v_conv [channels, conv]`` (last column = the current token), ``b [heads, hidden]``,
    ``a1 [decay_rank, hidden]``, ``a2 [heads*dim, decay_rank]``, ``A_log [heads]``, ``dt_bias [heads*dim]``, ``g1 [gate_rank, hidden]``,
    ``g2 [heads*vdim, gate_rank]``, ``norm [vdim]``, ``o [hidden, heads*vdim]``."""

    graph_safe = True   # launches do not depend on which requests are in the batch
    UNIT_EPS = 1e-6

    @staticmethod
    def spec(prefix: str, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, decay_rank: int, gate_rank: int,
             eps: float, out_scale: float = 1.0) -> PartSpec:
        nq, nk, nv = kv_heads * dim, heads * dim, heads * vdim
        t = {}
        for name, n in (("q", nq), ("k", nq), ("v", nv)):
            t[name] = TensorSpec(f"{prefix}.{name}", (n, hidden))
            t[name + "_conv"] = TensorSpec(f"{prefix}.{name}.conv", (n, conv), "unit")
        t.update({"b": TensorSpec(f"{prefix}.b", (heads, hidden)),
                  "a1": TensorSpec(f"{prefix}.a1", (decay_rank, hidden)), "a2": TensorSpec(f"{prefix}.a2", (nk, decay_rank)),
                  "A_log": TensorSpec(f"{prefix}.A_log", (heads,), "unit"), "dt_bias": TensorSpec(f"{prefix}.dt_bias", (nk,), "unit"),
                  "g1": TensorSpec(f"{prefix}.g1", (gate_rank, hidden)), "g2": TensorSpec(f"{prefix}.g2", (nv, gate_rank)),
                  "norm": TensorSpec(f"{prefix}.norm", (vdim,), "gain"), "o": TensorSpec(f"{prefix}.o", (hidden, nv))})
        return PartSpec("gated_delta", {"hidden": hidden, "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": int(conv),
                                        "decay_rank": decay_rank, "gate_rank": gate_rank, "eps": float(eps), "out_scale": float(out_scale)}, t)

    def __init__(self, spec: PartSpec, tensors: Dict[str, torch.Tensor], rt: Runtime):
        super().__init__(spec, tensors, rt)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim, self.taps = int(p["dim"]), int(p["vdim"]), int(p["conv"])
        if self.heads % self.kv_heads:
            raise ValueError(f"heads ({self.heads}) must be a multiple of kv_heads ({self.kv_heads})")
        self.eps, self.out_scale = float(p["eps"]), float(p.get("out_scale", 1.0))
        self.nq, self.nk, self.nv = self.kv_heads * self.dim, self.heads * self.dim, self.heads * self.vdim
        self.n_conv = 2 * self.nq + self.nv
        ra, rg = int(p["decay_rank"]), int(p["gate_rank"])
        # One product for everything that reads h: rows [q | k | v | a1 | g1 | zeros | b | zeros]. The inner vectors of decay
        # and gate lie together, filled up to a width that every matrix kernel takes (a zero channel adds nothing).
        self.inner = -(-(ra + rg) // 32) * 32
        fill = lambda n: torch.zeros((n, self.hidden), dtype=tensors["b"].dtype)
        self.b_col = self.n_conv + self.inner
        rows = [tensors[x] for x in ("q", "k", "v", "a1", "g1")] + [fill(self.inner - ra - rg), tensors["b"]]
        width = -(-(self.b_col + self.heads) // 4) * 4
        self.take_input(torch.cat(rows + [fill(width - self.b_col - self.heads)], dim=0), None, bool(p.get("joint_input")))
        # One product for both second layers: [a2 | 0 ; 0 | g2].
        w2 = torch.zeros((self.nk + self.nv, self.inner), dtype=tensors["a2"].dtype)
        w2[:self.nk, :ra] = tensors["a2"]
        w2[self.nk:, ra:ra + rg] = tensors["g2"]
        self.w_2 = rt.matrix(w2)
        self.conv_w = rt.vector32(torch.cat([tensors[n + "_conv"] for n in ("q", "k", "v")], dim=0))
        self.rate, self.dt_bias = rt.vector32(torch.exp(tensors["A_log"].double()).to(torch.float32)), rt.vector32(tensors["dt_bias"])
        self.gain = rt.vector32(tensors["norm"])
        self.w_o = rt.matrix(tensors["o"])
        self.conv_state = (self.taps - 1) * self.n_conv

    def state_need(self) -> StateNeed:
        # [the convolution's last taps-1 inputs | S as [head, value channel, key channel]]
        return StateNeed((self.conv_state + self.heads * self.vdim * self.dim,), torch.float32)

    def mix(self, p32: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        m, dev, ops, nq, nk, nv = p32.shape[0], p32.device, self.ops, self.nq, self.nk, self.nv
        qkv = torch.empty((m, self.n_conv), dtype=torch.float32, device=dev)
        ops.conv_step(p32[:, :self.n_conv], self.conv_w, None, "silu", cache.state, 0, ctx, qkv, self.taps)
        inner = torch.empty((m, self.inner), dtype=self.rt.dtype, device=dev)
        ops.unary(p32[:, self.n_conv:self.b_col], inner, "copy")
        zg = torch.empty((m, nk + nv), dtype=torch.float32, device=dev)
        ops.linear(inner, self.w_2, None, zg, "f32")
        o32 = torch.empty((m, nv), dtype=torch.float32, device=dev)
        ops.grouped_state_scan(qkv[:, :nq], qkv[:, nq:2 * nq], qkv[:, 2 * nq:], zg[:, :nk], cache.state, self.conv_state, ctx, o32, self.heads,
                               self.kv_heads, self.dim, self.vdim, beta32=p32[:, self.b_col:self.b_col + self.heads], rate32=self.rate,
                               dt_bias32=self.dt_bias, q_scale=self.dim ** -0.5, unit_eps=self.UNIT_EPS)
        gated = torch.empty((m, nv), dtype=self.rt.dtype, device=dev)
        ops.gated_norm(o32, gated, groups=self.heads, eps=self.eps, gain32=self.gain, gate32=zg[:, nk:], gate_kind="sigmoid",
                       out_scale=self.out_scale)
        return gated


register_part("general_delta", GeneralizedDeltaRule)
register_part("gated_delta", GatedDeltaRule)
