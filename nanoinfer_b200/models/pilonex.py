"""``Pilonex``: a decoder with several residual streams, whose layers are listed one by one in config.json and of which a
stretch may run several times with the same weights (every pass with a cache or state of its own). A sublayer reads a norm
(gain stored around zero) of a weighted sum of the streams, and its result goes back to all of them (``parts/streams.py``).
Mixers:

* ``parallel``: softmax attention (per-head norm of q and k, rotation of the first ``rot.dims`` elements with rescaled
  frequencies, a sliding window) beside the gated delta rule (short convolutions, unit keys, a decay per key channel), summed
  with the factors ``left_scale`` and ``right_scale``;
* ``mlstm``: a stabilized matrix memory with exponential gates.

The feed-forward is absent, dense or a mixture of experts; both use the clamped gated form
``min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u) + 1)``; the router's weights are the softmax over the chosen logits. The head is a
matrix of its own.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``streams``, ``loop`` (null or ``{start, stop, times}``: layers start .. stop-1
run ``times`` times), ``layers``: a list of ``{"type", "mixer", "mlp"}``. ``mixer`` of ``parallel``: ``left_scale right_scale``, ``left``: ``heads kv_heads dim vdim scale
mask.size rot.{dims, base, scaling.{factor, low, high, original}}``, ``right``: ``heads kv_heads dim vdim conv`` (the inner widths of its
decay and gate maps are the row counts of its ``a1`` and ``g1`` tensors, or ``decay_rank`` and ``gate_rank``, which the random-weights
mode writes); of ``mlstm``: ``heads dim vdim gate_cap``. ``mlp``: null, ``{"kind": "dense", "ff", "limit"}`` or ``{"kind": "moe", "expert": {"ff", "limit"},
"router": {"experts", "top"}}``.

Tensor names: ``embed``, ``head``, ``final.norm``, per layer i ``l<i>.norm1 norm2``, ``l<i>.hc1.{in out mix}``, ``l<i>.hc2.{in out mix}``,
``l<i>.mix.left.{q k v o q.norm k.norm}``, ``l<i>.mix.right.{q k v q.conv k.conv v.conv b A_log a1 a2 dt_bias g1 g2 norm o}``, ``l<i>.mix.{q k v g i i.b
f f.b norm o}`` (``mlstm``), ``l<i>.mlp.{gate up down}`` (dense) or ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate up down}``.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, List, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, ModelConfig
from ..parts.delta_rule import GatedDeltaRule
from ..parts.embedding import LinearHead, TokenEmbedding
from ..parts.feedforward import RoutedExperts, SwiGLU
from ..parts.flex_attention import FlexAttention
from ..parts.linear_state import StabilizedMatrixMemory
from ..parts.norm import RMSNorm
from ..parts.side_by_side import SideBySide
from ..parts.spec import LayerSpec, ModelPlan, ScheduleEntry
from ..parts.streams import StreamMix
from ..registry import register_architecture

_MIXERS = ("parallel", "mlstm")
# Positions are turned into angles in 32-bit floats, which hold every integer up to 2^24.
_MAX_POSITIONS = 1 << 24
_MAX_STREAMS = 16
# Of the clamped gated form g sigmoid(alpha g) (u + shift).
_GLU_ALPHA, _GLU_SHIFT = 1.702, 1.0
# The inner widths of a delta rule's two-layer maps: config key -> the tensor whose row count gives it.
_RANKS = {"decay_rank": "a1", "gate_rank": "g1"}


def _int(d: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"config.json: {where}.{key} must be an integer of at least {least}, got {v!r}")
    return v


def _num(d: Mapping[str, Any], key: str, where: str, positive: bool = True) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"config.json: {where}.{key} must be a {'positive ' if positive else ''}number, got {v!r}")
    return float(v)


def _obj(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _heads(m: Mapping[str, Any], where: str) -> None:
    if _int(m, "heads", where) % _int(m, "kv_heads", where):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _int(m, "dim", where)
    if "vdim" in m:
        _int(m, "vdim", where)


def _check_left(m: Mapping[str, Any], where: str) -> None:
    _heads(m, where)
    _num(m, "scale", where)
    if m.get("mask") is not None:
        _int(_obj(m, "mask", where), "size", where + ".mask")
    rot = _obj(m, "rot", where)
    dims = _int(rot, "dims", where + ".rot")
    if dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    _num(rot, "base", where + ".rot")
    if rot.get("scaling") is not None:
        sc = _obj(rot, "scaling", where + ".rot")
        for k in ("factor", "low", "high", "original"):
            _num(sc, k, where + ".rot.scaling")
        if sc["low"] > sc["high"]:
            raise ConfigError(f"config.json: {where}.rot.scaling.low must be at most high")


def _check_mlp(mlp: Any, where: str) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where} must be null or of kind 'dense' or 'moe'")
    if mlp["kind"] == "dense":
        _int(mlp, "ff", where)
        _num(mlp, "limit", where)
        return
    expert, router = _obj(mlp, "expert", where), _obj(mlp, "router", where)
    _int(expert, "ff", where + ".expert")
    _num(expert, "limit", where + ".expert")
    if _int(router, "top", where + ".router") > _int(router, "experts", where + ".router"):
        raise ConfigError(f"config.json: {where}.router.top must be at most experts")


@dataclass(frozen=True)
class PilonexConfig(ModelConfig):
    layers: Tuple[dict, ...] = ()
    norm_eps: float = 1e-6
    streams: int = 1
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)

    @classmethod
    def from_json_dict(cls, d: Mapping[str, Any]) -> "PilonexConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        eps = _num(_obj(d, "norm", "config"), "eps", "norm")
        streams = _int(d, "streams", "config")
        if streams > _MAX_STREAMS:
            raise ConfigError(f"config.json: config.streams must be at most {_MAX_STREAMS}")
        loop = None
        if d.get("loop") is not None:
            lp = _obj(d, "loop", "config")
            loop = (_int(lp, "start", "loop", least=0), _int(lp, "stop", "loop", least=0), _int(lp, "times", "loop"))
            if not (loop[0] <= loop[1] <= len(layers)):
                raise ConfigError("config.json: loop needs start <= stop <= the number of layers")
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {_MIXERS}")
            m = _obj(layer, "mixer", where)
            where += ".mixer"
            if layer["type"] == "mlstm":
                for k in ("heads", "dim"):
                    _int(m, k, where)
                if "vdim" in m:
                    _int(m, "vdim", where)
                _num(m, "gate_cap", where)
            else:
                _check_left(_obj(m, "left", where), where + ".left")
                r = _obj(m, "right", where)
                _heads(r, where + ".right")
                _int(r, "conv", where + ".right")
                for k in _RANKS:
                    if k in r:
                        _int(r, k, where + ".right")
                _num(m, "left_scale", where, positive=False)
                _num(m, "right_scale", where, positive=False)
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"layers[{i}].mlp")
        eos = d.get("eos_token_id")
        return cls(architecture=str(d.get("architecture") or "Pilonex"), model_type="pilonex",
                   vocab_size=_int(d, "vocab", "config"), hidden_size=_int(d, "width", "config"),
                   num_hidden_layers=len(layers), max_position_embeddings=_MAX_POSITIONS, tie_word_embeddings=False,
                   eos_token_id=int(eos) if isinstance(eos, int) and not isinstance(eos, bool) else -1,
                   layers=tuple(layers), norm_eps=eps, streams=streams, loop=loop)

    def with_tensor_shapes(self, shapes: Mapping[str, Any]) -> "PilonexConfig":
        """The inner widths of a delta rule's decay and gate maps are the row counts of their first matrices; config.json
        need not state them."""
        layers = []
        for i, layer in enumerate(self.layers):
            if layer["type"] == "parallel":
                right = dict(layer["mixer"]["right"])
                for key, tensor in _RANKS.items():
                    name = f"l{i}.mix.right.{tensor}"
                    if key not in right and name in shapes:
                        right[key] = int(tuple(shapes[name])[0])
                layer = dict(layer, mixer=dict(layer["mixer"], right=right))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def run_order(self) -> List[int]:
        """The layers in the order in which they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def to_json_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
             "streams": self.streams, "loop": None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop)),
             "layers": [dict(layer) for layer in self.layers]}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d


def _pair(prefix: str, hidden: int, m: Mapping[str, Any], eps: float):
    left, right = m["left"], m["right"]
    for key, tensor in _RANKS.items():
        if key not in right:
            raise ConfigError(f"{prefix}.right: the inner width of a two-layer map is given neither by '{key}' nor by the shape of "
                              f"'{prefix}.right.{tensor}'")
    rot = left["rot"]
    return SideBySide.spec(
        FlexAttention.spec(f"{prefix}.left", hidden, int(left["heads"]), int(left["kv_heads"]), int(left["dim"]), int(left.get("vdim", left["dim"])),
                           float(left["scale"]), eps, qk_norm=True, rot=(int(rot["dims"]), float(rot["base"])), rot_scaling=rot.get("scaling"),
                           window=0 if left.get("mask") is None else int(left["mask"]["size"]), out_scale=float(m["left_scale"])),
        GatedDeltaRule.spec(f"{prefix}.right", hidden, int(right["heads"]), int(right["kv_heads"]), int(right["dim"]),
                            int(right.get("vdim", right["dim"])), int(right["conv"]), int(right["decay_rank"]), int(right["gate_rank"]), eps,
                            float(m["right_scale"])))


def _feed_forward(prefix: str, hidden: int, mlp: Mapping[str, Any]):
    if mlp["kind"] == "dense":
        return SwiGLU.spec(prefix, hidden, int(mlp["ff"]), names=("gate", "up", "down"), glu=(_GLU_ALPHA, float(mlp["limit"]), _GLU_SHIFT))
    # the softmax over all logits, renormalized over the chosen ones, is the softmax over the chosen logits
    return RoutedExperts.spec(prefix, hidden, int(mlp["expert"]["ff"]), int(mlp["router"]["experts"]), int(mlp["router"]["top"]), score="softmax",
                              renormalize=True, weight_on="output", glu=(_GLU_ALPHA, float(mlp["expert"]["limit"]), _GLU_SHIFT))


def pilonex_plan(cfg: PilonexConfig) -> ModelPlan:
    h, eps = cfg.hidden_size, cfg.norm_eps
    layers: List[LayerSpec] = []
    ignored: List[str] = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer["mixer"]
        if layer["type"] == "mlstm":
            mixer = StabilizedMatrixMemory.spec(f"{p}.mix", h, int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), float(m["gate_cap"]), eps)
        else:
            mixer = _pair(f"{p}.mix", h, m, eps)
        parts = {"mixer_norm": RMSNorm.spec(h, eps, f"{p}.norm1", gain_offset=1.0), "mixer": mixer,
                 "mixer_streams": StreamMix.spec(f"{p}.hc1", cfg.streams)}
        if layer.get("mlp") is not None:
            parts["ffn_norm"] = RMSNorm.spec(h, eps, f"{p}.norm2", gain_offset=1.0)
            parts["ffn"] = _feed_forward(f"{p}.mlp", h, layer["mlp"])
            parts["ffn_streams"] = StreamMix.spec(f"{p}.hc2", cfg.streams)
        else:       # no feed-forward: no use for its norm and factors, should a checkpoint hold them
            ignored += [f"{p}.norm2"] + [f"{p}.hc2.{n}" for n in ("in", "out", "mix")]
        layers.append(LayerSpec("multi_stream", parts))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=h, vocab_size=cfg.vocab_size, max_position_embeddings=cfg.max_position_embeddings,
        embedding=TokenEmbedding.spec("embed", cfg.vocab_size, h), positions={}, layers=layers,
        schedule=[ScheduleEntry(i) for i in cfg.run_order()],
        final_norm=RMSNorm.spec(h, eps, "final.norm", gain_offset=1.0), lm_head=LinearHead.spec("head", cfg.vocab_size, h),
        eos_token_id=cfg.eos_token_id, ignored_tensors=tuple(ignored))


register_architecture("Pilonex", PilonexConfig, pilonex_plan)
