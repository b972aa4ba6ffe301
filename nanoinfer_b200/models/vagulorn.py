"""``Vagulorn``: a decoder whose layers are listed one by one in config.json. Every layer is a parallel block with ONE layer
norm (weight and bias) whose output both the mixer and the feed-forward read. Mixers:

* ``attention``: softmax attention with a per-head RMS norm of q and k, rotation of the first ``rot.dims`` elements (element i
  paired with i + dims/2) and a chunked mask;
* ``parallel``: softmax attention whose values are the projected keys (per-head norm of q and k, interleaved rotation, a sliding
  window beside kept first tokens, a gate per head) beside lightning attention (a fixed decay per head), summed with the factors
  ``left_scale`` and ``right_scale``;
* ``mamba2``: a state-space mixer with scalar decays per head.

The feed-forward is absent or ``W_down (gelu(W_gate h) * (W_up h))`` with the tanh form of gelu. The embedding is multiplied by
``embedding.scale``; the head is the embedding table without that factor.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers``: a list of ``{"type", "mixer": {...},
"mlp": {"kind": "dense", "ff"} | null}``. ``mixer`` of ``attention``: ``heads kv_heads dim vdim scale mask.size rot.{dims, base}`` (``mask`` may be absent); of
``parallel``: ``left_scale right_scale``, ``left``: the same with ``mask.{size, keep_first}`` (``vdim`` = ``dim``), ``right``: ``heads dim vdim
decay`` (a list, one per head); of ``mamba2``: ``heads vdim state groups norm_groups conv``.

Tensor names: ``embed``, ``final.norm``, ``final.norm.b``, per layer i ``l<i>.norm1``, ``l<i>.norm1.b``, ``l<i>.mix.{q k v o q.norm k.norm}``
(``attention``), ``l<i>.mix.left.{q k o g q.norm k.norm}``, ``l<i>.mix.right.{q k v g o norm}``, ``l<i>.mix.{in conv conv.b dt_bias A_log D norm
o}`` (``mamba2``), ``l<i>.mlp.{gate up down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Tuple

from ..config.model_config import ConfigError, ModelConfig
from ..parts.embedding import LinearHead, TokenEmbedding
from ..parts.feedforward import SwiGLU
from ..parts.flex_attention import FlexAttention
from ..parts.linear_state import LightningAttention, Mamba2Mixer
from ..parts.norm import LayerNorm
from ..parts.side_by_side import SideBySide
from ..parts.spec import LayerSpec, ModelPlan, ScheduleEntry
from ..registry import register_architecture

_MIXERS = ("attention", "parallel", "mamba2")
# Positions are turned into angles in 32-bit floats, which hold every integer up to 2^24.
_MAX_POSITIONS = 1 << 24


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


def _check_softmax(m: Mapping[str, Any], where: str, values_are_keys: bool) -> None:
    if _int(m, "heads", where) % _int(m, "kv_heads", where):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    dim = _int(m, "dim", where)
    if "vdim" in m and _int(m, "vdim", where) != dim and values_are_keys:
        raise ConfigError(f"config.json: {where}.vdim must equal dim: the values are the projected keys")
    _num(m, "scale", where, positive=False)
    rot = _obj(m, "rot", where)
    dims = _int(rot, "dims", where + ".rot")
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    _num(rot, "base", where + ".rot")
    if m.get("mask") is not None:       # without one every earlier position is seen
        mask = _obj(m, "mask", where)
        _int(mask, "size", where + ".mask")
        if mask.get("keep_first") is not None:
            _int(mask, "keep_first", where + ".mask", least=0)


def _check_lightning(m: Mapping[str, Any], where: str) -> None:
    heads = _int(m, "heads", where)
    _int(m, "dim", where)
    if "vdim" in m:
        _int(m, "vdim", where)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != heads \
            or any(isinstance(d, bool) or not isinstance(d, (int, float)) or not 0 <= d <= 1 for d in decay):
        raise ConfigError(f"config.json: {where}.decay must be a list of {heads} numbers between 0 and 1, one per head")


@dataclass(frozen=True)
class VagulornConfig(ModelConfig):
    layers: Tuple[dict, ...] = ()
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0

    @classmethod
    def from_json_dict(cls, d: Mapping[str, Any]) -> "VagulornConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        eps = _num(_obj(d, "norm", "config"), "eps", "norm")
        scale = 1.0 if d.get("embedding") is None else _num(_obj(d, "embedding", "config"), "scale", "embedding", positive=False)
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {_MIXERS}")
            m = _obj(layer, "mixer", where)
            where += ".mixer"
            if layer["type"] == "mamba2":
                for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv"):
                    _int(m, k, where)
                if m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]:
                    raise ConfigError(f"config.json: {where}: heads must be a multiple of groups, heads * vdim of norm_groups")
            elif layer["type"] == "attention":
                _check_softmax(m, where, values_are_keys=False)
            else:
                _check_softmax(_obj(m, "left", where), where + ".left", values_are_keys=True)
                _check_lightning(_obj(m, "right", where), where + ".right")
                _num(m, "left_scale", where, positive=False)
                _num(m, "right_scale", where, positive=False)
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: layers[{i}].mlp must be null or of kind 'dense'")
                _int(mlp, "ff", f"layers[{i}].mlp")
        eos = d.get("eos_token_id")
        return cls(architecture=str(d.get("architecture") or "Vagulorn"), model_type="vagulorn",
                   vocab_size=_int(d, "vocab", "config"), hidden_size=_int(d, "width", "config"),
                   num_hidden_layers=len(layers), max_position_embeddings=_MAX_POSITIONS, tie_word_embeddings=True,
                   eos_token_id=int(eos) if isinstance(eos, int) and not isinstance(eos, bool) else -1,
                   layers=tuple(layers), norm_eps=eps, embedding_scale=scale)

    def to_json_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
             "layers": [dict(layer) for layer in self.layers]}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d


def _softmax_dims(m: Mapping[str, Any]):
    return int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), float(m["scale"])


def _rot(m: Mapping[str, Any]):
    return int(m["rot"]["dims"]), float(m["rot"]["base"])


def _mask(m: Mapping[str, Any]):
    """(size, kept first tokens) of a mixer's mask; size 0 without one."""
    mask = m.get("mask")
    return (0, 0) if mask is None else (int(mask["size"]), int(mask.get("keep_first") or 0))


def _mixer(prefix: str, hidden: int, kind: str, m: Mapping[str, Any], eps: float):
    if kind == "mamba2":
        return Mamba2Mixer.spec(prefix, hidden, int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["norm_groups"]),
                                int(m["conv"]), eps)
    if kind == "attention":
        return FlexAttention.spec(prefix, hidden, *_softmax_dims(m), eps, qk_norm=True, rot=_rot(m), chunk=_mask(m)[0])
    left, right = m["left"], m["right"]
    window, keep_first = _mask(left)
    return SideBySide.spec(
        FlexAttention.spec(f"{prefix}.left", hidden, *_softmax_dims(left), eps, qk_norm=True, rot=_rot(left), rot_layout="interleaved",
                           values_from_keys=True, window=window, keep_first=keep_first,
                           out_gate="head", out_scale=float(m["left_scale"])),
        LightningAttention.spec(f"{prefix}.right", hidden, int(right["heads"]), int(right["dim"]), int(right.get("vdim", right["dim"])),
                                right["decay"], eps, float(m["right_scale"])))


def vagulorn_plan(cfg: VagulornConfig) -> ModelPlan:
    h, eps = cfg.hidden_size, cfg.norm_eps
    layers: List[LayerSpec] = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        parts = {"mixer_norm": LayerNorm.spec(h, eps, f"{p}.norm1", f"{p}.norm1.b"),
                 "mixer": _mixer(f"{p}.mix", h, layer["type"], layer["mixer"], eps)}
        if layer.get("mlp") is not None:
            parts["ffn"] = SwiGLU.spec(f"{p}.mlp", h, int(layer["mlp"]["ff"]), names=("gate", "up", "down"), act="gelu_tanh")
        layers.append(LayerSpec("parallel", parts))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=h, vocab_size=cfg.vocab_size, max_position_embeddings=cfg.max_position_embeddings,
        embedding=TokenEmbedding.spec("embed", cfg.vocab_size, h, cfg.embedding_scale), positions={}, layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))],
        final_norm=LayerNorm.spec(h, eps, "final.norm", "final.norm.b"), lm_head=LinearHead.spec("embed", cfg.vocab_size, h),
        eos_token_id=cfg.eos_token_id)


register_architecture("Vagulorn", VagulornConfig, vagulorn_plan)
