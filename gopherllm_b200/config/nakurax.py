"""The Nakurax design: a decoder with several residual streams (hyper-connections) whose layers mix tokens by attention
through a latent without positions, or by a chunked softmax attention beside a gated linear recurrence; a range of
layers may run several times.

config.json lists the layers one by one: ``layers[i].type`` is ``latent_attention`` or ``parallel``, ``layers[i].mixer``
the mixer's sizes and constants, ``layers[i].mlp`` a dense feed-forward or null.  ``loop``: the range start .. stop-1 is
passed ``times`` times before what follows it, every pass on cache entries of its own.  The scaled embedding fills
``streams`` equal streams; a sublayer reads a weighted sum of them and joins them all at once (see parts/block.py,
StreamsBlock), in front of it an RMS norm with a weight; the final norm reads the streams' sum, the head has weights
of its own.

  latent_attention  see parts/attention.py (LatentAttention): queries straight from the input, a normed latent of
                    kv_rank numbers per position, H heads of dim and vdim, no rotation, every earlier position is seen
  parallel          left_scale * left(h) + right_scale * right(h).  left: grouped-query attention without biases, the
                    first rot.dims dims of every head of q and k turned (dim 2i with dim 2i + 1), with rot.scaling at
                    frequencies stretched band by band; score = q . k * scale; a query sees its own chunk of mask.size
                    positions.  right: see parts/recurrent.py (GatedLinearUnit).
  dense             W_down relu(W_up h)^2, no biases

Every size and every constant that differs between models comes from config.json.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Optional

from .registry import Architecture, register_architecture
from .specs import (BlockSpec, FeedForwardSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, default_schedule,
                    looped_schedule)

# the design sets no longest sequence; the cache's size bounds one
UNBOUNDED_POSITIONS = 1 << 20
# factor of the recurrence's log decay
DECAY = 8.0


def _int(where: str, d: dict, key: str, least: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ValueError(f"config.json: {where}.{key} must be an integer of at least {least}, is {v!r}")
    return v


def _number(where: str, d: dict, key: str, positive: bool = True) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (positive and not v > 0):
        raise ValueError(f"config.json: {where}.{key} must be a {'positive ' if positive else ''}number, is {v!r}")
    return float(v)


def _object(where: str, d: dict, key: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ValueError(f"config.json: {where}.{key} must be an object")
    return v


@dataclass
class NakuraxConfig:
    """Typed view of a Nakurax config.json (key names are the file's own)."""
    vocab: int
    width: int
    layers: list
    norm_eps: float
    streams: int
    embedding_scale: float = 1.0
    loop: Optional[dict] = None
    architecture: str = "Nakurax"
    torch_dtype: str = "bfloat16"
    initializer_range: float = 0.05

    @classmethod
    def from_dict(cls, d: dict) -> "NakuraxConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm", "streams") if k not in d]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        embedding = _object("config", d, "embedding") if d.get("embedding") is not None else {}
        cfg = cls(vocab=_int("config", d, "vocab"), width=_int("config", d, "width"), layers=copy.deepcopy(d["layers"]),
                  norm_eps=_number("norm", _object("config", d, "norm"), "eps"), streams=_int("config", d, "streams"),
                  embedding_scale=_number("embedding", embedding, "scale", positive=False) if "scale" in embedding else 1.0,
                  loop=copy.deepcopy(d.get("loop")), architecture=str(d.get("architecture", "Nakurax")),
                  torch_dtype=str(d.get("torch_dtype", d.get("dtype", "bfloat16"))),
                  initializer_range=float(d.get("initializer_range", 0.05)))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps}, "streams": self.streams,
               "embedding": {"scale": self.embedding_scale}, "torch_dtype": self.torch_dtype,
               "initializer_range": self.initializer_range}
        if self.loop is not None:
            out["loop"] = copy.deepcopy(self.loop)
        return out

    def validate(self) -> None:
        if not isinstance(self.layers, list) or not self.layers:
            raise ValueError("config.json: layers must be a non-empty list")
        nakurax_model_spec(self)            # raises on anything a part or the schedule cannot take


def _rotation(where: str, m: dict, dim: int) -> PositionSpec:
    if m.get("rot") is None:
        return PositionSpec("none")
    rot = _object(where, m, "rot")
    where += ".rot"
    dims = rot.get("dims", 0)
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > dim:
        raise ValueError(f"config.json: {where}.dims must be even and at most {dim}, is {dims!r}")
    if dims == 0:
        return PositionSpec("none")
    extra = [("exact_angles", True)]
    if rot.get("scaling") is not None:
        s = _object(where, rot, "scaling")
        factor, low, high, original = (_number(where + ".scaling", s, k) for k in ("factor", "low", "high", "original"))
        if high < low:
            raise ValueError(f"config.json: {where}.scaling.high must not be less than low, {high} < {low}")
        extra.append(("bands", (factor, low, high, original)))
    return PositionSpec("rope", dims, _number(where, rot, "base"), interleaved=True, extra=tuple(extra))


def _latent_attention(cfg: NakuraxConfig, m: dict, where: str) -> MixerSpec:
    return MixerSpec(kind="latent_attention", hidden=cfg.width, num_heads=_int(where, m, "heads"), num_kv_heads=1,
                     head_dim=_int(where, m, "dim"), value_dim=_int(where, m, "vdim"), q_scale=1.0, bias=False,
                     extra=(("kv_rank", _int(where, m, "kv_rank")), ("score_scale", _number(where, m, "scale", positive=False)),
                            ("norm_eps", cfg.norm_eps)))


def _chunked_attention(cfg: NakuraxConfig, m: dict, where: str) -> MixerSpec:
    heads, kv = _int(where, m, "heads"), _int(where, m, "kv_heads")
    if heads % kv:
        raise ValueError(f"config.json: {where}.heads {heads} is not a multiple of kv_heads {kv}")
    dim = _int(where, m, "dim")
    extra = [("score_scale", _number(where, m, "scale", positive=False))]
    if m.get("mask") is not None:
        extra.append(("chunk", _int(where + ".mask", _object(where, m, "mask"), "size")))
    return MixerSpec(kind="attention_mixed", hidden=cfg.width, num_heads=heads, num_kv_heads=kv, head_dim=dim,
                     value_dim=_int(where, m, "vdim"), q_scale=1.0, bias=False, position=_rotation(where, m, dim),
                     extra=tuple(extra))


def _recurrent(cfg: NakuraxConfig, m: dict, where: str) -> MixerSpec:
    width, blocks = _int(where, m, "width"), _int(where, m, "blocks")
    if width % blocks:
        raise ValueError(f"config.json: {where}.width {width} does not form {blocks} equal blocks")
    return MixerSpec(kind="gated_linear_unit", hidden=cfg.width, bias=True,
                     extra=(("width", width), ("blocks", blocks), ("conv", _int(where, m, "conv")), ("decay", DECAY)))


def _parallel(cfg: NakuraxConfig, m: dict, where: str) -> MixerSpec:
    return MixerSpec(kind="scaled_pair", hidden=cfg.width, bias=False,
                     extra=(("left", _chunked_attention(cfg, _object(where, m, "left"), where + ".left")),
                            ("right", _recurrent(cfg, _object(where, m, "right"), where + ".right")),
                            ("left_scale", _number(where, m, "left_scale", positive=False)),
                            ("right_scale", _number(where, m, "right_scale", positive=False))))


_MIXERS = {"latent_attention": _latent_attention, "parallel": _parallel}


def _feed_forward(cfg: NakuraxConfig, mlp: Optional[dict], where: str) -> Optional[FeedForwardSpec]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind", "dense") != "dense":
        raise ValueError(f"config.json: {where} must be a feed-forward of kind dense, or null")
    return FeedForwardSpec(kind="dense", hidden=cfg.width, intermediate=_int(where, mlp, "ff"), activation="relu2", bias=False)


def nakurax_model_spec(cfg: NakuraxConfig) -> ModelSpec:
    norm = NormSpec("rmsnorm", cfg.width, cfg.norm_eps, bias=False)
    layers = []
    for i, L in enumerate(cfg.layers):
        where = f"layers[{i}]"
        if not isinstance(L, dict) or L.get("type") not in _MIXERS:
            raise ValueError(f"config.json: {where}.type must be one of {', '.join(sorted(_MIXERS))}")
        mixer = _MIXERS[L["type"]](cfg, _object(where, L, "mixer"), where + ".mixer")
        ffn = _feed_forward(cfg, L.get("mlp"), where + ".mlp")
        layers.append(BlockSpec(arrangement="streams", norm=norm, mixer=mixer, ffn=ffn,
                                norm2=norm if ffn is not None else None, extra=(("streams", cfg.streams),)))
    schedule = default_schedule(len(layers))
    if cfg.loop is not None:
        loop = cfg.loop
        if not isinstance(loop, dict):
            raise ValueError("config.json: loop must be an object")
        schedule = looped_schedule(len(layers), _int("loop", loop, "start", 0), _int("loop", loop, "stop", 0),
                                   _int("loop", loop, "times"), marked=False)
    return ModelSpec(hidden=cfg.width, vocab=cfg.vocab, max_positions=UNBOUNDED_POSITIONS, layers=tuple(layers),
                     schedule=schedule, final_norm=norm, tie_embeddings=False, head_bias=False,
                     embedding_scale=cfg.embedding_scale, streams=cfg.streams)


class NakuraxTensorNames:
    """Names of the tensors in a Nakurax safetensors file: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
    ``l<i>.mlp.*``, ``l<i>.hc1.*``, ``l<i>.hc2.*``, ``final.norm``, ``head``; a linear layer's weight carries no suffix, a
    bias ``.b``, a convolution's taps ``.conv`` and their bias ``.conv.b``."""
    _top = {"embedding": "embed", "final_norm/weight": "final.norm", "head/weight": "head"}
    _slots = {"norm": "norm1", "norm2": "norm2", "mixer": "mix", "ffn": "mlp", "hc1": "hc1", "hc2": "hc2"}

    def __init__(self, cfg: NakuraxConfig):
        self.cfg = cfg

    def top(self, key: str) -> str:
        return self._top[key]

    def layer(self, i: int, slot: str, key: str) -> str:
        """Parts spell a parameter "left.q.weight", "right.ra.bias", "conv.weight", "dkv.norm.weight", "lam", "mix"; the
        file spells them "left.q", "right.ra.b", "conv", "dkv.norm", "lam", "mix"."""
        base = f"l{i}.{self._slots[slot]}"
        if slot in ("norm", "norm2"):
            return base
        words = key.split(".")
        if words[-1] == "weight":
            words = words[:-1]
        elif words[-1] == "bias":
            words[-1] = "b"
        return ".".join([base] + words)


register_architecture(
    Architecture(name="nakurax", config_class=NakuraxConfig, build_spec=nakurax_model_spec,
                 tensor_names=NakuraxTensorNames),
)
