"""The Dibedra design: a decoder whose layers read one squashed copy of the stream with two sublayers side by side:
windowed softmax attention whose values are its keys, and a dense feed-forward or a mixture of experts some of which
are the identity.

config.json lists the layers one by one: ``layers[i].type`` is ``attention``, ``layers[i].mixer`` the mixer's sizes and
constants, ``layers[i].mlp`` a feed-forward (``kind`` dense or moe) or null.  A layer with ``weights_of: j`` has no
tensors of its own: it runs layer j's mixer, feed-forward and norm on a cache entry of its own.

    h = norm1(x);  x <- x + (mixer(h) + ff(h)),   norm(x) = tanh(alpha x) * w + b with one number alpha.

  attention   H query heads on G key/value heads of size dim, no biases; the values are the keys as projected (vdim =
              dim); every head of q and k divided by its root mean square times a weight of size dim that the heads
              share, then its first rot.dims dims turned (dim 2i with dim 2i + 1), with rot.scaling at stretched
              frequencies; score = q . k * scale; a window of the last mask.size positions; the result times
              sigmoid(W_g h), element by element, before the output projection.
  dense       W_down gelu(W_up h), the tanh form, no biases.
  moe         scores s = softmax(W_router h) over experts and identity experts; the ``top`` largest s + correction
              among the best groups.keep of groups.count groups of neighbours (a group counts by its largest s +
              correction), weighted by s as it is; an expert is W_down (g sigmoid(1.702 g) (u + 1)), g = min(W_gate h,
              limit), u = clamp(W_up h, -limit, limit); the last router.identity outputs stand for h itself.

The head has weights of its own, no bias, and its product is multiplied by logit_scale; the final norm has the same
squashing form.  Every size and every constant that differs between models comes from config.json.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Optional

from .registry import Architecture, register_architecture
from .specs import BlockSpec, FeedForwardSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, ScheduleEntry

# the design sets no longest sequence; the cache's size bounds one
UNBOUNDED_POSITIONS = 1 << 20
# of the experts' gated form
GATE_SLOPE, UP_SHIFT = 1.702, 1.0


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
class DibedraConfig:
    """Typed view of a Dibedra config.json (key names are the file's own)."""
    vocab: int
    width: int
    layers: list
    norm_eps: float
    logit_scale: float
    architecture: str = "Dibedra"
    torch_dtype: str = "bfloat16"
    initializer_range: float = 0.05

    @classmethod
    def from_dict(cls, d: dict) -> "DibedraConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm", "logit_scale") if k not in d]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        if not isinstance(d["norm"], dict):
            raise ValueError("config.json: norm must be an object with eps")
        cfg = cls(vocab=_int("config", d, "vocab"), width=_int("config", d, "width"),
                  layers=copy.deepcopy(d["layers"]), norm_eps=_number("norm", d["norm"], "eps"),
                  logit_scale=_number("config", d, "logit_scale"),
                  architecture=str(d.get("architecture", "Dibedra")),
                  torch_dtype=str(d.get("torch_dtype", d.get("dtype", "bfloat16"))),
                  initializer_range=float(d.get("initializer_range", 0.05)))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
                "torch_dtype": self.torch_dtype, "initializer_range": self.initializer_range}

    def validate(self) -> None:
        if not isinstance(self.layers, list) or not self.layers:
            raise ValueError("config.json: layers must be a non-empty list")
        dibedra_model_spec(self)            # raises on anything a part or the schedule cannot take


def _rotation(where: str, m: dict, dim: int) -> PositionSpec:
    rot = m.get("rot")
    if rot is None:
        return PositionSpec("none")
    if not isinstance(rot, dict):
        raise ValueError(f"config.json: {where}.rot must be an object")
    dims = rot.get("dims", 0)
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > dim:
        raise ValueError(f"config.json: {where}.rot.dims must be even and at most dim, is {dims!r}")
    if dims == 0:
        return PositionSpec("none")
    base = _number(where + ".rot", rot, "base")
    extra = [("exact_angles", True)]
    if rot.get("scaling") is not None:
        w, s = where + ".rot.scaling", _object(where + ".rot", rot, "scaling")
        if base == 1.0:
            raise ValueError(f"config.json: {where}.rot.base must not be 1 where the frequencies are stretched")
        extra.append(("yarn", tuple(_number(w, s, k) for k in ("factor", "original", "fast", "slow"))))
    return PositionSpec("rope", dims, base, interleaved=True, extra=tuple(extra))


def _attention(cfg: DibedraConfig, m: dict, where: str) -> MixerSpec:
    heads, kv = _int(where, m, "heads"), _int(where, m, "kv_heads")
    if heads % kv:
        raise ValueError(f"config.json: {where}.heads {heads} is not a multiple of kv_heads {kv}")
    dim = _int(where, m, "dim")
    if _int(where, m, "vdim") != dim:
        raise ValueError(f"config.json: {where}.vdim {m['vdim']} differs from dim {dim}: the values are the keys")
    window = _int(where + ".mask", _object(where, m, "mask"), "size") if m.get("mask") is not None else 0
    return MixerSpec(kind="attention", hidden=cfg.width, num_heads=heads, num_kv_heads=kv, head_dim=dim, window=window,
                     q_scale=_number(where, m, "scale", positive=False), bias=False,
                     qk_norm=NormSpec("rmsnorm", dim, cfg.norm_eps, bias=False), position=_rotation(where, m, dim),
                     extra=(("values", "keys"), ("gate", True)))


_MIXERS = {"attention": _attention}


def _feed_forward(cfg: DibedraConfig, mlp: Optional[dict], where: str) -> Optional[FeedForwardSpec]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ValueError(f"config.json: {where} must be a feed-forward of kind dense or moe, or null")
    if mlp["kind"] == "dense":
        return FeedForwardSpec(kind="dense", hidden=cfg.width, intermediate=_int(where, mlp, "ff"),
                               activation="gelu_new", bias=False)
    r, ex = _object(where, mlp, "router"), _object(where, mlp, "expert")
    experts, top = _int(where + ".router", r, "experts"), _int(where + ".router", r, "top")
    identity = _int(where + ".router", r, "identity", least=0) if r.get("identity") is not None else 0
    groups = keep = 1
    if r.get("groups") is not None:
        g = _object(where + ".router", r, "groups")
        groups, keep = _int(where + ".router.groups", g, "count"), _int(where + ".router.groups", g, "keep")
    n = experts + identity
    if n % groups or keep > groups or keep * (n // groups) < top:
        raise ValueError(f"config.json: {where}.router: top {top} of {n} outputs in {groups} groups of which {keep} stay "
                         f"is not possible")
    return FeedForwardSpec(kind="moe", hidden=cfg.width, intermediate=_int(where + ".expert", ex, "ff"),
                           activation="clipped", bias=False,
                           extra=(("experts", experts), ("top", top), ("identity", identity), ("groups", groups),
                                  ("keep", keep), ("group_by", "largest"), ("weights", "softmax_all"),
                                  ("correction", True), ("limit", _number(where + ".expert", ex, "limit")),
                                  ("slope", GATE_SLOPE), ("shift", UP_SHIFT)))


def own_layers(cfg: DibedraConfig) -> list:
    """Indices (in config.json's list) of the layers that have tensors of their own, in order."""
    return [i for i, L in enumerate(cfg.layers) if not (isinstance(L, dict) and L.get("weights_of") is not None)]


def dibedra_model_spec(cfg: DibedraConfig) -> ModelSpec:
    norm = NormSpec("dynamic_tanh", cfg.width, cfg.norm_eps)
    layers, schedule = [], []
    block_of = {}                    # layer of the file -> index of its block
    n = len(cfg.layers)
    for i, L in enumerate(cfg.layers):
        where = f"layers[{i}]"
        if not isinstance(L, dict) or L.get("type") not in _MIXERS:
            raise ValueError(f"config.json: {where}.type must be one of {', '.join(sorted(_MIXERS))}")
        if L.get("weights_of") is not None:
            continue
        mixer = _MIXERS[L["type"]](cfg, _object(where, L, "mixer"), where + ".mixer")
        block_of[i] = len(layers)
        layers.append(BlockSpec(arrangement="parallel", norm=norm, mixer=mixer,
                                ffn=_feed_forward(cfg, L.get("mlp"), where + ".mlp")))
    for i, L in enumerate(cfg.layers):
        where = f"layers[{i}]"
        source, hops = i, 0
        while cfg.layers[source].get("weights_of") is not None:       # a layer may name one that names another
            nxt = cfg.layers[source]["weights_of"]
            hops += 1
            if isinstance(nxt, bool) or not isinstance(nxt, int) or not 0 <= nxt < n or nxt == source or hops > n:
                raise ValueError(f"config.json: {where}.weights_of must lead to a layer with tensors of its own, "
                                 f"is {L.get('weights_of')!r}")
            source = nxt
        if source != i:
            theirs = cfg.layers[source]
            if any(theirs.get(k) != L.get(k) for k in ("type", "mixer", "mlp")):
                raise ValueError(f"config.json: {where} runs on layer {source}'s weights but its entry differs")
        schedule.append(ScheduleEntry(layer=block_of[source], cache=i))
    return ModelSpec(hidden=cfg.width, vocab=cfg.vocab, max_positions=UNBOUNDED_POSITIONS, layers=tuple(layers),
                     schedule=tuple(schedule), final_norm=norm, tie_embeddings=False, head_bias=False,
                     logit_scale=cfg.logit_scale)


class DibedraTensorNames:
    """Names of the tensors in a Dibedra safetensors file: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
    ``final.norm``, ``head``, with i the layer's place in config.json's list (a layer that runs on another's weights has
    none); a weight carries no suffix, a norm's offset is ``.b`` and its slope ``.alpha``."""
    _top = {"embedding": "embed", "final_norm/weight": "final.norm", "final_norm/bias": "final.norm.b",
            "final_norm/alpha": "final.norm.alpha", "head/weight": "head"}
    _slots = {"norm": "norm1", "mixer": "mix", "ffn": "mlp"}
    _mixer = {"out": "o", "q_norm": "q.norm", "k_norm": "k.norm"}

    def __init__(self, cfg: DibedraConfig):
        self.cfg = cfg
        self.file_index = own_layers(cfg)

    def top(self, key: str) -> str:
        return self._top[key]

    def layer(self, i: int, slot: str, key: str) -> str:
        """Parts spell a parameter "weight", "bias", "alpha", "out.weight", "q_norm.weight", "e3.gate.weight",
        "correction"; the file spells them "", "b", "alpha", "o", "q.norm", "e3.gate", "correction"."""
        words = key.split(".")
        if slot == "mixer":
            words[0] = self._mixer.get(words[0], words[0])
        if words[-1] == "weight":
            words = words[:-1]
        elif words[-1] == "bias":
            words[-1] = "b"
        return ".".join([f"l{self.file_index[i]}.{self._slots[slot]}"] + words)


register_architecture(
    Architecture(name="dibedra", config_class=DibedraConfig, build_spec=dibedra_model_spec,
                 tensor_names=DibedraTensorNames),
)
