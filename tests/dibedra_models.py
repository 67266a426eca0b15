"""Small Dibedra configurations for the tests, with weights made by the tests themselves.

The tensors are drawn here by name (the design's naming rules, restated), written with the library's container
writer and read back by the library and by the plain implementation, so a wrong name or shape on either side shows.
The configurations differ in every respect: widths (one a multiple of nothing), head counts (one key/value head, as many
as query heads, twelve query heads on one), head sizes that are no multiples of 16, joined heads narrower and wider than
the model, rotations of a part of a head, of the whole head and of nothing, with stretched frequencies and without,
windows shorter than a page, longer than two pages, of one position and none, one expert a token to all of them, one
group and several, no identity experts or as many as experts, layers without a feed-forward, layers on another's
weights (a later layer's, one that names another), factors on the logits of one and other than one.
"""
import json
import os
import tempfile

import torch

_A0 = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.3, "mask": {"size": 20},
       "rot": {"dims": 8, "base": 10000.0, "scaling": {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 2.0}}}
_A1 = {"heads": 6, "kv_heads": 1, "dim": 32, "vdim": 32, "scale": 0.2, "mask": {"size": 70}, "rot": {"dims": 32, "base": 500.0}}
_A_MOE = {"kind": "moe", "expert": {"ff": 24, "limit": 0.9},
          "router": {"experts": 6, "top": 3, "identity": 2, "groups": {"count": 4, "keep": 2}}}
ALPHA = dict(
    architecture="Dibedra", vocab=300, width=64, norm={"eps": 1e-6}, logit_scale=1.7,
    layers=[
        {"type": "attention", "mixer": _A0, "mlp": {"kind": "dense", "ff": 48}},
        {"type": "attention", "mixer": _A1, "mlp": _A_MOE},
        {"type": "attention", "mixer": _A0, "mlp": {"kind": "dense", "ff": 48}, "weights_of": 0},
        {"type": "attention", "mixer": _A1, "mlp": _A_MOE, "weights_of": 1},
        {"type": "attention", "mixer": dict(_A0, mask={"size": 1}), "mlp": None},
    ])

_B0 = {"heads": 3, "kv_heads": 3, "dim": 48, "vdim": 48, "scale": 0.15, "mask": {"size": 130},
       "rot": {"dims": 24, "base": 3000.0, "scaling": {"factor": 1.5, "original": 32, "fast": 4.0, "slow": 1.0}}}
_B1 = {"heads": 12, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.25}
_B_MOE = {"kind": "moe", "expert": {"ff": 32, "limit": 2.0}, "router": {"experts": 4, "top": 1, "identity": 4}}
BETA = dict(
    architecture="Dibedra", vocab=257, width=96, norm={"eps": 1e-5}, logit_scale=1.0,
    layers=[
        {"type": "attention", "mixer": _B1, "mlp": _B_MOE, "weights_of": 2},
        {"type": "attention", "mixer": _B0, "mlp": {"kind": "moe", "expert": {"ff": 40, "limit": 0.5},
                                                    "router": {"experts": 5, "top": 5, "identity": 0}}},
        {"type": "attention", "mixer": _B1, "mlp": _B_MOE},
        {"type": "attention", "mixer": _B1, "mlp": _B_MOE, "weights_of": 0},
    ])

# sizes that are multiples of nothing convenient
GAMMA = dict(
    architecture="Dibedra", vocab=91, width=36, norm={"eps": 3e-6}, logit_scale=0.8,
    layers=[
        {"type": "attention",
         "mixer": {"heads": 3, "kv_heads": 3, "dim": 6, "vdim": 6, "scale": 0.5, "mask": {"size": 3}, "rot": {"dims": 2, "base": 7.0}},
         "mlp": {"kind": "moe", "expert": {"ff": 5, "limit": 0.4},
                 "router": {"experts": 2, "top": 2, "identity": 1, "groups": {"count": 3, "keep": 3}}}},
        {"type": "attention",
         "mixer": {"heads": 5, "kv_heads": 1, "dim": 10, "vdim": 10, "scale": 0.4, "mask": {"size": 40},
                   "rot": {"dims": 10, "base": 50.0, "scaling": {"factor": 8.0, "original": 100, "fast": 3.0, "slow": 0.5}}},
         "mlp": {"kind": "dense", "ff": 13}},
        {"type": "attention",
         "mixer": {"heads": 2, "kv_heads": 2, "dim": 5, "vdim": 5, "scale": 0.6, "rot": {"dims": 4, "base": 100.0}},
         "mlp": {"kind": "moe", "expert": {"ff": 7, "limit": 1.1},
                 "router": {"experts": 3, "top": 1, "identity": 3, "groups": {"count": 2, "keep": 1}}}},
    ])

# layer sizes nearer a real model's: heads of 64 and 128, eight and twelve query heads on a key head, many experts
WIDE = dict(
    architecture="Dibedra", vocab=500, width=256, norm={"eps": 1e-6}, logit_scale=0.6,
    layers=[
        {"type": "attention",
         "mixer": {"heads": 16, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.12, "mask": {"size": 150},
                   "rot": {"dims": 32, "base": 10000.0, "scaling": {"factor": 2.0, "original": 128, "fast": 8.0, "slow": 1.0}}},
         "mlp": {"kind": "moe", "expert": {"ff": 64, "limit": 1.0},
                 "router": {"experts": 24, "top": 4, "identity": 8, "groups": {"count": 8, "keep": 3}}}},
        {"type": "attention",
         "mixer": {"heads": 12, "kv_heads": 1, "dim": 128, "vdim": 128, "scale": 0.09, "mask": {"size": 64}, "rot": {"dims": 128, "base": 1e6}},
         "mlp": {"kind": "dense", "ff": 512}},
        {"type": "attention",
         "mixer": {"heads": 2, "kv_heads": 1, "dim": 160, "vdim": 160, "scale": 0.08, "mask": {"size": 65}, "rot": {"dims": 64, "base": 1e4}},
         "mlp": {"kind": "moe", "expert": {"ff": 128, "limit": 1.5}, "router": {"experts": 8, "top": 2, "identity": 0}}},
    ])


def only(cfg, index, mlp=True):
    """A model of one layer of ``cfg`` (a mechanism alone), with or without its feed-forward."""
    layer = json.loads(json.dumps(cfg["layers"][index]))
    layer.pop("weights_of", None)
    if not mlp:
        layer["mlp"] = None
    out = {k: v for k, v in cfg.items() if k != "layers"}
    out["layers"] = [layer]
    return out


def tensor_shapes(cfg):
    """name -> (shape, how it is drawn)."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": ((V, W), "embed"), "head": ((V, W), "matrix")}

    def squash(name):
        s.update({name: ((W,), "gamma"), name + ".b": ((W,), "small"), name + ".alpha": ((), "slope")})
    squash("final.norm")
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        squash(p + "norm1")
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        s.update({p + "mix.q": ((H * D, W), "matrix"), p + "mix.k": ((G * D, W), "matrix"), p + "mix.q.norm": ((D,), "sharp"),
                  p + "mix.k.norm": ((D,), "sharp"), p + "mix.g": ((H * D, W), "matrix"), p + "mix.o": ((W, H * D), "matrix")})
        mlp = L.get("mlp")
        if not mlp:
            continue
        if mlp["kind"] == "dense":
            s.update({p + "mlp.up": ((mlp["ff"], W), "matrix"), p + "mlp.down": ((W, mlp["ff"]), "matrix")})
            continue
        F, r = mlp["expert"]["ff"], mlp["router"]
        n = r["experts"] + r.get("identity", 0)
        s.update({p + "mlp.router": ((n, W), "router"), p + "mlp.correction": ((n,), "correction")})
        for e in range(r["experts"]):
            s.update({f"{p}mlp.e{e}.gate": ((F, W), "matrix"), f"{p}mlp.e{e}.up": ((F, W), "matrix"),
                      f"{p}mlp.e{e}.down": ((W, F), "matrix")})
    return s


def draw(cfg, seed, sharp=1.0):
    """Random bfloat16 tensors for ``cfg``.  ``sharp``: factor on the weights of the head norms (a score feels its square)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, (shape, kind) in sorted(tensor_shapes(cfg).items()):
        z = torch.randn(shape, generator=g)
        if kind == "matrix":
            t = z * (1.5 / shape[-1] ** 0.5)
        elif kind == "sharp":
            t = sharp * (1.0 + 0.2 * z)
        elif kind == "router":
            t = z * (3.0 / shape[-1] ** 0.5)          # logits a few apart: few close calls
        elif kind == "embed":
            t = z
        elif kind == "gamma":
            t = 1.0 + 0.2 * z
        elif kind == "small":
            t = 0.3 * z
        elif kind == "slope":
            t = 0.6 + 0.1 * z
        elif kind == "correction":
            t = 0.3 * z                                # as large as the scores: it decides many choices
        else:
            raise ValueError(kind)
        out[name] = t.to(torch.bfloat16)
    return out


def write_folder(cfg, tensors, folder=None):
    from gopherllm_b200.weights.safetensors_io import write_file
    folder = folder or tempfile.mkdtemp(prefix="gl_dibedra_")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_file(os.path.join(folder, "model.safetensors"), sorted(tensors.items()), metadata={"format": "pt"})
    return folder


def read_folder(folder):
    """(config dict, name -> 64-bit tensor) with a reader of the tests' own: 8 bytes of length, a JSON header, the data."""
    import struct
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    raw = open(os.path.join(folder, "model.safetensors"), "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    header = json.loads(raw[8:8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16}
    tensors = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + a:8 + n + b]), dtype=kinds[e["dtype"]]).reshape(e["shape"])
        tensors[name] = t.to(torch.float64)
    return cfg, tensors
