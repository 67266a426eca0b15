"""Small Nakurax configurations for the tests, with weights made by the tests themselves.

The tensors are drawn here by name (the design's naming rules, restated), written with the library's container writer
and read back by the library and by the plain implementation, so a wrong name or shape on either side shows.  The
configurations differ in every respect: widths (one a multiple of nothing), one stream to five, head counts (one
key/value head, as many as query heads, six query heads on one; twelve and twenty-four on a latent), key and value sizes that
are no multiples of 16, value sizes larger and smaller than key sizes, latents narrower and wider than the model, rotations
of a part of a head, of the whole head and of nothing, with bands and without, chunks of one position, of less than a page, of a
page, and of more, one block and several, filters of one to four taps, recurrences narrower and wider than the model, layers
without a feed-forward, loops over a part, over everything and none.
"""
import json
import os
import tempfile

import torch

_BANDS = {"factor": 8.0, "low": 1.0, "high": 3.0, "original": 64}
_PAIR_A = {"left": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 32, "scale": 0.3, "mask": {"size": 20},
                    "rot": {"dims": 8, "base": 100.0, "scaling": _BANDS}},
           "right": {"width": 48, "blocks": 3, "conv": 3}, "left_scale": 0.7, "right_scale": 1.3}
ALPHA = dict(
    architecture="Nakurax", vocab=300, width=64, norm={"eps": 1e-6}, streams=3, embedding={"scale": 1.5},
    loop={"start": 1, "stop": 3, "times": 3},
    layers=[
        {"type": "latent_attention", "mixer": {"heads": 4, "dim": 16, "vdim": 32, "kv_rank": 48, "scale": 0.3},
         "mlp": {"kind": "dense", "ff": 96}},
        {"type": "parallel", "mixer": _PAIR_A, "mlp": {"kind": "dense", "ff": 40}},
        {"type": "latent_attention", "mixer": {"heads": 12, "dim": 8, "vdim": 16, "kv_rank": 32, "scale": 0.4}, "mlp": None},
        {"type": "parallel", "mixer": dict(_PAIR_A, right={"width": 80, "blocks": 1, "conv": 4}, left_scale=1.0, right_scale=-0.5),
         "mlp": None},
    ])

BETA = dict(
    architecture="Nakurax", vocab=257, width=96, norm={"eps": 1e-5}, streams=2, embedding={"scale": 1.0},
    layers=[
        {"type": "parallel",
         "mixer": {"left": {"heads": 3, "kv_heads": 3, "dim": 32, "vdim": 16, "scale": 0.2, "mask": {"size": 70},
                            "rot": {"dims": 32, "base": 3000.0}},
                   "right": {"width": 128, "blocks": 2, "conv": 1}, "left_scale": 1.0, "right_scale": 0.5},
         "mlp": {"kind": "dense", "ff": 64}},
        {"type": "latent_attention", "mixer": {"heads": 24, "dim": 16, "vdim": 16, "kv_rank": 96, "scale": 0.25},
         "mlp": {"kind": "dense", "ff": 160}},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 32, "vdim": 48, "kv_rank": 64, "scale": 0.2}, "mlp": None},
    ])

# sizes that are multiples of nothing convenient
GAMMA = dict(
    architecture="Nakurax", vocab=91, width=36, norm={"eps": 3e-6}, streams=5, embedding={"scale": 0.7},
    loop={"start": 0, "stop": 3, "times": 2},
    layers=[
        {"type": "latent_attention", "mixer": {"heads": 3, "dim": 6, "vdim": 10, "kv_rank": 14, "scale": 0.5},
         "mlp": {"kind": "dense", "ff": 13}},
        {"type": "parallel",
         "mixer": {"left": {"heads": 6, "kv_heads": 1, "dim": 6, "vdim": 10, "scale": 0.4, "mask": {"size": 3},
                            "rot": {"dims": 2, "base": 7.0, "scaling": {"factor": 2.0, "low": 1.0, "high": 2.0, "original": 10}}},
                   "right": {"width": 15, "blocks": 5, "conv": 2}, "left_scale": -0.5, "right_scale": 2.0},
         "mlp": {"kind": "dense", "ff": 21}},
        {"type": "parallel",
         "mixer": {"left": {"heads": 2, "kv_heads": 2, "dim": 5, "vdim": 3, "scale": 0.6, "mask": {"size": 1}},
                   "right": {"width": 28, "blocks": 7, "conv": 4}, "left_scale": 1.0, "right_scale": 1.0},
         "mlp": None},
    ])

# one stream, one head, a chunk of a page
DELTA = dict(
    architecture="Nakurax", vocab=120, width=48, norm={"eps": 1e-6}, streams=1, embedding={"scale": 2.0},
    loop={"start": 1, "stop": 2, "times": 1},
    layers=[
        {"type": "parallel",
         "mixer": {"left": {"heads": 1, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.3, "mask": {"size": 64},
                            "rot": {"dims": 16, "base": 50.0, "scaling": {"factor": 4.0, "low": 2.0, "high": 2.0, "original": 100}}},
                   "right": {"width": 24, "blocks": 1, "conv": 2}, "left_scale": 1.0, "right_scale": 1.0},
         "mlp": {"kind": "dense", "ff": 32}},
        {"type": "latent_attention", "mixer": {"heads": 1, "dim": 16, "vdim": 16, "kv_rank": 16, "scale": 0.3},
         "mlp": {"kind": "dense", "ff": 32}},
    ])


def only(cfg, index, mlp=True):
    """A model of one layer of ``cfg`` (a mechanism alone), with or without a feed-forward."""
    layer = json.loads(json.dumps(cfg["layers"][index]))
    if not mlp:
        layer["mlp"] = None
    elif layer["mlp"] is None:
        layer["mlp"] = {"kind": "dense", "ff": 24}
    out = {k: v for k, v in cfg.items() if k not in ("layers", "loop")}
    out["layers"] = [layer]
    return out


def tensor_shapes(cfg):
    """name -> (shape, how it is drawn)."""
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    s = {"embed": ((V, W), "embed"), "final.norm": ((W,), "gamma"), "head": ((V, W), "matrix")}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = ((W,), "gamma")
        s.update({p + "hc1.in": ((S,), "share"), p + "hc1.out": ((S,), "gamma"), p + "hc1.mix": ((S, S), "mix")})
        if L["type"] == "latent_attention":
            H, D, Vd, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            s.update({p + "mix.q": ((H * D, W), "query"), p + "mix.dkv": ((R, W), "matrix"), p + "mix.dkv.norm": ((R,), "gamma"),
                      p + "mix.uk": ((H * D, R), "query"), p + "mix.uv": ((H * Vd, R), "matrix"),
                      p + "mix.o": ((W, H * Vd), "matrix")})
        else:
            a, r = m["left"], m["right"]
            H, G, D, Vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            s.update({p + "mix.left.q": ((H * D, W), "query"), p + "mix.left.k": ((G * D, W), "query"),
                      p + "mix.left.v": ((G * Vd, W), "matrix"), p + "mix.left.o": ((W, H * Vd), "matrix")})
            C, B = r["width"], r["blocks"]
            n = C // B
            q = p + "mix.right."
            s.update({q + "y": ((C, W), "matrix"), q + "y.b": ((C,), "small"), q + "x": ((C, W), "matrix"), q + "x.b": ((C,), "small"),
                      q + "conv": ((C, r["conv"]), "taps"), q + "conv.b": ((C,), "small"),
                      q + "ra": ((B, n, n), "matrix"), q + "ra.b": ((B, n), "wide"), q + "ri": ((B, n, n), "matrix"),
                      q + "ri.b": ((B, n), "wide"), q + "lam": ((C,), "decay"), q + "o": ((W, C), "matrix")})
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            s[p + "norm2"] = ((W,), "gamma")
            s.update({p + "hc2.in": ((S,), "share"), p + "hc2.out": ((S,), "gamma"), p + "hc2.mix": ((S, S), "mix")})
            s.update({p + "mlp.up": ((F, W), "matrix"), p + "mlp.down": ((W, F), "matrix")})
    return s


def draw(cfg, seed, long_memory=False, sharp=1.0):
    """Random tensors (bfloat16) for ``cfg``.  ``long_memory``: decays near one, so that the recurrence still holds tokens
    from hundreds of positions back.  ``sharp``: factor on the attentions' query and key weights."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, (shape, kind) in sorted(tensor_shapes(cfg).items()):
        z = torch.randn(shape, generator=g)
        if kind == "matrix":
            t = z * (1.0 / shape[-1] ** 0.5)
        elif kind == "query":
            t = z * (sharp / shape[-1] ** 0.5)
        elif kind in ("embed", "wide"):
            t = z
        elif kind == "gamma":
            t = 1.0 + 0.2 * z
        elif kind == "small":
            t = 0.1 * z
        elif kind == "taps":
            t = 0.6 * z
        elif kind == "share":
            t = (1.0 + 0.5 * z) / shape[0]
        elif kind == "mix":
            t = 0.7 * torch.eye(shape[0]) + 0.15 * z
        elif kind == "decay":
            t = z - (7.0 if long_memory else 3.0)
        else:
            raise ValueError(kind)
        out[name] = t.to(torch.bfloat16)
    return out


def write_folder(cfg, tensors, folder=None):
    from gopherllm_b200.weights.safetensors_io import write_file
    folder = folder or tempfile.mkdtemp(prefix="gl_nakurax_")
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
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16}
    tensors = {}
    for name, e in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + a:8 + n + b]), dtype=kinds[e["dtype"]]).reshape(e["shape"])
        tensors[name] = t.to(torch.float64)
    return cfg, tensors
