"""The Dibedra design on the CPU: its configuration, tensor names, schedule and cache needs in the library,
and the plain implementation's own sanity."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import dibedra_models as dm
import plain_dibedra as pd
from gopherllm_b200.api import build_model
from gopherllm_b200.cache.sequence_cache import SequenceCache
from gopherllm_b200.config.registry import architecture_from_config
from gopherllm_b200.parts.base import KVRequest
from gopherllm_b200.parts.position import stretched_frequencies
from gopherllm_b200.weights.loader import tensor_table


def build(cfg):
    arch = architecture_from_config(cfg)
    typed = arch.config_class.from_dict(cfg)
    return arch, typed, build_model(arch, typed)


@pytest.mark.parametrize("cfg", [dm.ALPHA, dm.BETA, dm.GAMMA, dm.WIDE], ids=["ALPHA", "BETA", "GAMMA", "WIDE"])
def test_declared_tensors_are_the_files_tensors(cfg):
    arch, typed, model = build(cfg)
    assert arch.name == "dibedra"
    table = tensor_table(model.parameters(), arch.tensor_names(typed))
    want = dm.tensor_shapes(cfg)
    assert set(table) == set(want)
    for name, (shape, _) in want.items():
        assert tuple(table[name][1].shape) == tuple(shape), name
    assert table["final.norm.alpha"][1].shape == () and table["final.norm.alpha"][1].kind == "vector"


def test_every_constant_of_the_file_reaches_the_spec():
    _, typed, model = build(dm.ALPHA)
    spec = model.spec
    assert not spec.tie_embeddings and not spec.head_bias and spec.logit_scale == 1.7 and spec.final_norm.kind == "dynamic_tanh"
    assert len(spec.layers) == 3 and all(b.arrangement == "parallel" and b.norm.kind == "dynamic_tanh" and b.norm2 is None for b in spec.layers)
    a, b, c = (x.mixer for x in spec.layers)
    assert (a.kind, a.num_heads, a.num_kv_heads, a.head_dim, a.window, a.q_scale, a.bias) == ("attention", 4, 2, 16, 20, 0.3, False)
    assert (a.qk_norm.kind, a.qk_norm.dim, a.qk_norm.eps, a.qk_norm.bias) == ("rmsnorm", 16, 1e-6, False)
    assert (a.position.kind, a.position.rotary_dim, a.position.theta, a.position.interleaved) == ("rope", 8, 10000.0, True)
    assert a.position.option("yarn") == (4.0, 64.0, 16.0, 2.0) and b.position.option("yarn") is None and b.position.option("exact_angles")
    assert a.option("values") == "keys" and a.option("gate") and (b.window, c.window) == (70, 1)
    dense, moe, none = (x.ffn for x in spec.layers)
    assert (dense.kind, dense.intermediate, dense.activation, dense.bias) == ("dense", 48, "gelu_new", False) and none is None
    assert (moe.kind, moe.intermediate, moe.activation) == ("moe", 24, "clipped")
    assert [moe.option(k) for k in ("experts", "top", "identity", "groups", "keep", "group_by", "weights", "correction", "limit", "slope",
                                    "shift")] == [6, 3, 2, 4, 2, "largest", "softmax_all", True, 0.9, 1.702, 1.0]
    assert typed.to_dict()["layers"] == dm.ALPHA["layers"] and typed.to_dict()["logit_scale"] == 1.7
    none_of_it = build(dm.BETA)[2].spec.layers
    assert none_of_it[1].mixer.position.kind == "none" and none_of_it[1].mixer.window == 0
    assert (none_of_it[0].ffn.option("identity"), none_of_it[0].ffn.option("groups"), none_of_it[0].ffn.option("keep")) == (0, 1, 1)


def test_layers_that_run_on_another_layers_weights():
    arch, typed, model = build(dm.BETA)
    # layer 0 names layer 2, layer 3 names layer 0; every run has a cache entry of its own
    assert [(e.layer, e.cache, e.writes) for e in model.spec.schedule] == [(1, 0, True), (0, 1, True), (1, 2, True), (1, 3, True)]
    names = arch.tensor_names(typed)
    assert names.layer(0, "mixer", "q_norm.weight") == "l1.mix.q.norm" and names.layer(1, "mixer", "out.weight") == "l2.mix.o"
    assert names.layer(1, "norm", "alpha") == "l2.norm1.alpha" and names.layer(0, "norm", "bias") == "l1.norm1.b"
    assert names.layer(1, "ffn", "correction") == "l2.mlp.correction" and names.layer(1, "ffn", "e3.down.weight") == "l2.mlp.e3.down"
    reqs = model.cache_requests()
    assert reqs == [KVRequest(1, 16, 0), KVRequest(3, 48, 130), KVRequest(1, 16, 0), KVRequest(1, 16, 0)]
    cache = SequenceCache(reqs, max_tokens=256, max_positions=256, dtype=torch.float32, device="cpu", max_slots=2)
    assert len(cache.groups) == 2 and cache.bytes_per_position() == 4 * 2 * (3 * 16 + 3 * 48)


def _with(cfg, path, value):
    out = copy.deepcopy(cfg)
    at = out
    for k in path[:-1]:
        at = at[k]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return out


@pytest.mark.parametrize("path,value", [
    (("layers", 2, "weights_of"), 2), (("layers", 2, "weights_of"), 1), (("layers", 2, "weights_of"), 9), (("layers", 0, "weights_of"), 2),
    (("layers", 0, "mixer", "vdim"), 8), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "rot", "dims"), 7),
    (("layers", 0, "mixer", "rot", "dims"), 18), (("layers", 0, "mixer", "rot", "scaling"), 2.0),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0), (("layers", 0, "mixer", "rot", "base"), 1.0),
    (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "scale"), KeyError), (("layers", 0, "mixer", "dim"), KeyError),
    (("layers", 1, "mlp", "router", "top"), 5), (("layers", 1, "mlp", "router", "groups", "count"), 3),
    (("layers", 1, "mlp", "router", "groups", "keep"), 5), (("layers", 1, "mlp", "expert", "limit"), KeyError),
    (("layers", 0, "mlp", "kind"), "gated"), (("layers", 0, "type"), "mamba"), (("logit_scale",), KeyError), (("norm",), 1e-5),
    (("layers",), []), (("width",), 0),
])
def test_refused_configurations(path, value):
    cfg = _with(dm.ALPHA, path, value)
    for L in cfg["layers"]:               # (a changed entry is refused for itself, not for differing from its copy)
        if path[-1] != "weights_of":
            L.pop("weights_of", None)
    with pytest.raises(ValueError):
        build(cfg)


def test_command_line_inspects_and_writes_a_random_folder(tmp_path, capsys):
    from gopherllm_b200 import cli
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(dm.GAMMA))
    folder = tmp_path / "model"
    assert cli.main([str(folder), "--random-config", str(cfg_path), "--seed", "3"]) == 0
    cfg, tensors = dm.read_folder(str(folder))
    assert set(tensors) == set(dm.tensor_shapes(dm.GAMMA)) and tensors["l0.norm1.alpha"].shape == ()
    logits = pd.forward(cfg, tensors, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 91) and torch.isfinite(logits).all()
    assert cli.main([str(folder), "--inspect"]) == 0
    assert "dibedra" in capsys.readouterr().out.lower()


# -- the plain implementation by hand ------------------------------------------------------------------------------
def test_plain_model_is_causal_and_its_windows_end():
    cfg = dm.ALPHA
    t = {k: v.double() for k, v in dm.draw(cfg, 3).items()}
    toks = [int(x) for x in np.random.default_rng(0).integers(0, cfg["vocab"], size=40)]
    a = pd.forward(cfg, t, toks)
    other = list(toks)
    other[30] = (other[30] + 1) % cfg["vocab"]
    b = pd.forward(cfg, t, other)
    assert float((a[:30] - b[:30]).abs().max()) == 0.0 and float((a[30:] - b[30:]).abs().max()) > 1e-6
    one = dm.only(dm.GAMMA, 0)            # a window of 3 alone forgets a token three positions on
    t1 = {k: v.double() for k, v in dm.draw(one, 4).items()}
    toks = [int(x) for x in np.random.default_rng(1).integers(0, one["vocab"], size=12)]
    a = pd.forward(one, t1, toks)
    other = list(toks)
    other[4] = (other[4] + 1) % one["vocab"]
    b = pd.forward(one, t1, other)
    moved = (a - b).abs().max(-1).values
    assert (moved[4:7] > 1e-9).all() and float(moved[7:].max()) == 0.0 and float(moved[:4].max()) == 0.0


def test_plain_mechanisms_by_hand():
    d = lambda *v: torch.tensor(v, dtype=torch.float64)
    w = {"n": d(2.0, 3.0), "n.b": d(0.5, -0.5), "n.alpha": torch.tensor(0.5, dtype=torch.float64)}
    assert torch.allclose(pd.dynamic_tanh(d(1.0, -4.0), w, "n"), d(2 * math.tanh(0.5) + 0.5, 3 * math.tanh(-2.0) - 0.5))
    assert torch.allclose(pd.gelu_tanh(d(1.0)), d(0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715))))
    # an expert of one inner number: the gate is cut from above only, the up projection on both sides
    e = lambda g, u: pd.expert(d(1.0)[None], {"e.gate": d(g)[None], "e.up": d(u)[None], "e.down": d(1.0)[None]}, "e.", 0.7)[0, 0]
    sg = lambda z: 1 / (1 + math.exp(-z))
    for g, u, gc, uc in ((0.5, 0.2, 0.5, 0.2), (2.0, 3.0, 0.7, 0.7), (-5.0, -3.0, -5.0, -0.7)):
        assert abs(float(e(g, u)) - gc * sg(1.702 * gc) * (uc + 1)) < 1e-12
    # the router: experts 0, 1 | 2, identity 3; the correction decides the group and the choice, not the weights
    r = {"experts": 3, "top": 1, "identity": 1, "groups": {"count": 2, "keep": 1}}
    w = {"r.router": torch.eye(4, dtype=torch.float64), "r.correction": d(0.0, -2.0, -0.9, 0.1)}
    h = d(2.0, 0.0, 1.0, 0.0)[None]
    s = torch.softmax(h[0], -1)
    ids, weights = pd.route(h, w, "r.", r)
    assert ids.tolist() == [[0]] and torch.allclose(weights[0], s[:1])
    w["r.correction"] = d(-3.0, -2.0, -2.5, -2.1)          # all negative: the dropped group must not win by counting as 0
    ids, weights = pd.route(h, w, "r.", r)
    assert ids.tolist() == [[1]] and torch.allclose(weights[0], s[1:2])
    ids, weights = pd.route(h, w, "r.", dict(r, top=2))
    assert ids.tolist() == [[1, 0]]
    # rotation: neighbours turned together, position 0 turns nothing
    x = torch.arange(12, dtype=torch.float64).view(2, 1, 6) + 1.0
    n = pd.rotate_pairs(x, {"dims": 4, "base": 100.0})
    u, a0, a1 = x[1, 0], 1.0, 100.0 ** -0.5
    assert torch.equal(n[0], x[0]) and torch.equal(n[..., 4:], x[..., 4:])
    assert torch.allclose(n[1, 0, :4], torch.stack([u[0] * math.cos(a0) - u[1] * math.sin(a0), u[1] * math.cos(a0) + u[0] * math.sin(a0),
                                                    u[2] * math.cos(a1) - u[3] * math.sin(a1), u[3] * math.cos(a1) + u[2] * math.sin(a1)]))


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (96, 700.0, 3.0, 2048, 24.0, 1.5), (8, 10000.0, 4.0, 64, 16.0, 2.0), (10, 50.0, 8.0, 100, 3.0, 0.5), (16, 7.0, 0.5, 4096, 1.0, 1.0),
    (24, 1e6, 1.0, 32, 4.0, 1.0), (2, 5.0, 3.0, 10, 1e3, 1e2)])
def test_stretched_frequencies(dims, base, factor, original, fast, slow):
    """The library's table against the plain implementation's, both ends of the ramp and ramps of no length included."""
    rot = {"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    freq, gain = pd.pair_frequencies(rot)
    got, g2 = stretched_frequencies(dims, base, factor, original, fast, slow)
    assert np.allclose(got, freq, rtol=1e-12, atol=0) and abs(gain - g2) < 1e-15
    assert abs(gain - (0.1 * math.log(factor) + 1.0)) < 1e-15
