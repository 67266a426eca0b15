"""The Nakurax design on the CPU: its configuration, tensor names, schedule and cache needs in the library, and the
plain implementation's own sanity."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import nakurax_models as nm
import plain_nakurax as pn
from gopherllm_b200.api import build_model
from gopherllm_b200.cache.sequence_cache import PAGE, RELEASED, KVView, SequenceCache, StateView
from gopherllm_b200.config.registry import architecture_from_config
from gopherllm_b200.config.specs import ModelSpec
from gopherllm_b200.parts.base import KVRequest, StateRequest
from gopherllm_b200.parts.position import banded_frequencies
from gopherllm_b200.weights.loader import check_folder, tensor_table


def build(cfg):
    arch = architecture_from_config(cfg)
    typed = arch.config_class.from_dict(cfg)
    return arch, typed, build_model(arch, typed)


@pytest.mark.parametrize("cfg", [nm.ALPHA, nm.BETA, nm.GAMMA, nm.DELTA], ids=["ALPHA", "BETA", "GAMMA", "DELTA"])
def test_declared_tensors_are_the_files_tensors(cfg):
    arch, typed, model = build(cfg)
    assert arch.name == "nakurax"
    table = tensor_table(model.parameters(), arch.tensor_names(typed))
    want = nm.tensor_shapes(cfg)
    assert set(table) == set(want)
    for name, (shape, _) in want.items():
        assert tuple(table[name][1].shape) == tuple(shape), name


def test_every_constant_of_the_file_reaches_the_spec():
    _, typed, model = build(nm.ALPHA)
    spec = model.spec
    assert not spec.tie_embeddings and not spec.head_bias and spec.final_norm.eps == 1e-6
    assert (spec.streams, spec.embedding_scale) == (3, 1.5)
    assert all(b.arrangement == "streams" and b.option("streams") == 3 for b in spec.layers)
    latent, pair, bare, other = (b.mixer for b in spec.layers)
    assert (latent.kind, latent.num_heads, latent.head_dim, latent.value_dim, latent.window) == ("latent_attention", 4, 16, 32, 0)
    assert (latent.option("kv_rank"), latent.option("score_scale"), latent.option("norm_eps")) == (48, 0.3, 1e-6)
    assert not any(latent.option(k) for k in ("q_rank", "rot", "sink", "gate"))
    assert pair.kind == "scaled_pair" and (pair.option("left_scale"), pair.option("right_scale")) == (0.7, 1.3)
    left, right = pair.option("left"), pair.option("right")
    assert (left.kind, left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.window) == ("attention_mixed", 4, 2, 16, 32, 0)
    assert left.option("chunk") == 20 and left.option("score_scale") == 0.3 and not left.bias and not left.option("sink")
    p = left.position
    assert (p.kind, p.rotary_dim, p.theta, p.interleaved, p.option("bands")) == ("rope", 8, 100.0, True, (8.0, 1.0, 3.0, 64.0))
    assert right.kind == "gated_linear_unit" and [right.option(k) for k in ("width", "blocks", "conv", "decay")] == [48, 3, 3, 8.0]
    assert other.option("right_scale") == -0.5
    assert spec.layers[0].ffn.intermediate == 96 and spec.layers[0].ffn.activation == "relu2" and not spec.layers[0].ffn.bias
    assert spec.layers[2].ffn is None and spec.layers[2].norm2 is None
    assert typed.to_dict()["layers"] == nm.ALPHA["layers"] and typed.to_dict()["loop"] == nm.ALPHA["loop"]
    _, _, plain_rot = build(nm.BETA)
    assert plain_rot.spec.layers[0].mixer.option("left").position.option("bands") is None
    _, _, no_rot = build(nm.GAMMA)
    assert no_rot.spec.layers[2].mixer.option("left").position.kind == "none"


def test_looped_layers_keep_entries_of_their_own():
    _, _, model = build(nm.ALPHA)
    runs = model.spec.schedule
    assert [e.layer for e in runs] == [0, 1, 2, 1, 2, 1, 2, 3] == pn.run_order(nm.ALPHA)
    assert [e.cache for e in runs] == list(range(8)) and all(e.writes and e.enter is None for e in runs)
    for cfg in (nm.BETA, nm.GAMMA, nm.DELTA):
        assert [e.layer for e in build(cfg)[2].spec.schedule] == pn.run_order(cfg)
    reqs = model.cache_requests()
    # the latent is all that is kept of a position; the pair keeps pages by chunks, and S and the filter's inputs
    assert reqs[0] == KVRequest(1, 48, 0, value_dim=48, values_in_keys=True)
    assert reqs[1] == (KVRequest(2, 16, 0, value_dim=32, chunk=20), StateRequest((48 + 48 * 2,))) and reqs[3] == reqs[5] == reqs[1]
    cache = SequenceCache(reqs, max_tokens=256, max_positions=256, dtype=torch.float32, device="cpu", max_slots=2)
    kv, state = cache.view(3)
    assert isinstance(kv, KVView) and isinstance(state, StateView)
    assert cache.view(1)[0].k.data_ptr() != kv.k.data_ptr() and cache.view(1)[1].rows.data_ptr() != state.rows.data_ptr()


@pytest.mark.parametrize("chunk", [1, 20, 64, 70, 130])
def test_pages_before_a_chunk_are_given_back(chunk):
    cache = SequenceCache([KVRequest(1, 16, chunk=chunk), KVRequest(1, 16)], max_tokens=1024, max_positions=1024,
                          dtype=torch.float32, device="cpu", max_slots=2)
    s = cache.open()
    for n in list(range(1, 300)) + [301, 360, 512, 513, 700]:
        cache.reserve([(s, n)])
        cache.commit(s, n)
        first = n // chunk * chunk                 # what the next token, at position n, still sees
        pages = cache._pages[s][0]
        assert all((p == RELEASED) == ((i + 1) * PAGE <= first) for i, p in enumerate(pages)), (chunk, n)
        assert RELEASED not in cache._pages[s][1]
        cache.check()
    cache.close(s)
    cache.check()


def test_banded_frequencies_are_the_plain_ones():
    for rot in (nm._PAIR_A["left"]["rot"], {"dims": 64, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}},
                {"dims": 16, "base": 50.0, "scaling": {"factor": 4.0, "low": 2.0, "high": 2.0, "original": 100}}):
        s = rot["scaling"]
        got = banded_frequencies(rot["dims"], rot["base"], s["factor"], s["low"], s["high"], s["original"])
        want = pn.frequencies(rot).numpy()
        assert np.allclose(got, want, rtol=1e-13)
        base = pn.frequencies({"dims": rot["dims"], "base": rot["base"]}).numpy()
        ratio = base / want
        assert np.isclose(ratio.max(), s["factor"]) and np.isclose(ratio.min(), 1.0)         # both ends of the bands occur
    ratio = pn.frequencies({"dims": 64, "base": 500000.0}).numpy() / pn.frequencies(
        {"dims": 64, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}}).numpy()
    assert ((ratio > 1.01) & (ratio < 7.99)).any()                                           # and the blend between


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
    (("streams",), 0), (("streams",), 17), (("streams",), KeyError), (("width",), KeyError), (("norm", "eps"), 0.0),
    (("layers", 0, "type"), "attention"), (("layers", 0, "mixer", "kv_rank"), 0), (("layers", 0, "mixer", "heads"), True),
    (("layers", 0, "mixer", "scale"), KeyError), (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mlp", "ff"), 0),
    (("layers", 1, "mixer", "left", "kv_heads"), 3), (("layers", 1, "mixer", "left", "mask", "size"), 0),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7), (("layers", 1, "mixer", "left", "rot", "dims"), 18),
    (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), 0.0), (("layers", 1, "mixer", "left", "rot", "scaling", "low"), 5.0),
    (("layers", 1, "mixer", "right", "blocks"), 5), (("layers", 1, "mixer", "right", "conv"), 0),
    (("layers", 1, "mixer", "left_scale"), "x"), (("loop", "stop"), 5), (("loop", "times"), 0), (("loop", "start"), 4)])
def test_configurations_that_are_refused(path, value):
    with pytest.raises((ValueError, KeyError)):
        build(_with(nm.ALPHA, path, value))


def test_a_models_blocks_share_its_streams():
    _, _, model = build(nm.ALPHA)
    spec = model.spec
    import dataclasses
    with pytest.raises(ValueError):
        dataclasses.replace(spec, streams=2)
    with pytest.raises(ValueError):
        dataclasses.replace(spec, streams=0)
    assert isinstance(dataclasses.replace(spec, vocab=10), ModelSpec)


def test_plain_layers_do_not_look_ahead():
    for cfg in (nm.ALPHA, nm.GAMMA):
        t = {k: v.double() for k, v in nm.draw(cfg, 2).items()}
        toks = [int(x) for x in np.random.default_rng(0).integers(0, cfg["vocab"], size=12)]
        a, b = pn.forward(toks, t, cfg), pn.forward(toks[:7], t, cfg)
        assert torch.allclose(a[:7], b, atol=1e-10)


def test_plain_rotation_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0, 6.0]]], dtype=torch.float64).repeat(3, 1, 1)      # [T=3, 1 head, 6]
    y = pn.rotate(x, {"dims": 4, "base": 100.0})
    assert torch.equal(y[0], x[0]) and torch.equal(y[:, :, 4:], x[:, :, 4:])                         # position 0; the unrotated rest
    for p in (1, 2):
        for i, f in enumerate((1.0, 100.0 ** -0.5)):                                               # pairs (0, 1) and (2, 3)
            u, v = float(x[p, 0, 2 * i]), float(x[p, 0, 2 * i + 1])
            assert math.isclose(float(y[p, 0, 2 * i]), u * math.cos(p * f) - v * math.sin(p * f), abs_tol=1e-12)
            assert math.isclose(float(y[p, 0, 2 * i + 1]), v * math.cos(p * f) + u * math.sin(p * f), abs_tol=1e-12)


def test_plain_chunks_by_hand():
    """Keys that are all zero: every visible value counts the same, so a position's output is its chunk's mean so far."""
    T, W, size = 8, 4, 3
    w = {k: v.double() for k, v in {"q": torch.zeros(4, W), "k": torch.zeros(4, W), "v": torch.eye(4, W), "o": torch.eye(W, 4)}.items()}
    h = torch.randn(T, W, dtype=torch.float64)
    got = pn.chunked_attention(h, w, "", {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "mask": {"size": size}})
    for t in range(T):
        assert torch.allclose(got[t], h[t // size * size:t + 1].mean(0), atol=1e-12)


def test_plain_latent_by_hand():
    """Keys and values built from the latent, one head: the output is a softmax over c's products."""
    torch.manual_seed(1)
    T, W, R, D, V = 5, 6, 3, 4, 2
    w = {k: torch.randn(s, dtype=torch.float64) for k, s in (("q", (D, W)), ("dkv", (R, W)), ("dkv.norm", (R,)), ("uk", (D, R)),
                                                             ("uv", (V, R)), ("o", (W, V)))}
    h = torch.randn(T, W, dtype=torch.float64)
    c = torch.stack([x / math.sqrt(float((x * x).mean()) + 1e-5) * w["dkv.norm"] for x in h @ w["dkv"].T])
    got = pn.latent_attention(h, w, "", {"heads": 1, "dim": D, "vdim": V, "scale": 0.7}, 1e-5)
    for t in range(T):
        e = [math.exp(0.7 * float((w["q"] @ h[t]) @ (w["uk"] @ c[j]))) for j in range(t + 1)]
        o = sum(e[j] * (w["uv"] @ c[j]) for j in range(t + 1)) / sum(e)
        assert torch.allclose(got[t], w["o"] @ o, atol=1e-10)


def test_plain_recurrence_by_hand():
    """S_t = sum_j (prod of the decays behind j) sqrt(1 - a_j^2) i_j u_j, decays from the gates."""
    torch.manual_seed(2)
    T, C = 6, 4
    u, r, i, lam = torch.randn(T, C).double(), torch.rand(T, C).double(), torch.rand(T, C).double(), torch.randn(C).double()
    a = torch.exp(-8.0 * r * torch.nn.functional.softplus(lam))
    got = pn.gated_recurrence(u, r, i, lam)
    for t in range(T):
        want = sum(a[j + 1:t + 1].prod(0) * torch.sqrt(1 - a[j] ** 2) * i[j] * u[j] for j in range(t + 1))
        assert torch.allclose(got[t], want, atol=1e-10)
    gates = pn.block_gate(torch.tensor([[1.0, 2.0, 3.0, 4.0]]).double(), torch.tensor([[[1.0, 0.0], [1.0, 1.0]], [[0.0, 2.0], [-1.0, 0.0]]]).double(),
                          torch.tensor([[0.5, 0.0], [0.0, 1.0]]).double())
    assert torch.allclose(gates[0], torch.sigmoid(torch.tensor([1.5, 3.0, 8.0, -2.0]).double()))      # [out, in], a part at a time


def test_plain_streams_by_hand():
    X = torch.tensor([[[1.0]], [[10.0]]], dtype=torch.float64)                        # two streams of one number
    w = {"in": torch.tensor([0.5, 0.25]), "out": torch.tensor([2.0, 3.0]), "mix": torch.tensor([[1.0, 4.0], [0.1, 5.0]])}
    got = pn.hyper_connected(X, {k: v.double() for k, v in w.items()}, "", lambda u: u + 1.0)
    y = 0.5 * 1 + 0.25 * 10 + 1
    assert torch.allclose(got.reshape(-1), torch.tensor([1 * 1.0 + 0.1 * 10 + 2 * y, 4 * 1 + 5 * 10 + 3 * y]).double(), atol=1e-5)


def test_command_line_inspects_and_writes_a_random_folder(tmp_path, capsys):
    from gopherllm_b200.cli import main
    cfg_file = tmp_path / "c.json"
    cfg_file.write_text(json.dumps(nm.GAMMA))
    folder = str(tmp_path / "m")
    assert main([folder, "--random-config", str(cfg_file), "--seed", "3"]) == 0
    arch, typed, model = build(nm.GAMMA)
    check_folder(folder, tensor_table(model.parameters(), arch.tensor_names(typed)))
    capsys.readouterr()
    assert main([folder, "--inspect"]) == 0
    out = capsys.readouterr().out
    assert "architecture: Nakurax" in out and "supported: true" in out
    cfg, t = nm.read_folder(folder)
    assert torch.isfinite(pn.forward([1, 2, 3, 4, 5], t, cfg)).all()
