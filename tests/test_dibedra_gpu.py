"""The Dibedra design through the library's loader, cache, step function, scheduler and kernels, against
the plain implementation (tests/plain_dibedra.py) on small models whose weights the tests make themselves."""
import copy
import json

import numpy as np
import pytest
import torch

import dibedra_models as dm
import plain_dibedra as pd

pytestmark = pytest.mark.gpu

# the largest |difference| of a position's logits is bounded by TOL * max(1, max|reference|), the mean over
# positions by MEAN_TOL
TOL = {"float32": 3e-4, "bfloat16": 1e-1}
MEAN_TOL = {"float32": 1e-4, "bfloat16": 3e-2}
_REF = {}


def plain_logits(folder, tokens):
    key = (folder, tuple(tokens))
    if key not in _REF:
        cfg, t = dm.read_folder(folder)
        _REF[key] = pd.forward(cfg, t, list(tokens)).numpy()
    return _REF[key]


def load(folder, dtype, max_tokens=4096, **kw):
    import gopherllm_b200 as gl
    return gl.load(folder, dtype=dtype, max_tokens=max_tokens, **kw)


def feed(model, slot, tokens, cuts):
    """Feed ``tokens`` in pieces of the given sizes (the rest one by one); logits of every position."""
    out, at = [], 0
    cuts = list(cuts)
    while at < len(tokens):
        n = min(cuts.pop(0) if cuts else 1, len(tokens) - at)
        out.append(model.step([(slot, tokens[at:at + n])], [list(range(n))]).cpu().numpy())
        at += n
    return np.concatenate(out, 0)


def check(got, ref, dtype, what="", outliers=0):
    """``outliers``: so many positions are left out of the bound: positions where a sixteen-bit router logit falls on the
    other side of a close call and the token meets another expert than in the 64-bit run (with one expert a token that
    changes the whole feed-forward's output).  The 32-bit run of the same test allows none."""
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert np.isfinite(got).all(), what
    err = np.abs(got - ref).max(-1)
    bound = TOL[dtype] * max(1.0, float(np.abs(ref).max()))
    if outliers:
        err = np.sort(err)[::-1][outliers:] if len(err) > outliers else err * 0
    worst = int(err.argmax())
    assert err.max() <= bound, f"{what} {dtype}: position {worst} differs by {err.max():.3e} (bound {bound:.3e})"
    mean_bound = MEAN_TOL[dtype] * max(1.0, float(np.abs(ref).max()))
    assert err.mean() <= mean_bound, f"{what} {dtype}: positions differ by {err.mean():.3e} on average (bound {mean_bound:.3e})"


def loose(dtype, n):
    """Positions of n that a bfloat16 router may send to another expert than the 64-bit one."""
    return max(1, n // 40) if dtype == "bfloat16" else 0


def tokens_for(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)]


FOLDERS = {}


def folder_for(name, cfg, seed, **kw):
    key = (name, seed, tuple(sorted(kw.items())))
    if key not in FOLDERS:
        FOLDERS[key] = dm.write_folder(cfg, dm.draw(cfg, seed, **kw))
    return FOLDERS[key]


def _double(tensors):
    return {k: v.double() for k, v in tensors.items()}


# every query head its own key head, eight and more on one, head sizes the tensor-core kernels take and others
MANY = dict(
    architecture="Dibedra", vocab=200, width=64, norm={"eps": 1e-6}, logit_scale=0.9,
    layers=[
        {"type": "attention", "mixer": {"heads": 16, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.3, "mask": {"size": 100},
                                        "rot": {"dims": 16, "base": 1000.0}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 11, "kv_heads": 1, "dim": 32, "vdim": 32, "scale": 0.2,
                                        "rot": {"dims": 10, "base": 1000.0}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 8, "kv_heads": 8, "dim": 80, "vdim": 80, "scale": 0.1, "mask": {"size": 64},
                                        "rot": {"dims": 6, "base": 1000.0}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 10, "kv_heads": 1, "dim": 24, "vdim": 24, "scale": 0.2, "mask": {"size": 65},
                                        "rot": {"dims": 24, "base": 1000.0}}, "mlp": None},
    ])

ALONE = [("dense", dm.only(dm.ALPHA, 0)), ("six_heads_on_one_mixture", dm.only(dm.ALPHA, 1)),
         ("window_of_one", dm.only(dm.ALPHA, 4)), ("no_rotation_no_window_top1", dm.only(dm.BETA, 2)),
         ("all_experts_no_identity", dm.only(dm.BETA, 1)), ("odd_window_three_all_outputs", dm.only(dm.GAMMA, 0)),
         ("odd_dense", dm.only(dm.GAMMA, 1)), ("odd_head_of_five_top1", dm.only(dm.GAMMA, 2)),
         ("sixteen_on_one", dm.only(MANY, 0)), ("eleven_on_one", dm.only(MANY, 1)), ("heads_of_eighty", dm.only(MANY, 2)),
         ("ten_on_one_heads_of_24", dm.only(MANY, 3)), ("many", MANY),
         ("groups_of_four_mixture", dm.only(dm.WIDE, 0)), ("heads_of_160", dm.only(dm.WIDE, 2))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg", ALONE, ids=[a[0] for a in ALONE])
def test_each_mechanism_alone(name, cfg, dtype):
    """One layer of one kind: a whole prompt across a page's edge, then single tokens."""
    folder = folder_for(name, cfg, 11)
    toks = tokens_for(cfg, 90, 1)
    m = load(folder, dtype)
    s = m.open_sequence()
    got = feed(m, s, toks, [70])
    m.engine.check_device()
    check(got, plain_logits(folder, toks), dtype, name, outliers=loose(dtype, 90))
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg_name", ["ALPHA", "BETA", "GAMMA"])
def test_whole_pieces_and_single_tokens(cfg_name, dtype):
    """The same tokens whole, in pieces of many sizes down to two, and mostly one by one."""
    cfg = getattr(dm, cfg_name)
    folder = folder_for(cfg_name, cfg, 5)
    toks = tokens_for(cfg, 150, 2)
    ref = plain_logits(folder, toks)
    m = load(folder, dtype)
    whole = None
    for cuts in ([150], [2, 2, 3, 57, 1, 64, 2, 19], [40]):
        s = m.open_sequence()
        got = feed(m, s, toks, cuts)
        m.close_sequence(s)
        check(got, ref, dtype, f"{cfg_name} cuts {cuts}", outliers=loose(dtype, 150))
        whole = got if whole is None else whole
        if dtype == "float32":
            assert np.abs(got - whole).max() <= 5e-5 * max(1.0, np.abs(whole).max()), f"{cfg_name}: cuts {cuts} against the whole prompt"
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_nearer_a_real_layer(dtype):
    folder = folder_for("WIDE", dm.WIDE, 21)
    toks = tokens_for(dm.WIDE, 330, 4)
    ref = plain_logits(folder, toks)
    m = load(folder, dtype)
    for cuts in ([330], [130, 66, 100]):
        s = m.open_sequence()
        check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}", outliers=loose(dtype, 330))
        m.close_sequence(s)
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(dtype):
    """Sequences of one to four tokens: a window that is not full yet, a softmax over one key."""
    for cfg_name in ("ALPHA", "GAMMA"):
        cfg = getattr(dm, cfg_name)
        folder = folder_for(cfg_name, cfg, 5)
        m = load(folder, dtype)
        for n in (1, 2, 3, 4):
            toks = tokens_for(cfg, n, 20 + n)
            for cuts in ([n], []):
                s = m.open_sequence()
                check(feed(m, s, toks, cuts), plain_logits(folder, toks), dtype, f"{cfg_name}: {n} tokens, cuts {cuts}",
                      outliers=loose(dtype, 1))
                m.close_sequence(s)
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(dtype):
    """Three prompts of different lengths as one batch, then decoded together while the shorter ones leave;
    every sequence must get what it gets alone."""
    cfg = dm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    lens, prompt = [9, 140, 71], [5, 131, 66]
    seqs = [tokens_for(cfg, n, 30 + i) for i, n in enumerate(lens)]
    m = load(folder, dtype)
    slots = [m.open_sequence() for _ in seqs]
    got = [[] for _ in seqs]
    out = m.step([(slots[i], seqs[i][:prompt[i]]) for i in range(3)], [list(range(p)) for p in prompt]).cpu().numpy()
    at = 0
    for i, p in enumerate(prompt):
        got[i].append(out[at:at + p])
        at += p
    pos = list(prompt)
    while any(pos[i] < lens[i] for i in range(3)):
        live = [i for i in range(3) if pos[i] < lens[i]]
        out = m.step([(slots[i], [seqs[i][pos[i]]]) for i in live]).cpu().numpy()
        for r, i in enumerate(live):
            got[i].append(out[r:r + 1])
            pos[i] += 1
            if pos[i] == lens[i]:
                m.close_sequence(slots[i])
    m.engine.check_device()
    for i in range(3):
        check(np.concatenate(got[i], 0), plain_logits(folder, seqs[i]), dtype, f"sequence {i} in the batch",
              outliers=loose(dtype, lens[i]))
    if dtype == "float32":
        alone = load(folder, dtype)
        s = alone.open_sequence()
        one = feed(alone, s, seqs[2], [prompt[2]])
        assert np.abs(one - np.concatenate(got[2], 0)).max() <= 2e-5 * max(1.0, np.abs(one).max())
        alone.close()
    m.close()


def test_many_sequences_in_one_token_steps():
    """Batches of one-token steps of the sizes at which another kernel takes the products and the experts (8, 17, 40, 70
    sequences of different lengths), against the plain implementation."""
    cfg = dm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    m = load(folder, "bfloat16", max_tokens=70 * 128)
    for n in (8, 17, 40, 70):
        lens = [3 + (7 * i) % 75 for i in range(n)]
        seqs = [tokens_for(cfg, lens[i] + 2, 500 + (i % 12)) for i in range(n)]          # (twelve token streams, cut at many lengths)
        slots = [m.open_sequence() for _ in range(n)]
        m.step([(slots[i], seqs[i][:lens[i]]) for i in range(n)], [[] for _ in range(n)])
        for k in range(2):
            out = m.step([(slots[i], [seqs[i][lens[i] + k]]) for i in range(n)]).cpu().numpy()
        ref = np.stack([plain_logits(folder, seqs[i])[-1] for i in range(n)])
        check(out, ref, "bfloat16", f"{n} sequences", outliers=loose("bfloat16", n))
        for s in slots:
            m.close_sequence(s)
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_used_again(dtype):
    """A sequence that takes the slot and the pages another one left must not see them; the windows' groups give
    pages back while a sequence grows, and those are used again too."""
    cfg = dm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    a, b, c = tokens_for(cfg, 130, 40), tokens_for(cfg, 90, 41), tokens_for(cfg, 70, 42)
    m = load(folder, dtype, max_tokens=512)
    sa = m.open_sequence()
    feed(m, sa, a, [100])
    sb = m.open_sequence()
    gb = [feed(m, sb, b[:50], [50])]
    m.close_sequence(sa)
    sc = m.open_sequence()                      # takes a's slot and pages while b is still live
    assert sc == sa
    gc = feed(m, sc, c, [33, 2])
    gb.append(feed(m, sb, b[50:], [7]))
    m.engine.check_device()
    check(gc, plain_logits(folder, c), dtype, "the sequence in the used slot", outliers=loose(dtype, 70))
    check(np.concatenate(gb, 0), plain_logits(folder, b), dtype, "the sequence that stayed", outliers=loose(dtype, 90))
    m.engine.cache.check()
    m.close()


def _shows(cfg, tensors, toks, ref, change, what, factor=30, least=5):
    """``change`` (a function of copies of configuration and 64-bit tensors) must move the plain implementation's logits."""
    other_cfg, other = copy.deepcopy(cfg), _double(tensors)
    change(other_cfg, other)
    moved = np.abs(pd.forward(other_cfg, other, toks).numpy() - ref).max(-1)
    scale = max(1.0, float(np.abs(ref).max()))
    assert (moved > factor * TOL["float32"] * scale).sum() >= least, f"the test's model does not show {what}"


def test_keys_at_the_windows_edges_decide():
    """Attention alone with a sharp softmax (scores of tens): a position's output is mostly its best key's value, so a
    window one position too long or too short changes whole rows, and so do the gate, a missing head norm, values
    that are normed or turned, and a missing gain of the stretched rotation.  Prompts that end on, before and after the
    window's length and the pages' edges, pieces of two tokens, and single tokens while the window passes over them."""
    cfg = dm.only(dm.ALPHA, 0, mlp=False)
    tensors = dm.draw(cfg, 17, sharp=2.2)
    folder = dm.write_folder(cfg, tensors)
    toks = tokens_for(cfg, 170, 3)
    ref = plain_logits(folder, toks)
    for off in (-1, 1):
        def window(c, t):
            c["layers"][0]["mixer"]["mask"]["size"] += off
        _shows(cfg, tensors, toks, ref, window, "its window's edge")

    def no_gate(c, t):
        t["l0.mix.g"] = t["l0.mix.g"] * 0.0

    def plain_rotation(c, t):
        del c["layers"][0]["mixer"]["rot"]["scaling"]

    def norm_weight(c, t):
        t["l0.mix.k.norm"] = t["l0.mix.k.norm"].flip(0)
    for change, what in ((no_gate, "the gate"), (plain_rotation, "the stretched rotation"), (norm_weight, "the key norm's weight")):
        _shows(cfg, tensors, toks, ref, change, what)
    keep = pd.keys_and_values
    for pick, what in ((lambda k, v: (k, k), "that the values are the keys before norm and rotation"), (lambda k, v: (v, v), "the keys' norm")):
        pd.keys_and_values = lambda *a: pick(*keep(*a))
        try:
            _shows(cfg, tensors, toks, ref, lambda c, t: None, what)
        finally:
            pd.keys_and_values = keep
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([170], [19], [20, 2, 2], [21], [63, 1, 1, 20, 2], [64, 19, 21, 20], [5]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}")
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


@pytest.mark.parametrize("index,size", [(0, 64), (0, 63), (0, 65), (0, 128), (1, 96)])
def test_windows_that_end_on_page_borders(index, size):
    """Windows of a page, one position less and more, two pages: each edge decides (sharp softmax), in one prompt, in
    pieces and one by one."""
    cfg = dm.only(dm.ALPHA, index, mlp=False)
    cfg["layers"][0]["mixer"]["mask"]["size"] = size
    tensors = dm.draw(cfg, 37, sharp=2.2)
    folder = dm.write_folder(cfg, tensors)
    toks = tokens_for(cfg, 200, 8)
    ref = plain_logits(folder, toks)
    for off in (-1, 1):
        def window(c, t):
            c["layers"][0]["mixer"]["mask"]["size"] += off
        _shows(cfg, tensors, toks, ref, window, "its window's edge", factor=10, least=1)
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([200], [size, 2, 2], [size - 1], [64, 64, 2]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"window {size} cuts {cuts}")
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


def test_far_keys_and_page_edges():
    """Attention over all earlier positions with a sharp softmax: the logits late in a sequence hang on single keys
    hundreds of positions back (the test changes early tokens and sees late logits move) and on the rotation's
    frequencies; pieces end on, before and after the pages' edges."""
    cfg = dm.only(dm.ALPHA, 0, mlp=False)
    del cfg["layers"][0]["mixer"]["mask"]
    tensors = dm.draw(cfg, 23, sharp=2.5)
    folder = dm.write_folder(cfg, tensors)
    toks = tokens_for(cfg, 330, 50)
    ref = plain_logits(folder, toks)
    scale = max(1.0, float(np.abs(ref).max()))
    other = list(toks)
    for j in range(8):
        other[j] = (other[j] + 1 + j) % cfg["vocab"]
    moved = np.abs(plain_logits(folder, other)[300:] - ref[300:]).max(-1)
    assert (moved > 30 * TOL["float32"] * scale).sum() >= 3, "the test's model does not look far back"

    def halves(c, t):
        c["layers"][0]["mixer"]["rot"]["scaling"]["factor"] *= 1.1
    _shows(cfg, tensors, toks, ref, halves, "the rotation far back")
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([330], [63, 1, 1, 63, 2], [129], [64, 64, 64], [65, 63], [320]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}")
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


def test_router_correction_groups_identity_and_clipping_show():
    """A mixture behind a window of one, its choice decided by a correction that is negative for most outputs (a dropped
    group must not win by counting as zero), its weights the scores without it, some choices the input itself, the gate
    and the up projection clipped hard: each of these moves the plain implementation's logits, and the library follows
    for few tokens (a kernel an expert row) and many (grouped products)."""
    cfg = dm.only(dm.ALPHA, 4)
    cfg["layers"][0]["mlp"] = {"kind": "moe", "expert": {"ff": 24, "limit": 0.5},
                               "router": {"experts": 7, "top": 4, "identity": 5, "groups": {"count": 4, "keep": 2}}}
    tensors = dm.draw(cfg, 29)
    tensors["l0.mlp.correction"] = (tensors["l0.mlp.correction"].float() * 2 - 1.2).to(torch.bfloat16)
    folder = dm.write_folder(cfg, tensors)
    toks = tokens_for(cfg, 120, 6)
    ref = plain_logits(folder, toks)
    r = lambda c: c["layers"][0]["mlp"]["router"]
    ids, _ = pd.route(pd.dynamic_tanh(_double(tensors)["embed"][torch.tensor(toks)], _double(tensors), "l0.norm1"), _double(tensors), "l0.mlp.", r(cfg))
    assert (ids >= 7).any() and (ids < 7).any()

    def zero(c, t):
        t["l0.mlp.correction"] = t["l0.mlp.correction"] * 0.0

    def one_group(c, t):
        del r(c)["groups"]

    def limit(c, t):
        c["layers"][0]["mlp"]["expert"]["limit"] = 0.6
    for change, what in ((zero, "the correction"), (one_group, "the groups"), (limit, "the limit")):
        _shows(cfg, tensors, toks, ref, change, what)
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([120], [100, 6], [20, 2, 3]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"router, cuts {cuts}", outliers=loose(dtype, 120))
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    """A few tokens of prompt, then single tokens across two pages' edges and past the longer window (captured
    steps in bfloat16)."""
    cfg = dm.BETA
    folder = folder_for("BETA", cfg, 9)
    toks = tokens_for(cfg, 160, 60)
    m = load(folder, dtype)
    s = m.open_sequence()
    got = feed(m, s, toks, [3])
    m.engine.check_device()
    check(got, plain_logits(folder, toks), dtype, "long decoding", outliers=loose(dtype, 160))
    m.close()


def _greedy(folder, prompt, n):
    pcfg, t = dm.read_folder(folder)
    seq = list(prompt)
    for _ in range(n):
        logits = pd.forward(pcfg, t, seq)[-1]
        top2 = torch.topk(logits, 2).values
        if float(top2[0] - top2[1]) < 1e-3:        # a tie within rounding proves nothing either way
            break
        seq.append(int(logits.argmax()))
    return seq[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Model.generate, greedy, for prompts of different lengths in one call: the tokens the plain
    implementation chooses; and the on-device loop chooses what Model.generate chooses."""
    from gopherllm_b200.sampling.sampler import DeviceSampler, SamplerConfig
    cfg = dm.GAMMA
    folder = folder_for("GAMMA", cfg, 3)
    prompts = [tokens_for(cfg, n, 70 + n) for n in (4, 37, 66)]
    m = load(folder, "float32")
    outs = m.generate(prompts, max_tokens=8, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, stop_tokens=())
    for p, o in zip(prompts, outs):
        want = _greedy(folder, p, 8)
        assert o.tokens[:len(want)] == want, (o.tokens, want)
    m.close()
    mb = load(folder_for("ALPHA", dm.ALPHA, 5), "bfloat16")
    prompt = tokens_for(dm.ALPHA, 21, 90)
    want = mb.generate([prompt], max_tokens=12, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, stop_tokens=())[0].tokens
    assert len(want) == 12
    s = mb.open_sequence()
    first = int(mb.step([(s, prompt)])[0].argmax())
    assert first == want[0]
    sampler = DeviceSampler(SamplerConfig.greedy(), [1], [prompt], dm.ALPHA["vocab"], mb.engine.device)
    chosen = mb.engine.decode_loop([s], [first], 11, sampler).cpu().numpy()[:, 0].tolist()
    assert [first] + chosen == want
    mb.engine.check_device()
    mb.close()


def test_command_line_generates():
    """python -m gopherllm_b200 on a Dibedra folder: greedy tokens equal the plain implementation's, and the
    isolated kernel bench knows the parts' products."""
    import os
    import subprocess
    import sys
    cfg = dm.GAMMA
    folder = folder_for("GAMMA", cfg, 3)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    run = lambda *a: subprocess.run([sys.executable, "-m", "gopherllm_b200", folder, *a], cwd=root,
                                    capture_output=True, text=True, timeout=600)
    prompt = tokens_for(cfg, 9, 77)
    want = _greedy(folder, prompt, 5)
    p = run("--prompt", " ".join(map(str, prompt)), "--max-tokens", "5", "--temp", "0", "--repeat-penalty", "1",
            "--dtype", "float32", "--stop", "100000")
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(x) for x in p.stdout.split()][:len(want)] == want
    p = run("--kernel-bench-json", "--kernel-bench-runs", "2")
    assert p.returncode == 0, p.stderr[-2000:]
    assert json.loads(p.stdout)["kernels"]


def test_replay_of_a_trace(tmp_path):
    """The trace runner's loop on a Dibedra model: a batch of two requests, one ends, the other goes on."""
    from gopherllm_b200.engine.replay import run
    cfg = dm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    a, b = tokens_for(cfg, 70, 80), tokens_for(cfg, 12, 81)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 63, 65]},
                                                 {"id": "b", "tokens": b[:11], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]},
                                                 {"id": "b", "tokens": b[11:], "want": [0]}], "end": ["b"]})]
    lines += [json.dumps({"step": 2 + i, "entries": [{"id": "a", "tokens": [a[67 + i]], "want": [0]}],
                          "end": ["a"] if i == 2 else []}) for i in range(3)]
    m = load(folder, "float32")
    said = []
    run(m, lines, str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(5)]
    ra, rb = plain_logits(folder, a), plain_logits(folder, b)
    got0 = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(3, -1)
    check(got0, ra[[0, 63, 65]], "float32", "step 0")
    got1 = np.fromfile(tmp_path / "1.f32", dtype="<f4").reshape(2, -1)
    check(got1, np.stack([ra[66], rb[11]]), "float32", "step 1")
    got4 = np.fromfile(tmp_path / "4.f32", dtype="<f4").reshape(1, -1)
    check(got4, ra[69:70], "float32", "step 4")
    assert not m.engine.cache.live_slots()
    m.close()


def test_kernels_of_the_design_alone():
    """The squashing, the gate, the clipped gated form, the router's choice and the experts with identity choices,
    each against torch at sizes of their own."""
    from gopherllm_b200 import ops
    dev = torch.device("cuda:0")
    g = torch.Generator().manual_seed(5)
    for R, D in ((7, 36), (300, 64), (3, 5)):
        x, w, b, alpha = torch.randn(R, D, generator=g) * 3, torch.randn(D, generator=g), torch.randn(D, generator=g), torch.tensor([0.7])
        rows = torch.tensor([R - 1, 0], dtype=torch.int32)
        want = torch.tanh(alpha.double() * x.double()) * w.double() + b.double()
        for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2)):
            got = ops.dynamic_tanh(x.to(dev), w.to(dev), b.to(dev), alpha.to(dev), dtype).double().cpu()
            assert (got - want).abs().max() <= tol * want.abs().max(), (R, D, dtype)
            got = ops.dynamic_tanh(x.to(dev), w.to(dev), b.to(dev), alpha.to(dev), dtype, rows=rows.to(dev)).double().cpu()
            assert (got - want[rows.long()]).abs().max() <= tol * want.abs().max()
    x, gate = torch.randn(9, 10, generator=g), torch.randn(9, 17, generator=g)
    for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 2e-2)):
        xd, gd = x.to(dev, dtype), gate.to(dev, dtype)
        want = xd.float().cpu() * torch.sigmoid(gd.float().cpu()[:, 4:14])
        assert (ops.sigmoid_gate(xd, gd, 4).float().cpu() - want).abs().max() <= tol
    act = ("clipped", 0.8, 1.702, 1.0)

    def clipped(gg, u):
        gg, u = torch.clamp(gg, max=0.8), torch.clamp(u, -0.8, 0.8)
        return gg * torch.sigmoid(1.702 * gg) * (u + 1.0)
    for F in (16, 10):
        gu = torch.randn(11, 2 * F, generator=g)
        for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 2e-2)):
            gud = gu.to(dev, dtype)
            ref = gud.float().cpu()
            assert (ops.gated_act(gud, act).float().cpu() - clipped(ref[:, :F], ref[:, F:])).abs().max() <= tol
    # the choice: softmax over 12 outputs, a negative correction, three groups of four of which two stay
    logits, corr = torch.randn(200, 12, generator=g) * 2, torch.randn(12, generator=g) * 0.4 - 0.5
    ids, weights = ops.moe_route(logits.to(dev), 3, groups=3, keep=2, softmax_all=True, correction=corr.to(dev), group_largest=True)
    s = torch.softmax(logits.double(), -1)
    choice = (s + corr.double()).view(200, 3, 4)
    keep = torch.topk(choice.amax(-1), 2, dim=-1).indices
    mask = torch.zeros(200, 3, dtype=torch.bool).scatter_(1, keep, True)
    best = torch.topk(choice.masked_fill(~mask[..., None], float("-inf")).view(200, 12), 3, dim=-1).indices
    assert (ids.cpu().long() == best).all() and (weights.cpu() - torch.gather(s, 1, best)).abs().max() <= 1e-6
    xr, wr = torch.randn(40, 20, generator=g), torch.randn(12, 20, generator=g)
    a = ops.moe_route_from(xr.to(dev), wr.to(dev), 3, groups=3, keep=2, softmax_all=True, correction=corr.to(dev), group_largest=True)
    b = ops.moe_route((xr @ wr.T).to(dev), 3, groups=3, keep=2, softmax_all=True, correction=corr.to(dev), group_largest=True)
    assert torch.equal(a[0], b[0]) and (a[1] - b[1]).abs().max() <= 1e-5
    # the experts: 4 of them and 3 identities, few tokens and many, sizes the tensor cores take and others
    for T, W, F in ((3, 24, 16), (5, 10, 6), (300, 64, 32), (70, 36, 12)):
        x, wg = torch.randn(T, W, generator=g), torch.randn(4, 2 * F, W, generator=g) * W ** -0.5
        wd, add = torch.randn(4, W, F, generator=g) * F ** -0.5, torch.randn(T, W, generator=g)
        ids = torch.stack([torch.randperm(7, generator=g)[:3] for _ in range(T)]).to(torch.int32)
        weights = torch.rand(T, 3, generator=g)
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 4e-2)):
            xd, gd, dd = x.to(dev, dtype), wg.to(dev, dtype), wd.to(dev, dtype)
            got = ops.moe_experts(xd, ids.to(dev), weights.to(dev), gd, dd, add=add.to(dev), act=act, identity=True).cpu()
            xs, gs, ds = xd.float().cpu(), gd.float().cpu(), dd.float().cpu()
            want = add.clone()
            for t in range(T):
                for k in range(3):
                    e = int(ids[t, k])
                    y = xs[t] if e >= 4 else ds[e] @ clipped(gs[e, :F] @ xs[t], gs[e, F:] @ xs[t])
                    want[t] += weights[t, k] * y
            assert (got - want).abs().max() <= tol * max(1.0, want.abs().max()), (T, W, F, dtype)


@pytest.mark.parametrize("heads,kv,dim,half,window,gated,from_keys", [
    (8, 2, 64, 16, 0, True, True), (16, 1, 32, 16, 70, True, True), (12, 1, 16, 5, 33, False, True), (4, 4, 128, 64, 130, True, False),
    (6, 2, 80, 40, 64, False, False)])
def test_one_token_attention_with_normed_heads(heads, kv, dim, half, window, gated, from_keys):
    """The one-token kernel that norms, turns, stores, attends and gates against the separate kernels (cache write,
    32-bit attention, gate) on the same cache, for every number of splits."""
    from gopherllm_b200 import ops
    dev = torch.device("cuda:0")
    g = torch.Generator().manual_seed(9)
    lens = [1, 64, 65, 200]
    B, pages_each = len(lens), 4
    ld = (heads + (1 if from_keys else 2) * kv + (heads if gated else 0)) * dim
    qkv = torch.randn(B, ld, generator=g).to(dev, torch.bfloat16)
    k0 = torch.randn(B * pages_each, kv, 64, dim, generator=g).to(dev, torch.bfloat16)
    v0 = torch.randn(B * pages_each, kv, 64, dim, generator=g).to(dev, torch.bfloat16)
    pages = torch.randperm(B * pages_each, generator=g).view(B, pages_each).to(dev, torch.int32)
    ctx = torch.tensor([n - 1 for n in lens], dtype=torch.int32, device=dev)
    ang = torch.randn(B, half, generator=g)
    cos, sin = torch.cos(ang).to(dev), torch.sin(ang).to(dev)
    gq, gk = (1 + 0.3 * torch.randn(dim, generator=g)).to(dev), (1 + 0.3 * torch.randn(dim, generator=g)).to(dev)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    gate_off = (heads + (1 if from_keys else 2) * kv) * dim if gated else -1
    kr, vr = k0.clone(), v0.clone()
    q = torch.empty(B, heads * dim, dtype=torch.bfloat16, device=dev)
    ops.qkv_to_cache(qkv, q, kr, vr, i32(list(range(B))), ctx, pages, heads, kv, dim, 0.2, cos, sin, interleaved=True,
                     q_norm=(gq, None), k_norm=(gk, None), norm_eps=1e-5, norm_rms=True, v_from_k=from_keys)
    want = torch.empty_like(q)
    ops.attention_generic(q, want, kr, vr, i32(list(range(B))), i32([1] * B), ctx, pages, heads, kv, dim, 1, window=window)
    if gated:
        ops.sigmoid_gate(want, qkv, gate_off)
    # the separate kernel itself, against torch
    raw = qkv.float().cpu()
    qh = raw[:, :heads * dim].view(B, heads, dim)
    qh = qh / torch.sqrt((qh * qh).mean(-1, keepdim=True) + 1e-5) * gq.cpu()
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    u, w = qh[..., 0:2 * half:2], qh[..., 1:2 * half:2]
    qh = torch.cat([torch.stack([u * c - w * s, w * c + u * s], -1).flatten(-2), qh[..., 2 * half:]], -1) * 0.2
    assert (q.float().cpu().view(B, heads, dim) - qh).abs().max() <= 1e-2
    for splits in (1, 2, 4, 8):
        kd, vd = k0.clone(), v0.clone()
        out = torch.empty_like(q)
        ops.attention_decode_head(qkv, out, kd, vd, ctx, pages, heads, kv, dim, splits, gq, gk, 1e-5, window, cos, sin, 0.2, True,
                                  from_keys, gate_off)
        assert (kd.float() - kr.float()).abs().max() <= 2e-2 and torch.equal(vd, vr)
        assert (out.float() - want.float()).abs().max() <= 3e-2, splits
    # written where it belongs and nowhere else
    changed = (kd != k0).any(-1).any(1)
    at = torch.zeros_like(changed)
    for b, n in enumerate(lens):
        at[int(pages[b, (n - 1) // 64]), (n - 1) % 64] = True
    assert not (changed & ~at).any()
    ops.check_wait_failures()


@pytest.mark.parametrize("tiles", [1, 2])
@pytest.mark.parametrize("heads,kv,dim,window,gated", [(4, 2, 64, 0, True), (2, 1, 80, 100, True), (3, 3, 16, 64, False), (2, 2, 96, 0, True),
                                                      (2, 1, 128, 300, True)])
def test_prompt_attention_with_a_gate_in_both_block_forms(heads, kv, dim, window, gated, tiles):
    """The tcgen05 prompt kernel with blocks of one tile and of two (where the head size has both), unequal runs behind
    cached positions, with and without a window and a gate, against the 32-bit kernel and the gate's own pass."""
    from ctypes import c_int
    from gopherllm_b200 import ops
    from gopherllm_b200.csrc import catalog
    dev = torch.device("cuda:0")
    g = torch.Generator().manual_seed(13)
    qlens, ctxs = [300, 1, 129, 64], [0, 70, 130, 5]
    B, T, pages_each = len(qlens), sum(qlens), 5
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    q = (0.4 * torch.randn(T, heads * dim, generator=g)).to(dev, torch.bfloat16)
    k = torch.randn(B * pages_each, kv, 64, dim, generator=g).to(dev, torch.bfloat16)
    v = torch.randn(B * pages_each, kv, 64, dim, generator=g).to(dev, torch.bfloat16)
    gate = torch.randn(T, 8 + heads * dim, generator=g).to(dev, torch.bfloat16)
    pages = torch.randperm(B * pages_each, generator=g).view(B, pages_each).to(dev, torch.int32)
    starts = [sum(qlens[:b]) for b in range(B)]
    args = (i32(starts), i32(qlens), i32(ctxs), pages, heads, kv, dim, max(qlens))
    want = torch.empty_like(q)
    ops.attention_generic(q, want, k, v, *args, window=window)
    if gated:
        ops.sigmoid_gate(want, gate, 8)
    lib = ops._lib("attention_prefill_tc.cu", catalog.head_dim_defines(dim))
    lib.gl_attention_prefill_tc_tiles(c_int(tiles))
    try:
        got = torch.empty_like(q)
        ops.attention_prefill_tc(q, got, k, v, *args, window, gate if gated else None, 8)
        torch.cuda.synchronize()
    finally:
        lib.gl_attention_prefill_tc_tiles(c_int(0))
    ops.check_wait_failures()
    assert (got.float() - want.float()).abs().max() <= 3e-2
