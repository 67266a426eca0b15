"""The Nakurax design through the library's loader, cache, step function, scheduler and kernels, against the plain
implementation (tests/plain_nakurax.py) on small models whose weights the tests make themselves."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import nakurax_models as nm
import plain_nakurax as pn

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

# the largest |difference| of a position's logits is bounded by TOL * max(1, max|reference|), the mean over positions by
# MEAN_TOL
TOL = {"float32": 3e-4, "bfloat16": 1e-1}
MEAN_TOL = {"float32": 1e-4, "bfloat16": 3e-2}
_REF = {}
FOLDERS = {}


def plain_logits(folder, tokens):
    key = (folder, tuple(tokens))
    if key not in _REF:
        cfg, t = nm.read_folder(folder)
        _REF[key] = pn.forward(list(tokens), t, cfg).numpy()
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


def check(got, ref, dtype, what=""):
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert np.isfinite(got).all(), what
    err = np.abs(got - ref).max(-1)
    size = max(1.0, float(np.abs(ref).max()))
    worst = int(err.argmax())
    assert err.max() <= TOL[dtype] * size, f"{what} {dtype}: position {worst} differs by {err.max():.3e} (bound {TOL[dtype] * size:.3e})"
    assert err.mean() <= MEAN_TOL[dtype] * size, f"{what} {dtype}: positions differ by {err.mean():.3e} on average (bound {MEAN_TOL[dtype] * size:.3e})"


def tokens_for(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)]


def folder_for(name, cfg, seed, **kw):
    key = (name, seed, tuple(sorted(kw.items())))
    if key not in FOLDERS:
        FOLDERS[key] = nm.write_folder(cfg, nm.draw(cfg, seed, **kw))
    return FOLDERS[key]


def _double(tensors):
    return {k: v.double() for k, v in tensors.items()}


def one_side(cfg, index, left):
    """The pair of ``cfg``'s layer with one side's factor zero: the other mechanism alone."""
    out = nm.only(cfg, index, mlp=False)
    out["layers"][0]["mixer"]["left_scale" if not left else "right_scale"] = 0.0
    return out


# layer sizes nearer a real model's: heads of 64 and 128, a latent of 192, chunks of several pages
WIDE = dict(
    architecture="Nakurax", vocab=500, width=320, norm={"eps": 1e-6}, streams=4, embedding={"scale": 1.0},
    loop={"start": 0, "stop": 2, "times": 2},
    layers=[
        {"type": "latent_attention", "mixer": {"heads": 16, "dim": 64, "vdim": 64, "kv_rank": 192, "scale": 0.12},
         "mlp": {"kind": "dense", "ff": 512}},
        {"type": "parallel",
         "mixer": {"left": {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 64, "scale": 0.09, "mask": {"size": 150},
                            "rot": {"dims": 64, "base": 10000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 128}}},
                   "right": {"width": 384, "blocks": 2, "conv": 4}, "left_scale": 1.1, "right_scale": 0.8},
         "mlp": {"kind": "dense", "ff": 512}},
    ])
# a latent longer than the tensor-core kernels take
RANK = dict(
    architecture="Nakurax", vocab=100, width=64, norm={"eps": 1e-6}, streams=2, embedding={"scale": 1.0},
    layers=[{"type": "latent_attention", "mixer": {"heads": 8, "dim": 16, "vdim": 24, "kv_rank": 320, "scale": 0.3},
             "mlp": {"kind": "dense", "ff": 64}}])

ALONE = [("latent", nm.only(nm.ALPHA, 0)), ("latent_twelve_heads", nm.only(nm.ALPHA, 2, mlp=False)),
         ("latent_twentyfour_heads", nm.only(nm.BETA, 1)), ("latent_two_heads", nm.only(nm.BETA, 2)),
         ("latent_odd", nm.only(nm.GAMMA, 0)), ("latent_one_head", nm.only(nm.DELTA, 1)), ("latent_long", RANK),
         ("pair", nm.only(nm.ALPHA, 1)), ("pair_bare_one_block", nm.only(nm.ALPHA, 3, mlp=False)),
         ("pair_one_tap", nm.only(nm.BETA, 0)), ("pair_odd", nm.only(nm.GAMMA, 1)), ("pair_chunks_of_one", nm.only(nm.GAMMA, 2)),
         ("pair_one_stream", nm.only(nm.DELTA, 0)),
         ("chunked_attention_alone", one_side(nm.ALPHA, 1, left=True)), ("recurrence_alone", one_side(nm.ALPHA, 1, left=False)),
         ("recurrence_alone_odd", one_side(nm.GAMMA, 2, left=False))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg", ALONE, ids=[a[0] for a in ALONE])
def test_each_mechanism_alone(name, cfg, dtype):
    """One layer of one kind: a whole prompt across a page's edge, then single tokens."""
    folder = folder_for(name, cfg, 11)
    toks = tokens_for(cfg, 78, 1)
    m = load(folder, dtype)
    s = m.open_sequence()
    got = feed(m, s, toks, [70])
    m.engine.check_device()
    check(got, plain_logits(folder, toks), dtype, name)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg_name", ["ALPHA", "BETA", "GAMMA", "DELTA"])
def test_whole_pieces_and_single_tokens(cfg_name, dtype):
    """The same tokens whole, in pieces of many sizes down to two, and mostly one by one."""
    cfg = getattr(nm, cfg_name)
    folder = folder_for(cfg_name, cfg, 5)
    toks = tokens_for(cfg, 150, 2)
    ref = plain_logits(folder, toks)
    m = load(folder, dtype)
    for cuts in ([150], [2, 2, 3, 57, 1, 64, 2, 19], [40]):
        s = m.open_sequence()
        got = feed(m, s, toks, cuts)
        m.close_sequence(s)
        check(got, ref, dtype, f"{cfg_name} cuts {cuts}")
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_nearer_a_real_layer(dtype):
    """Also longer than the recurrence's pieces of 256 tokens, in runs that end just before and behind one."""
    folder = folder_for("WIDE", WIDE, 21, long_memory=True)
    toks = tokens_for(WIDE, 530, 4)
    ref = plain_logits(folder, toks)
    m = load(folder, dtype)
    for cuts in ([530], [130, 66, 324], [255, 2, 256, 2], [257, 260]):
        s = m.open_sequence()
        check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}")
        m.close_sequence(s)
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(dtype):
    """Sequences of one to five tokens: the filter's zeros before the start, a recurrence that starts empty, a chunk of
    one key."""
    for cfg_name in ("ALPHA", "GAMMA"):
        cfg = getattr(nm, cfg_name)
        folder = folder_for(cfg_name, cfg, 5)
        m = load(folder, dtype)
        for n in (1, 2, 3, 4, 5):
            toks = tokens_for(cfg, n, 20 + n)
            for cuts in ([n], []):
                s = m.open_sequence()
                check(feed(m, s, toks, cuts), plain_logits(folder, toks), dtype, f"{cfg_name}: {n} tokens, cuts {cuts}")
                m.close_sequence(s)
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(dtype):
    """Prompts of different lengths as one batch, then decoded together while the shorter ones leave; every sequence
    must get what it gets alone."""
    cfg = nm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    lens, prompt = [9, 140, 71, 4], [5, 131, 66, 1]
    n = len(lens)
    seqs = [tokens_for(cfg, k, 30 + i) for i, k in enumerate(lens)]
    m = load(folder, dtype)
    slots = [m.open_sequence() for _ in seqs]
    got = [[] for _ in seqs]
    out = m.step([(slots[i], seqs[i][:prompt[i]]) for i in range(n)], [list(range(p)) for p in prompt]).cpu().numpy()
    at = 0
    for i, p in enumerate(prompt):
        got[i].append(out[at:at + p])
        at += p
    pos = list(prompt)
    while any(pos[i] < lens[i] for i in range(n)):
        live = [i for i in range(n) if pos[i] < lens[i]]
        out = m.step([(slots[i], [seqs[i][pos[i]]]) for i in live]).cpu().numpy()
        for r, i in enumerate(live):
            got[i].append(out[r:r + 1])
            pos[i] += 1
            if pos[i] == lens[i]:
                m.close_sequence(slots[i])
    m.engine.check_device()
    for i in range(n):
        check(np.concatenate(got[i], 0), plain_logits(folder, seqs[i]), dtype, f"sequence {i} in the batch")
    if dtype == "float32":
        alone = load(folder, dtype)
        s = alone.open_sequence()
        one = feed(alone, s, seqs[2], [prompt[2]])
        assert np.abs(one - np.concatenate(got[2], 0)).max() <= 2e-5 * max(1.0, np.abs(one).max())
        alone.close()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_pieces_beside_single_tokens(dtype):
    """One step with a prompt, a later piece of another sequence and single tokens of two more."""
    cfg = nm.BETA
    folder = folder_for("BETA", cfg, 5)
    seqs = [tokens_for(cfg, k, 130 + i) for i, k in enumerate((90, 100, 70, 67))]
    m = load(folder, dtype)
    slots = [m.open_sequence() for _ in seqs]
    done = [0, 31, 69, 66]
    for i in (1, 2, 3):
        m.step([(slots[i], seqs[i][:done[i]])])
    runs = [(slots[i], seqs[i][done[i]:]) for i in range(4)]
    out = m.step(runs, [list(range(len(r[1]))) for r in runs]).cpu().numpy()
    at = 0
    for i in range(4):
        k = len(seqs[i]) - done[i]
        check(out[at:at + k], plain_logits(folder, seqs[i])[done[i]:], dtype, f"sequence {i}")
        at += k
    m.engine.check_device()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_used_again(dtype):
    """A sequence that takes the slot, the state rows (the recurrence, the filter's inputs) and the pages another one
    left must not see them."""
    cfg = nm.ALPHA
    folder = folder_for("ALPHA", cfg, 5, long_memory=True)
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
    check(gc, plain_logits(folder, c), dtype, "the sequence in the used slot")
    check(np.concatenate(gb, 0), plain_logits(folder, b), dtype, "the sequence that stayed")
    m.engine.cache.check()
    m.close()


def test_keys_at_the_chunks_edges_decide():
    """Chunked attention alone with a sharp softmax: a position's output is mostly the value of its best key, so a chunk
    one position too long or too short changes whole rows.  Prompts and pieces that end on, before and behind chunks' and
    pages' edges, and single tokens across several chunks; chunks that divide a page, that do not, and of more than one."""
    for size in (16, 20, 70):
        cfg = one_side(nm.ALPHA, 1, left=True)
        left = cfg["layers"][0]["mixer"]["left"]
        left["mask"]["size"], left["scale"] = size, 1.0
        tensors = nm.draw(cfg, 17, sharp=2.0)
        folder = nm.write_folder(cfg, tensors)
        toks = tokens_for(cfg, 170, 3)
        ref = plain_logits(folder, toks)
        scale = max(1.0, float(np.abs(ref).max()))
        for off in (-1, 1):
            other = copy.deepcopy(cfg)
            other["layers"][0]["mixer"]["left"]["mask"]["size"] += off
            moved = np.abs(pn.forward(toks, _double(tensors), other).numpy() - ref).max(-1)
            assert (moved > 30 * TOL["float32"] * scale).sum() >= 5, "the test's model does not show its chunks' edges"
        for dtype in ("float32", "bfloat16"):
            m = load(folder, dtype)
            for cuts in ([170], [size - 1], [size, 2, 2], [size + 1], [63, 1, 1, 20, 2], [64, size - 1, size + 1], [5]):
                s = m.open_sequence()
                check(feed(m, s, toks, cuts), ref, dtype, f"chunks of {size}, cuts {cuts}")
                m.close_sequence(s)
            m.engine.check_device()
            m.close()


def test_one_far_key_of_a_latent():
    """Latent attention alone; one token's key, by hand, outscores all others for every query, so everything behind it
    hangs on that one key, across hundreds of positions and several pages."""
    cfg = nm.only(nm.ALPHA, 0, mlp=False)
    t = {k: v.float() for k, v in nm.draw(cfg, 19).items()}
    special = cfg["vocab"] - 1
    H, D = 4, 16
    t["embed"][:, :2] = 0.0
    t["embed"][:, 0] = 1.0                       # every query has this, the special key alone has the other
    t["embed"][special, 1] = 2.0
    t["l0.norm1"][:2] = 1.0
    for h in range(H):
        t["l0.mix.q"][h * D] = 0.0
        t["l0.mix.q"][h * D, 0] = 6.0
        t["l0.mix.uk"][h * D] = 0.0
        t["l0.mix.uk"][h * D, 0] = 3.0
    t["l0.mix.dkv"][0] = 0.0
    t["l0.mix.dkv"][0, 1] = 4.0
    t["l0.mix.dkv.norm"][0] = 1.0
    folder = nm.write_folder(cfg, {k: v.to(torch.bfloat16) for k, v in t.items()})
    toks = [x if x != special else 0 for x in tokens_for(cfg, 400, 9)]
    toks[5] = special
    ref = plain_logits(folder, toks)
    other = list(toks)
    other[5] = 1
    assert np.abs(plain_logits(folder, other)[390:] - ref[390:]).max() > 0.2 * np.abs(ref).max(), "the far key does not show"
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([400], [370], [6, 2, 2, 190], [64, 64, 200]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}")
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


def test_far_tokens_through_the_recurrence():
    """A recurrence alone that forgets slowly: the logits late in a sequence hang on tokens hundreds of positions back,
    through its state; pieces end on, before and behind pages' edges."""
    cfg = one_side(nm.ALPHA, 1, left=False)
    folder = folder_for("recurrence_far", cfg, 7, long_memory=True)
    toks = tokens_for(cfg, 300, 50)
    ref = plain_logits(folder, toks)
    other = [(x + 1) % cfg["vocab"] for x in toks[:20]] + toks[20:]
    moved = np.abs(plain_logits(folder, other)[290:] - ref[290:]).max()
    assert moved > 20 * TOL["float32"] * max(1.0, np.abs(ref).max()), "the test's model forgets its early tokens"
    for dtype in ("float32", "bfloat16"):
        m = load(folder, dtype)
        for cuts in ([300], [63, 1, 1, 63, 2], [129], [64, 64, 64], [200]):
            s = m.open_sequence()
            check(feed(m, s, toks, cuts), ref, dtype, f"cuts {cuts}")
            m.close_sequence(s)
        m.engine.check_device()
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    """A few tokens of prompt, then single tokens across pages' and chunks' edges (captured steps in bfloat16)."""
    cfg = nm.ALPHA
    folder = folder_for("ALPHA", cfg, 9, long_memory=True)
    toks = tokens_for(cfg, 210, 60)
    m = load(folder, dtype)
    s = m.open_sequence()
    got = feed(m, s, toks, [3])
    m.engine.check_device()
    check(got, plain_logits(folder, toks), dtype, "long decoding")
    m.close()


def test_equal_layers_repeat_recorded_launches():
    """Layers of one kind in a row, looped: from the third run on recorded launches are repeated, with each run's own
    tensors, cache entry and next layer; the result is that of running every layer itself."""
    from gopherllm_b200 import ops
    cfg = dict(nm.ALPHA, loop={"start": 2, "stop": 3, "times": 3})
    cfg["layers"] = [nm.ALPHA["layers"][0]] * 7 + [nm.ALPHA["layers"][1]] * 2
    folder = folder_for("repeated", cfg, 5)
    toks = tokens_for(cfg, 90, 2)
    m = load(folder, "float32")
    out = []
    for repeat in (True, False):
        ops.REPEAT_LAYERS, ops.TAPE_REPEATS = repeat, 0
        try:
            s = m.open_sequence()
            out.append(feed(m, s, toks, [40, 30, 20]))
            m.close_sequence(s)
            assert (ops.TAPE_REPEATS > 0) == repeat
        finally:
            ops.REPEAT_LAYERS = True
    assert np.array_equal(out[0], out[1])
    check(out[0], plain_logits(folder, toks), "float32", "repeated layers")
    m.close()


@pytest.mark.parametrize("streams,width", [(1, 7), (2, 64), (3, 36), (4, 2048), (5, 130), (8, 512), (16, 1025)])
def test_streams_kernel(streams, width):
    """Joining and reading n streams against the equations in 64-bit: two branches with factors, one branch, no reading,
    reading alone, selected rows, with a norm and without."""
    from gopherllm_b200 import ops
    g = torch.Generator().manual_seed(streams)
    T = 11
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, a, b = rnd(T, streams, width), rnd(T, width), rnd(T, width)
    mix, out_w, in_w, gamma = rnd(streams, streams), rnd(streams), rnd(streams), rnd(width)
    d = lambda t: t.to(DEV)

    def joined(y):
        return torch.einsum("tsd,su->tud", x.double(), mix.double()) + out_w.double()[None, :, None] * y.double()[:, None, :]

    def read(X, normed=True):
        u = torch.einsum("tsd,s->td", X, in_w.double())
        return u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-5) * gamma.double() if normed else u

    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        h = torch.empty((T, width), dtype=dtype, device=DEV)
        xd = d(x).clone()
        ops.streams_join(xd, [(d(a), 0.7), (d(b), -1.3)], d(mix), d(out_w), d(in_w), d(gamma), 1e-5, h)
        want = joined(0.7 * a - 1.3 * b)
        assert (xd.cpu().double() - want).abs().max() < 2e-5 * max(1.0, float(want.abs().max()))
        ref = read(want)
        assert (h.cpu().double() - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))
        xd = d(x).clone()
        ops.streams_join(xd, [(d(a), 1.0)], d(mix), d(out_w))
        assert (xd.cpu().double() - joined(a)).abs().max() < 2e-5 * max(1.0, float(joined(a).abs().max()))
        xd = d(x).clone()
        ops.streams_read(xd, d(in_w), d(gamma), 1e-5, h)
        ref = read(x.double())
        assert torch.equal(xd.cpu(), x) and (h.cpu().double() - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))
        rows = torch.tensor([9, 0, 4], dtype=torch.int32)
        h3 = torch.empty((3, width), dtype=dtype, device=DEV)
        ops.streams_read(xd, d(in_w), None, 0.0, h3, rows=d(rows))
        ref = read(x.double(), normed=False)[rows.long()]
        assert (h3.cpu().double() - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))


class _Ctx:
    def __init__(self, qlens, slots):
        i = lambda v: torch.tensor(v, dtype=torch.int32).to(DEV)
        self.n_seqs, self.max_qlen = len(qlens), max(qlens)
        self.seq_qlen, self.seq_slot = i(qlens), i(slots)
        self.seq_qstart = i([sum(qlens[:k]) for k in range(len(qlens))])
        self.tok_seq = i([k for k, n in enumerate(qlens) for _ in range(n)])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("blocks,size", [(1, 5), (3, 16), (2, 40), (5, 24), (1, 200), (3, 72)])
def test_gated_unit_kernels(blocks, size, dtype):
    """The gates' products, the decays (from near one to near zero) and the recurrence against 64-bit on the same
    rounded inputs: runs of several lengths from a state that is not zero, then one token a sequence."""
    from gopherllm_b200 import ops
    g = torch.Generator().manual_seed(blocks * size)
    C = blocks * size
    rnd = lambda *s: torch.randn(*s, generator=g)
    ra, ri, rb, ib = rnd(blocks, size, size) / size ** 0.5, rnd(blocks, size, size) / size ** 0.5, rnd(blocks, size), rnd(blocks, size)
    ra, ri = ra.to(dtype), ri.to(dtype)
    lam = torch.linspace(-14.0, 4.0, C)
    rate = (-8.0 * torch.nn.functional.softplus(lam.double())).float()
    w = torch.stack([ra, ri], 2).reshape(blocks, 2 * size, size).contiguous()
    bias = torch.stack([rb.reshape(-1), ib.reshape(-1)], 1).reshape(-1).contiguous()
    state = rnd(6, C + 3)
    dev_state = state.to(DEV)
    S = state[:, :C].double()
    for qlens, slots in (([300, 1, 37], [4, 0, 2]), ([256, 2], [2, 4]), ([1, 1, 1], [0, 2, 4]), ([1] * 6, [5, 4, 3, 2, 1, 0])):
        T = sum(qlens)
        u, y = rnd(T, C).to(dtype), rnd(T, C + 8).to(dtype)
        got = ops.gated_unit(u.to(DEV), w.to(DEV), bias.to(DEV), rate.to(DEV), y.to(DEV), 8, dev_state, _Ctx(qlens, slots)).cpu().double()
        r, i = pn.block_gate(u.double(), ra.double(), rb.double()), pn.block_gate(u.double(), ri.double(), ib.double())
        log_a = rate.double() * r
        a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u.double()
        want = torch.zeros(T, C, dtype=torch.float64)
        at = 0
        for n, slot in zip(qlens, slots):
            for t in range(at, at + n):
                S[slot] = a[t] * S[slot] + b[t]
                want[t] = S[slot] * pn.gelu_tanh(y[t, 8:].double())
            at += n
        tol = 3e-5 if dtype == torch.float32 else 1e-2
        assert ((got - want).abs() <= tol * (1.0 + want.abs())).all(), (qlens, float((got - want).abs().max()))
        kept = dev_state.cpu()
        assert torch.equal(kept[:, C:], state[:, C:])
        assert ((kept[:, :C].double() - S).abs() <= 3e-5 * (1.0 + S.abs())).all(), qlens


def _greedy(folder, prompt, n):
    pcfg, t = nm.read_folder(folder)
    seq = list(prompt)
    for _ in range(n):
        logits = pn.forward(seq, t, pcfg)[-1]
        top2 = torch.topk(logits, 2).values
        if float(top2[0] - top2[1]) < 1e-3:        # a tie within rounding proves nothing either way
            break
        seq.append(int(logits.argmax()))
    return seq[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Model.generate, greedy, for prompts of different lengths in one call: the tokens the plain implementation
    chooses."""
    cfg = nm.GAMMA
    folder = folder_for("GAMMA", cfg, 3)
    prompts = [tokens_for(cfg, n, 70 + n) for n in (4, 37, 66)]
    m = load(folder, "float32")
    outs = m.generate(prompts, max_tokens=8, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, stop_tokens=())
    for p, o in zip(prompts, outs):
        want = _greedy(folder, p, 8)
        assert want and o.tokens[:len(want)] == want, (o.tokens, want)
    m.close()
    mb = load(folder, "bfloat16")
    outs_b = mb.generate(prompts, max_tokens=8, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, stop_tokens=())
    assert all(len(o.tokens) == 8 for o in outs_b)
    mb.engine.check_device()
    mb.close()


def test_generation_on_the_device_equals_the_entry_points():
    """The on-device loop (captured steps, two streams) greedy, against Model.generate."""
    from gopherllm_b200.sampling.sampler import DeviceSampler, SamplerConfig
    cfg = nm.ALPHA
    folder = folder_for("ALPHA", cfg, 5)
    prompt = tokens_for(cfg, 21, 90)
    m = load(folder, "bfloat16")
    want = m.generate([prompt], max_tokens=12, temperature=0.0, top_k=0, top_p=1.0, repeat_penalty=1.0, stop_tokens=())[0].tokens
    s = m.open_sequence()
    first = int(m.step([(s, prompt)])[0].argmax())
    assert first == want[0]
    sampler = DeviceSampler(SamplerConfig.greedy(), [1], [prompt], cfg["vocab"], m.engine.device)
    chosen = m.engine.decode_loop([s], [first], 11, sampler).cpu().numpy()[:, 0].tolist()
    assert [first] + chosen == want
    m.engine.check_device()
    m.close()


def test_command_line_generates_and_samples():
    """python -m gopherllm_b200 on a Nakurax folder: greedy tokens equal the plain implementation's, a sampled run with
    the sampler's options ends by length, and the isolated kernel bench knows the parts' products."""
    import os
    import subprocess
    import sys
    cfg = nm.GAMMA
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
    p = run("--prompt", " ".join(map(str, prompt)), "--max-tokens", "12", "--temp", "0.9", "--top-k", "20", "--top-p", "0.95",
            "--seed", "4", "--stop", "100000")
    assert p.returncode == 0, p.stderr[-2000:]
    out = [int(x) for x in p.stdout.split()]
    assert len(out) == 12 and all(0 <= x < cfg["vocab"] for x in out) and "finish=length" in p.stderr
    p = run("--kernel-bench-json", "--kernel-bench-runs", "2")
    assert p.returncode == 0, p.stderr[-2000:]
    assert json.loads(p.stdout)["kernels"]


def test_replay_of_a_trace(tmp_path):
    """The trace runner's loop on a Nakurax model: a batch of two requests, one ends, the other goes on."""
    from gopherllm_b200.engine.replay import run
    cfg = nm.ALPHA
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
    check(np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(3, -1), ra[[0, 63, 65]], "float32", "step 0")
    check(np.fromfile(tmp_path / "1.f32", dtype="<f4").reshape(2, -1), np.stack([ra[66], rb[11]]), "float32", "step 1")
    check(np.fromfile(tmp_path / "4.f32", dtype="<f4").reshape(1, -1), ra[69:70], "float32", "step 4")
    assert not m.engine.cache.live_slots()
    m.close()


def _paged(qlens, ctxs, heads, dim, vdim, g):
    """A cache's pages in scattered order filled with random keys and values: (k, v, pages, context, per-sequence lists)."""
    lens = [q + c for q, c in zip(qlens, ctxs)]
    per = max(-(-n // 64) for n in lens) + 1
    n_pages = len(lens) * per + 3
    order = torch.randperm(n_pages, generator=g)[:len(lens) * per].reshape(len(lens), per)
    k = torch.randn(n_pages, heads, 64, dim, generator=g).to(torch.bfloat16)
    v = torch.randn(n_pages, heads, 64, vdim, generator=g).to(torch.bfloat16)
    ctx = _Ctx(qlens, list(range(len(qlens))))
    i = lambda x: torch.tensor(x, dtype=torch.int32).to(DEV)
    ctx.seq_ctx, ctx.max_len, ctx.total_len = i(ctxs), max(lens), sum(lens)
    ctx.seq_base = i([sum(lens[:j]) for j in range(len(lens))])
    ctx.tok_pos = i([c + j for c, q in zip(ctxs, qlens) for j in range(q)])
    keys = [torch.cat([k[p].transpose(0, 1) for p in order[b]], 0)[:n].double() for b, n in enumerate(lens)]      # [n, heads, dim]
    vals = [torch.cat([v[p].transpose(0, 1) for p in order[b]], 0)[:n].double() for b, n in enumerate(lens)]
    return k.to(DEV), v.to(DEV), order.to(torch.int32).contiguous().to(DEV), ctx, keys, vals


def _attend(q, keys, vals, qlens, ctxs, scale, first_key, sinks=None):
    """64-bit attention of q [T, H, D] on per-sequence keys [n, G, D] and values [n, G, V]."""
    out, at = [], 0
    for b, n in enumerate(qlens):
        H, G = q.shape[1], keys[b].shape[1]
        for j in range(n):
            p = ctxs[b] + j
            lo = first_key(p)
            kk = keys[b][lo:p + 1].repeat_interleave(H // G, 1)
            s = torch.einsum("hd,nhd->hn", q[at + j].double(), kk) * scale
            vv = vals[b][lo:p + 1].repeat_interleave(H // vals[b].shape[1], 1)
            e = torch.exp(s - s.max(-1, keepdim=True).values)
            den = e.sum(-1, keepdim=True)
            if sinks is not None:
                den = den + torch.exp(sinks.double()[:, None] - s.max(-1, keepdim=True).values)
            out.append(torch.einsum("hn,nhv->hv", e / den, vv))
        at += n
    return torch.stack(out).reshape(at, -1)


@pytest.mark.parametrize("tiles", [1, 2])
@pytest.mark.parametrize("chunk", [0, 1, 24, 64, 100, 300])
def test_prompt_kernel_with_chunks_and_a_factor(chunk, tiles):
    """The tcgen05 prompt kernel: scattered pages, shared key heads, runs that start inside chunks, both block forms."""
    from gopherllm_b200 import ops
    from gopherllm_b200.csrc import catalog
    H, G, D = 4, 2, 32
    qlens, ctxs = [300, 2, 65], [0, 129, 63]
    g = torch.Generator().manual_seed(chunk)
    k, v, pages, ctx, keys, vals = _paged(qlens, ctxs, G, D, D, g)
    q = torch.randn(sum(qlens), H * D, generator=g).to(torch.bfloat16)
    lib = ops._lib("attention_prefill_tc.cu", catalog.head_dim_defines(D))
    try:
        lib.gl_attention_prefill_tc_tiles(tiles)
        got = ops.attention_prefill_tc_chunked(q.to(DEV), k, v, ctx, pages, H, G, D, chunk=chunk, score_scale=0.37).cpu().double()
    finally:
        lib.gl_attention_prefill_tc_tiles(0)
    ops.check_wait_failures()
    want = _attend(q.view(-1, H, D), keys, vals, qlens, ctxs, 0.37, lambda p: p - p % chunk if chunk else 0)
    assert (got - want).abs().max() < 3e-2 and (got - want).abs().mean() < 3e-3


@pytest.mark.parametrize("dim,vdim", [(32, 32), (64, 64), (16, 32), (48, 16)])
def test_attention_on_rows(dim, vdim):
    """Keys and values as rows of one matrix, queries inside wider rows: both kernels (equal and unequal sizes)."""
    from gopherllm_b200 import ops
    H = 3
    for qlens, ctxs in (([200, 17, 64], [0, 0, 0]), ([40, 2, 130], [70, 190, 1])):
        g = torch.Generator().manual_seed(dim + vdim)
        lens = [a + b for a, b in zip(qlens, ctxs)]
        ctx = _Ctx(qlens, [0, 1, 2])
        i = lambda x: torch.tensor(x, dtype=torch.int32).to(DEV)
        ctx.seq_ctx, ctx.max_len, ctx.total_len = i(ctxs), max(lens), sum(lens)
        ctx.seq_base = i([sum(lens[:j]) for j in range(3)])
        kv = torch.randn(sum(lens), H * (dim + vdim), generator=g).to(torch.bfloat16)
        proj = torch.randn(sum(qlens), 24 + H * dim + 8, generator=g).to(torch.bfloat16)
        got = ops.attention_rows(proj.to(DEV), 24, kv.to(DEV), ctx, torch.zeros((3, 4), dtype=torch.int32, device=DEV), H, dim, vdim, 0.2)
        ops.check_wait_failures()
        base = [sum(lens[:j]) for j in range(3)]
        keys = [kv[b:b + n, :H * dim].view(n, H, dim).double() for b, n in zip(base, lens)]
        vals = [kv[b:b + n, H * dim:].view(n, H, vdim).double() for b, n in zip(base, lens)]
        want = _attend(proj[:, 24:24 + H * dim].reshape(-1, H, dim), keys, vals, qlens, ctxs, 0.2, lambda p: 0)
        got = got.cpu().double()
        assert (got - want).abs().max() < 3e-2 and (got - want).abs().mean() < 3e-3


@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 4, 16, 32), (6, 2, 32, 16), (5, 1, 64, 64), (12, 3, 48, 48), (40, 2, 32, 32)])
def test_one_token_attention_of_any_group(heads, groups, dim, vdim):
    """The kernel whose rows are query heads, from one head a key head to twenty: windows, chunks, sinks, contexts cut
    into ranges, some of them empty."""
    from gopherllm_b200 import ops
    ctxs = [0, 1, 63, 64, 200, 390]
    g = torch.Generator().manual_seed(heads)
    k, v, pages, ctx, keys, vals = _paged([1] * len(ctxs), ctxs, groups, dim, vdim, g)
    q = torch.randn(len(ctxs), heads * dim, generator=g).to(torch.bfloat16)
    sinks = torch.randn(heads, generator=g)
    for kw, lo in (({}, lambda p: 0), (dict(chunk=50), lambda p: p - p % 50), (dict(window=70), lambda p: max(0, p - 69))):
        for s in (None, sinks):
            got = ops.attention_mixed(q.to(DEV), k, v, ctx, pages, heads, groups, dim, vdim, score_scale=0.3,
                                      sinks=None if s is None else s.to(DEV), **kw).cpu().double()
            want = _attend(q.view(-1, heads, dim), keys, vals, [1] * len(ctxs), ctxs, 0.3, lo, s)
            assert (got - want).abs().max() < 3e-2, (kw, s is not None, float((got - want).abs().max()))


@pytest.mark.parametrize("batch", [1, 7, 20])
@pytest.mark.parametrize("heads,rank,out", [(4, 32, 24), (12, 48, 64), (32, 256, 40)])
def test_one_token_attention_with_a_product_behind_it(heads, rank, out, batch):
    """Values inside the key rows, ranges put together and a matrix per head behind them, gated or not, with and without
    a sink, against the separate kernels' mathematics in 64-bit."""
    from gopherllm_b200 import ops
    g = torch.Generator().manual_seed(rank)
    ctxs = [int(x) for x in torch.randint(0, 500, (batch,), generator=g)]
    k, _, pages, ctx, keys, _ = _paged([1] * batch, ctxs, 1, rank, rank, g)
    q = torch.randn(batch, heads * rank, generator=g).to(torch.bfloat16)
    w = (torch.randn(heads, out, rank, generator=g) / rank ** 0.5).to(torch.bfloat16)
    gate = torch.randn(batch, heads + 9, generator=g).to(torch.bfloat16)
    sinks = torch.randn(heads, generator=g)
    for s in (None, sinks):
        for gt in (None, gate):
            got = ops.attention_mixed(q.to(DEV), k, k, ctx, pages, heads, 1, rank, rank, score_scale=0.2, values_in_keys=True,
                                      sinks=None if s is None else s.to(DEV), project=w.to(DEV), gate=None if gt is None else gt.to(DEV),
                                      gate_off=5).cpu().double()
            y = _attend(q.view(-1, heads, rank), keys, keys, [1] * batch, ctxs, 0.2, lambda p: 0, s).view(batch, heads, rank)
            want = torch.einsum("hnr,bhr->bhn", w.double(), y)
            if gt is not None:
                want = want * torch.sigmoid(gt[:, 5:5 + heads].double())[:, :, None]
            assert (got - want.reshape(batch, -1)).abs().max() < 3e-2


def test_prompts_on_latents_and_on_keys_built_from_them():
    """Both forms of a prompt's latent attention, in pieces that go on from cached latents: each against the plain
    implementation, with key and value sizes equal and unequal."""
    from gopherllm_b200.parts import attention
    for name, cfg in (("latent", nm.only(nm.ALPHA, 0)), ("latent_twentyfour_heads", nm.only(nm.BETA, 1)), ("WIDE_latent", nm.only(WIDE, 0))):
        folder = folder_for(name, cfg, 11)
        toks = tokens_for(cfg, 200, 8)
        ref = plain_logits(folder, toks)
        m = load(folder, "bfloat16")
        for built in (True, False):
            attention.LATENT_BUILDS_KEYS = built
            try:
                for cuts in ([200], [90, 110], [33, 64, 103]):
                    s = m.open_sequence()
                    check(feed(m, s, toks, cuts), ref, "bfloat16", f"{name}, keys built {built}, cuts {cuts}")
                    m.close_sequence(s)
                a, b = m.open_sequence(), m.open_sequence()
                m.step([(a, toks[:50])])
                out = m.step([(a, toks[50:120]), (b, toks[:150])], [list(range(70)), list(range(150))]).cpu().numpy()
                check(out[:70], ref[50:120], "bfloat16", f"{name}, keys built {built}, a piece in a batch")
                check(out[70:], ref[:150], "bfloat16", f"{name}, keys built {built}, a prompt in a batch")
                m.close_sequence(a)
                m.close_sequence(b)
            finally:
                attention.LATENT_BUILDS_KEYS = True
        m.engine.check_device()
        m.close()


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolution_of_many_tokens(taps, dtype):
    """Without an activation and with silu: sequences whose ends cut the groups of four tokens everywhere, some of one
    token, going on from kept inputs, as many tokens as the form that shares its rows takes."""
    from gopherllm_b200 import ops
    g = torch.Generator().manual_seed(taps)
    C = 1024
    qlens = [1, 2, 601, 3, 5, 1, 700, 1203, 130]
    T, B = sum(qlens), len(qlens)
    ctx = _Ctx(qlens, list(range(B)))
    x = torch.randn(T, C + 16, generator=g).to(dtype)
    w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    tail0 = torch.randn(B, 3 + C * (taps - 1), generator=g)
    for silu in (False, True):
        state = tail0.clone().to(DEV)
        got = ops.conv_silu(x.to(DEV), w.to(DEV), bias.to(DEV), state, 3, ctx, x_off=8, silu=silu).cpu().double()
        at = 0
        for b, n in enumerate(qlens):
            before = tail0[b, 3:].view(C, taps - 1).double().T                       # oldest first
            rows = torch.cat([before, x[at:at + n, 8:8 + C].double()], 0)
            want = bias.double() + sum(rows[j:j + n] * w[:, j].double() for j in range(taps))
            if silu:
                want = want * torch.sigmoid(want)
            tol = 1e-4 if dtype == torch.float32 else 1e-2
            assert ((got[at:at + n] - want).abs() <= tol * (1.0 + want.abs())).all(), (b, silu)
            kept = state[b, 3:].view(C, taps - 1).cpu().double().T
            assert torch.equal(kept, rows[n:]) and torch.equal(state[b, :3].cpu(), tail0[b, :3])
            at += n


@pytest.mark.parametrize("half", [0, 4, 6, 16])
def test_neighbouring_dims_turned_piece_by_piece(half):
    """Queries turned, scaled and left, keys and values to scattered cache rows, in 16-byte pieces: bfloat16 against
    64-bit on the same inputs."""
    from gopherllm_b200 import ops
    H, G, D, V = 6, 2, 32, 40
    qlens, ctxs = [70, 1, 9], [5, 64, 127]
    g = torch.Generator().manual_seed(half)
    _, _, pages, ctx, _, _ = _paged(qlens, ctxs, G, D, V, g)
    T = sum(qlens)
    per = int(pages.shape[1])
    k = torch.full((per * 3 + 3, G, 64, D), 7.0, dtype=torch.bfloat16, device=DEV)
    v = torch.full((per * 3 + 3, G, 64, V), 7.0, dtype=torch.bfloat16, device=DEV)
    qkv = torch.randn(T, (H + G) * D + G * V + 8, generator=g).to(torch.bfloat16)
    angle = torch.randn(T, half, generator=g, dtype=torch.float64)
    cos, sin = torch.cos(angle).float(), torch.sin(angle).float()
    for scale in (1.0, 0.3):
        q = ops.qkv_rownorm_to_cache(qkv.to(DEV), k, v, ctx, pages, H, G, D, V, scale, cos.to(DEV) if half else None,
                                     sin.to(DEV) if half else None, True, None, None, 0.0).cpu().double().view(T, H, D)

        def turned(x):
            y = x.double().clone()
            if half:
                a, b = x[..., 0:2 * half:2].double(), x[..., 1:2 * half:2].double()
                c, s = cos.double()[:, None], sin.double()[:, None]
                y[..., 0:2 * half:2], y[..., 1:2 * half:2] = a * c - b * s, b * c + a * s
            return y
        assert (q - scale * turned(qkv[:, :H * D].view(T, H, D))).abs().max() < 2e-2
        keys, vals = turned(qkv[:, H * D:(H + G) * D].view(T, G, D)), qkv[:, (H + G) * D:(H + G) * D + G * V].view(T, G, V)
        at, pg = 0, pages.cpu()
        for b, n in enumerate(qlens):
            for j in range(n):
                p = ctxs[b] + j
                page, r = int(pg[b, p // 64]), p % 64
                assert (k[page, :, r].cpu().double() - keys[at + j]).abs().max() < 2e-2
                assert torch.equal(v[page, :, r].cpu(), vals[at + j])
            at += n
        written = sum(qlens)
        assert int((k[..., 0] != 7.0).sum()) <= written * G and int((v.float() != 7.0).any(-1).sum()) <= written * G
