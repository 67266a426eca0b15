"""Arrangements of norm, mixer and feed-forward in one layer."""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..config.specs import BlockSpec
from .base import Block, ParamSpec, Part, build_feed_forward, build_mixer, build_norm, register_block


class AssembledBlock(Block):
    """A block put together from child parts.  ``children()`` says which: a dict from slot name to
    part, in a fixed order; parameters, loading and the capture flag walk it, so an arrangement with
    more parts (a norm after a branch, a third branch) overrides ``children`` and ``forward`` and
    nothing else.  A parameter's key is "<slot>/<the child's own key>".  This base builds the usual
    four from the spec: ``norm``, ``mixer``, ``ffn`` and, if the spec has one, ``norm2``."""

    def __init__(self, spec: BlockSpec):
        self.spec = spec
        self.norm = build_norm(spec.norm)
        self.norm2 = build_norm(spec.norm2) if spec.norm2 is not None else None
        self.mixer = build_mixer(spec.mixer)
        self.ffn = build_feed_forward(spec.ffn) if spec.ffn is not None else None

    def children(self) -> Dict[str, object]:
        c = {"norm": self.norm}
        if self.norm2 is not None:
            c["norm2"] = self.norm2
        c["mixer"] = self.mixer
        if self.ffn is not None:
            c["ffn"] = self.ffn
        return c

    def parameters(self) -> Dict[str, ParamSpec]:
        return {f"{slot}/{k}": v for slot, part in self.children().items() for k, v in part.parameters().items()}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        for slot, part in self.children().items():
            pre = slot + "/"
            part.load({k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)})

    def cache_request(self):
        return self.mixer.cache_request()

    def products(self):
        return [(f"{slot}.{name}", w, b, act) for slot, part in self.children().items()
                for name, w, b, act in part.products()]

    @property
    def capturable(self):
        return all(part.capturable for part in self.children().values())

    @property
    def launches_only(self):
        return all(part.launches_only for part in self.children().values())


class ParallelBlock(AssembledBlock):
    """x ← (x + ffn(n)) + mixer(n), n = norm(x): one norm feeds both branches
    (model.go:2738-2740) and both are added to the residual, the feed-forward
    first (model.go:2812-2815).  A layer without a feed-forward (``spec.ffn`` None) is x ← x + mixer(n)."""

    def _decode_step_as_one_kernel(self, x, ctx, cache) -> bool:
        """With one token a sequence a layer is a stream of weights and cached keys and values; where
        every part offers its fused form and the kernel takes the sizes, the whole block runs as one
        persistent kernel that keeps that stream going from the norm to the residual sum."""
        if not (ctx.is_decode and ctx.act_dtype == torch.bfloat16 and self.ffn is not None and self.norm.fusable is not None
                and self.mixer.decode_fusable is not None and self.ffn.fusable is not None):
            return False
        m = self.mixer.decode_fusable(ctx, cache)
        if m is None:
            return False
        w_up, b_up, act, w_down, b_down = self.ffn.fusable()
        half = 0 if m["cos"] is None else m["cos"].shape[1]
        if not ops.decode_layer_takes(x, m["w_qkv"], w_up, m["w_out"], w_down, m["k"].dtype, m["head_dim"],
                                      m["num_heads"] // m["num_kv_heads"], half, m["interleaved"], m["head_norm"],
                                      longest=ctx.max_len):
            return False
        g, b, eps, rms = self.norm.fusable()
        ops.decode_layer(x, g, b, eps, rms, m["w_qkv"], m["b_qkv"], w_up, b_up, act, m["w_out"], m["b_out"],
                         w_down, b_down, m["k"], m["v"], ctx.seq_ctx, m["pages"], m["num_heads"], m["num_kv_heads"],
                         m["head_dim"], m["q_scale"], m["cos"], m["sin"], m["window"], m["writes"])
        return True

    def forward(self, x, ctx, cache):
        if self._decode_step_as_one_kernel(x, ctx, cache):
            return x
        xn = self.norm.forward(x, ctx.act_dtype)
        if self.ffn is None:
            self.mixer.forward(xn, ctx, cache, (x,), x)
            return x
        side = getattr(ctx, "side_stream", None)
        if self.ffn.until_last is not None and self.mixer.until_last is not None:
            # The branches' last products end on the same rows and columns: they run as one product
            # over the joined K where the kernels can (one kernel, one pass over the residual stream),
            # else one after the other.  What comes before them runs on two streams in decode steps:
            # with few tokens every kernel is a stream of weights, and the feed-forward's first product
            # keeps memory busy while the mixer's small kernels start and finish.
            if side is None and self.ffn.first_product is not None and self.mixer.first_product is not None:
                # many tokens: the branches' first products read the same rows and run as one grid
                wm, bm, am = self.mixer.first_product()
                wf, bf, af = self.ffn.first_product()
                ym, yf = ops.linear_fork(xn, wm, bm, am, wf, bf, af, ctx.act_dtype)
                h, w2, b2 = self.ffn.until_last(xn, ctx, first=yf)
                o, wo, bo = self.mixer.until_last(xn, ctx, cache, first=ym)
            elif side is None:
                h, w2, b2 = self.ffn.until_last(xn, ctx)
                o, wo, bo = self.mixer.until_last(xn, ctx, cache)
            else:
                main = torch.cuda.current_stream()
                fork, join = torch.cuda.Event(), torch.cuda.Event()
                fork.record(main)
                side.wait_event(fork)
                with torch.cuda.stream(side):
                    h, w2, b2 = self.ffn.until_last(xn, ctx)
                    join.record(side)
                o, wo, bo = self.mixer.until_last(xn, ctx, cache)
                main.wait_event(join)
            ops.linear_pair(h, w2, b2, o, wo, bo, add0=x, out=x)
            return x
        if side is None or not self.mixer.deferred_add:
            # each branch adds itself onto the residual stream in its last product's epilogue,
            # the feed-forward first: (x + mlp) + attn, the reference's order
            self.ffn.forward(xn, ctx, (x,), x)
            self.mixer.forward(xn, ctx, cache, (x,), x)
            return x
        # Both branches read the same normalised input, so the feed-forward runs on a second
        # stream beside the mixer and leaves its result in a buffer of its own; the mixer's last
        # product adds both the residual and that buffer.  With few tokens every kernel is a
        # stream of weights: the second stream keeps memory busy while the mixer's small kernels
        # start and finish, and nothing of the feed-forward is left on the path from one layer's
        # norm to the next.  The sum is the same three terms in 32-bit, added as (attn + x) + mlp.
        main = torch.cuda.current_stream()
        y = ops.empty(x.shape, torch.float32, x.device)
        fork, join = torch.cuda.Event(), torch.cuda.Event()
        fork.record(main)
        side.wait_event(fork)
        with torch.cuda.stream(side):
            self.ffn.forward(xn, ctx, (), y)
            join.record(side)
        def mlp():                   # resolved by the mixer just before its last product
            main.wait_event(join)
            return y

        self.mixer.forward(xn, ctx, cache, (x, mlp), x)
        return x


class SequentialBlock(AssembledBlock):
    """x ← x + mixer(norm(x)); x ← x + ffn(norm2(x)) (model.go:2806-2811)."""

    def __init__(self, spec: BlockSpec):
        if spec.norm2 is None:
            raise ValueError("a sequential block needs norm2")
        super().__init__(spec)

    def forward(self, x, ctx, cache):
        self.mixer.forward(self.norm.forward(x, ctx.act_dtype), ctx, cache, (x,), x)
        self.ffn.forward(self.norm2.forward(x, ctx.act_dtype), ctx, (x,), x)
        return x


class TwoNormParallelBlock(AssembledBlock):
    """x <- x + (mixer(norm(x)) + ffn(norm2(x))): both branches read the same x, each through a norm of
    its own.  A layer without a feed-forward (``spec.ffn`` None, no norm2) is x <- x + mixer(norm(x))."""

    def __init__(self, spec: BlockSpec):
        if (spec.ffn is None) != (spec.norm2 is None):
            raise ValueError("the second norm comes with the feed-forward: both or neither")
        super().__init__(spec)

    def _norms(self, x, ctx):
        """Both branches' inputs; two RMS norms with the same eps read the row once."""
        a = self.norm.fusable() if self.norm.fusable is not None else None
        b = self.norm2.fusable() if self.norm2.fusable is not None else None
        if a is not None and b is not None and a[3] and b[3] and a[1] is None and b[1] is None and a[2] == b[2]:
            return ops.rms_norm_pair(x, a[0], b[0], a[2], ctx.act_dtype)
        return self.norm.forward(x, ctx.act_dtype), self.norm2.forward(x, ctx.act_dtype)

    def forward(self, x, ctx, cache):
        if self.ffn is None:
            self.mixer.forward(self.norm.forward(x, ctx.act_dtype), ctx, cache, (x,), x)
            return x
        xn, xn2 = self._norms(x, ctx)
        if self.ffn.until_last is not None and self.mixer.until_last is not None:
            # the branches' last products end on the same rows and columns: one product over the joined K
            # where the kernels can, added onto the residual stream in its epilogue
            h, w2, b2 = self.ffn.until_last(xn2, ctx)
            o, wo, bo = self.mixer.until_last(xn, ctx, cache)
            ops.linear_pair(h, w2, b2, o, wo, bo, add0=x, out=x)
            return x
        y = self.ffn.forward(xn2, ctx, (), None)
        self.mixer.forward(xn, ctx, cache, (y, x), x)
        return x


class PostNormBlock(AssembledBlock):
    """x <- x + norm(mixer(x)); x <- x + norm2(ffn(x)): the sublayers read the residual stream itself (rounded to
    the activation type where that is not 32-bit) and what they return is RMS-normed before it is added.  A layer
    without a feed-forward (``spec.ffn`` None, no norm2) is the first half alone.  A mixer that offers
    ``branches`` (two outputs with a factor each) is summed in the pass that norms and adds; that pass also
    leaves the stream's rounded copy for the feed-forward.  Option ``branch_scale`` m: x <- x + m * norm(...) for
    both sublayers (the factor is taken into the norms' weights once, when they are loaded).  Option
    ``hand_on_rounded``: the pass that closes the layer also leaves the stream's rounded copy in the step's context, and
    the next layer of this kind takes it from there instead of rounding the stream again (the model drops the copy
    before a layer that does not take it)."""

    takes_rounded_stream = True

    def __init__(self, spec: BlockSpec):
        if (spec.ffn is None) != (spec.norm2 is None):
            raise ValueError("the second norm comes with the feed-forward: both or neither")
        super().__init__(spec)
        for n in (self.norm, self.norm2):
            if n is not None and not (getattr(n, "rms", False) and n.fusable is not None and not n.spec.bias):
                raise ValueError("a block that norms its sublayers' outputs takes RMS norms without bias")
        self.branch_scale = float(spec.option("branch_scale", 1.0))
        self.hand_on = bool(spec.option("hand_on_rounded", False))
        self.w1 = self.w2 = None                 # the norms' weights times the factor

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        super().load(tensors)
        if self.branch_scale != 1.0:
            self.w1 = (self.norm.fusable()[0] * self.branch_scale).contiguous()
            if self.norm2 is not None:
                self.w2 = (self.norm2.fusable()[0] * self.branch_scale).contiguous()

    def forward(self, x, ctx, cache):
        h = ctx.scratch.pop("stream_rounded", None)
        if h is None or h.shape != x.shape or h.dtype != ctx.act_dtype:
            h = ops.round_rows(x, ctx.act_dtype)
        hand_on = ctx.act_dtype if self.hand_on and ctx.act_dtype != torch.float32 else None
        w, _, eps, _ = self.norm.fusable()
        if self.w1 is not None:
            w = self.w1
        copy = ctx.act_dtype if self.ffn is not None and ctx.act_dtype != torch.float32 else None
        branches = getattr(self.mixer, "branches", None)
        if branches is not None:
            (a, sa), (b, sb) = branches(h, ctx, cache)
            _, h = ops.post_norm_add(a, w, eps, add=x, out=x, scale=sa, second=(b, sb),
                                     rounded=copy if self.ffn is not None else hand_on)
        else:
            y = self.mixer.forward(h, ctx, cache, (), None)
            _, h = ops.post_norm_add(y, w, eps, add=x, out=x, rounded=copy if self.ffn is not None else hand_on)
        if self.ffn is None:
            if hand_on is not None:
                ctx.scratch["stream_rounded"] = h
            return x
        w2, _, eps2, _ = self.norm2.fusable()
        if self.w2 is not None:
            w2 = self.w2
        y = self.ffn.forward(h if h is not None else x, ctx, (), None)
        _, h = ops.post_norm_add(y, w2, eps2, add=x, out=x, rounded=hand_on)
        if hand_on is not None:
            ctx.scratch["stream_rounded"] = h
        return x


class StreamsBlock(AssembledBlock):
    """Hyper-connections: the residual is n streams x_1 .. x_n (option ``streams``) in one tensor [T, n, hidden].  A
    sublayer reads one combination of a token's streams X [n, hidden] and returns into all of them,
        y = sublayer(norm(X^T i)),   X <- M^T X + o y^T,
    with i ("in"), M ("mix", row s: where stream s goes) and o ("out") of its own for the mixer ("hc1") and the feed-forward ("hc2"); a layer without a feed-forward
    (``spec.ffn`` None, no norm2) is the first half alone.  One kernel joins a sublayer's result, reads the streams for
    the next sublayer and norms what it read, across layers too: a run finds its input in the step's context and leaves
    the next run's there (see Block).  A mixer that offers ``branches`` is summed inside that kernel."""

    def __init__(self, spec: BlockSpec):
        if (spec.ffn is None) != (spec.norm2 is None):
            raise ValueError("the second norm comes with the feed-forward: both or neither")
        super().__init__(spec)
        for n in (self.norm, self.norm2):
            if n is not None and not (getattr(n, "rms", False) and n.fusable is not None and not n.spec.bias):
                raise ValueError("a block of several streams takes RMS norms without bias")
        self.streams = int(spec.option("streams", 1))
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"a block works on 1 to {ops.MAX_STREAMS} streams, not {self.streams}")
        self.hc1 = StreamWeights(self.streams)
        self.hc2 = StreamWeights(self.streams) if self.ffn is not None else None

    def children(self) -> Dict[str, object]:
        c = super().children()
        c["hc1"] = self.hc1
        if self.hc2 is not None:
            c["hc2"] = self.hc2
        return c

    def opening(self):
        gamma, _, eps, _ = self.norm.fusable()
        return self.hc1.weight_in, gamma, eps

    def forward(self, x, ctx, cache):
        h = ctx.scratch["streams_input"]                # every run's input passes through this one buffer
        branches = getattr(self.mixer, "branches", None)
        y = branches(h, ctx, cache) if branches is not None else [(self.mixer.forward(h, ctx, cache, (), None), 1.0)]
        after = ctx.next_block.opening() if ctx.next_block is not None else (None, None, 0.0)
        if self.ffn is None:
            ops.streams_join(x, y, self.hc1.mix, self.hc1.weight_out, *after, h=h)
            return x
        gamma, _, eps, _ = self.norm2.fusable()
        ops.streams_join(x, y, self.hc1.mix, self.hc1.weight_out, self.hc2.weight_in, gamma, eps, h=h)
        y = self.ffn.forward(h, ctx, (), None)
        ops.streams_join(x, [(y, 1.0)], self.hc2.mix, self.hc2.weight_out, *after, h=h)
        return x


class StreamWeights(Part):
    """How a sublayer reads n streams ("in" [n]), where they go behind it ("mix" [n, n], a row a stream) and how much of its
    result each takes ("out" [n])."""
    capturable = True
    launches_only = True

    def __init__(self, streams: int):
        self.n = streams
        self.weight_in = self.weight_out = self.mix = None

    def parameters(self) -> Dict[str, ParamSpec]:
        n = self.n
        return {"in": ParamSpec((n,), "vector", "share"), "out": ParamSpec((n,), "vector", "gamma"),
                "mix": ParamSpec((n, n), "vector", "near_identity")}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight_in, self.weight_out, self.mix = tensors["in"], tensors["out"], tensors["mix"]


register_block("parallel", ParallelBlock)
register_block("parallel_two_norms", TwoNormParallelBlock)
register_block("sequential", SequentialBlock)
register_block("post_norm", PostNormBlock)
register_block("streams", StreamsBlock)
