"""A decoder model as data plus parts: embedding, the scheduled runs of its
blocks, the final norm and the output head."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..config.specs import ModelSpec
from ..parts.base import ParamSpec, StateRequest, build_block, build_norm


def _tensor_addresses(part, prefix: str) -> Dict[str, int]:
    """name -> address (0 for None) of the tensors an object holds as attributes, in lists, tuples and
    dicts, and inside the parts it holds; names are attribute paths, so equal for equal parts."""
    out: Dict[str, int] = {}

    def walk(v, name, depth):
        if isinstance(v, torch.Tensor):
            out[name] = v.data_ptr()
        elif isinstance(v, (list, tuple)):
            for i, u in enumerate(v):
                walk(u, f"{name}[{i}]", depth)
        elif isinstance(v, dict):
            for k, u in v.items():
                walk(u, f"{name}[{k!r}]", depth)
        elif hasattr(v, "parameters") and hasattr(v, "load") and depth < 8:
            for k, u in sorted(vars(v).items()):
                walk(u, f"{name}.{k}", depth + 1)

    for k, v in sorted(vars(part).items()):
        walk(v, prefix + k, 0)
    return out


class DecoderModel:
    """Built from a ModelSpec alone.  One block per entry of ``spec.layers``;
    ``spec.schedule`` says which block runs when and on which cache entry, so a
    block may run twice or read an entry another run wrote."""

    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.blocks = [build_block(b) for b in spec.layers]
        self.final_norm = build_norm(spec.final_norm)
        self.embedding_norm = build_norm(spec.embedding_norm) if spec.embedding_norm is not None else None
        self.pass_vectors: Optional[torch.Tensor] = None       # one learned vector per pass over a looped range
        self._keeps_embedding = any(e.enter is not None and e.enter.add_embedding for e in spec.schedule)
        self.embedding: Optional[torch.Tensor] = None
        self.pair_embedding: Optional[torch.Tensor] = None     # hashed embedding of (token before, token), if the spec has it
        self.positions: Optional[torch.Tensor] = None          # learned absolute positions, if the spec has them
        self.head_weight: Optional[torch.Tensor] = None
        self.head_bias: Optional[torch.Tensor] = None
        self._ones: Optional[torch.Tensor] = None              # weights of a sum of all streams
        self._held: Dict[int, Dict[str, int]] = {}             # layer -> addresses of its tensors (see run)

    # -- parameters -------------------------------------------------------
    def parameters(self) -> Dict[str, ParamSpec]:
        s = self.spec
        p: Dict[str, ParamSpec] = {"embedding": ParamSpec((s.vocab, s.hidden))}
        for i, b in enumerate(self.blocks):
            for k, v in b.parameters().items():
                p[f"layers/{i}/{k}"] = v
        if s.position_table:
            p["positions"] = ParamSpec((s.position_table, s.hidden))
        if s.pair_embedding is not None:
            p["pair_embedding"] = ParamSpec((s.pair_embedding.buckets + 1, s.hidden))
        for k, v in self.final_norm.parameters().items():
            p[f"final_norm/{k}"] = v
        if self.embedding_norm is not None:
            for k, v in self.embedding_norm.parameters().items():
                p[f"embedding_norm/{k}"] = v
        if s.pass_vectors:
            p["pass_vectors"] = ParamSpec((s.pass_vectors, s.hidden), "vector", "bias")
        if not s.tie_embeddings:
            p["head/weight"] = ParamSpec((s.vocab, s.hidden))
        if s.head_bias:
            # with tied embeddings a file may lack the bias: zeros then
            p["head/bias"] = ParamSpec((s.vocab,), "vector", "bias", optional=s.tie_embeddings)
        return p

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.embedding = tensors["embedding"]
        self.positions = tensors["positions"] if self.spec.position_table else None
        self.pair_embedding = tensors["pair_embedding"] if self.spec.pair_embedding is not None else None
        for i, b in enumerate(self.blocks):
            pre = f"layers/{i}/"
            b.load({k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)})
        self.final_norm.load({k[len("final_norm/"):]: v for k, v in tensors.items()
                              if k.startswith("final_norm/")})
        if self.embedding_norm is not None:
            self.embedding_norm.load({k[len("embedding_norm/"):]: v for k, v in tensors.items()
                                      if k.startswith("embedding_norm/")})
        self.pass_vectors = tensors["pass_vectors"] if self.spec.pass_vectors else None
        self.head_weight = self.embedding if self.spec.tie_embeddings else tensors["head/weight"]
        self.head_bias = tensors.get("head/bias")
        self._ones = torch.ones(self.spec.streams, dtype=torch.float32, device=self.embedding.device) if self.spec.streams else None
        self._held = {}

    @property
    def capturable(self) -> bool:
        """True if a step of this model can be recorded into a CUDA graph."""
        return (self.final_norm.capturable and all(b.capturable for b in self.blocks)
                and (self.embedding_norm is None or self.embedding_norm.capturable))

    def weight_bytes(self) -> int:
        seen, n = set(), 0
        for t in self._all_tensors():
            if t is not None and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                n += t.numel() * t.element_size()
        return n

    def _all_tensors(self):
        yield self.embedding
        yield self.pair_embedding
        yield self.positions
        yield self.head_weight
        yield self.head_bias
        yield self.pass_vectors
        stack = list(self.blocks) + [self.final_norm] + ([self.embedding_norm] if self.embedding_norm is not None else [])
        while stack:
            part = stack.pop()
            for v in vars(part).values():
                if isinstance(v, torch.Tensor):
                    yield v
                elif hasattr(v, "parameters") and hasattr(v, "load"):
                    stack.append(v)

    # -- cache --------------------------------------------------------------
    def cache_requests(self) -> List:
        """What each cache entry must hold: the request of the block whose run writes it."""
        reqs: List = [None] * self.spec.num_cache_entries
        if self.spec.embedding_cache_entry is not None:
            reqs.append(StateRequest((1,)))          # the token before, as the bits of an int32
        for e in self.spec.schedule:
            if e.cache is not None and e.writes:
                reqs[e.cache] = self.blocks[e.layer].cache_request()
        for e in self.spec.schedule:
            if e.cache is not None and not e.writes:
                want, have = self.blocks[e.layer].cache_request(), reqs[e.cache]
                if want != have:
                    raise ValueError(f"layer {e.layer} reads cache entry {e.cache} but needs {want}, "
                                     f"the entry holds {have}")
        return reqs

    # -- compute ------------------------------------------------------------
    def forward(self, ctx, cache) -> torch.Tensor:
        """Run the step described by ctx; float32 logits [len(ctx.want_rows), vocab]."""
        x = self.begin(ctx, cache)
        self.run(x, ctx, cache, 0, len(self.spec.schedule))
        return self.finish(x, ctx)

    # The same step in three pieces, for a caller that captures it as more than one CUDA graph.
    def begin(self, ctx, cache=None) -> torch.Tensor:
        """The residual stream of the step's tokens, float32 [tokens, hidden].  ``cache`` is needed by an
        embedding that keeps something per sequence."""
        pair = self.spec.pair_embedding
        if pair is not None:
            if cache is None:
                raise ValueError("this model's embedding keeps the token before per sequence: begin() needs the cache")
            last = cache.view(self.spec.embedding_cache_entry).rows.view(torch.int32)
            x = ops.embed_pair(self.embedding, self.pair_embedding, ctx, last, pair.mul_prev, pair.mul_cur,
                               self.spec.embedding_scale)
        else:
            x = ops.embed(self.embedding, ctx.tokens, self.spec.embedding_scale, copies=self.spec.streams)
        if self.positions is not None:
            ops.add_rows(self.positions, ctx.tok_pos, x)
        if self.embedding_norm is not None:
            x = self.embedding_norm.forward(x, torch.float32)
        if self._keeps_embedding:
            # later passes over a looped range add the stream as it is now; it is kept with the step's
            # context (a captured step's context lives as long as its graphs)
            ctx.scratch["embedding_output"] = x
            x = x.clone()
        if self.spec.streams and self.spec.schedule:
            # a run's input is read from the streams by what comes before it; one buffer serves all runs
            h = ops.empty((ctx.n_tokens, self.spec.hidden), ctx.act_dtype, x.device)
            ctx.scratch["streams_input"] = ops.streams_read(x, *self.blocks[self.spec.schedule[0].layer].opening(), h=h)
        return x

    def run(self, x, ctx, cache, start: int, stop: int) -> None:
        """Runs start..stop-1 of the schedule, updating x in place.

        The layers of a model are mostly the same block with other tensors, and what the host does
        for one run of a block (the parts' choices, checks, argument records) costs more time than
        the kernels of a short prompt take.  So the launches of a block's run are recorded, compared
        with the launches of the next run of an equal block (they must be the same but for the two
        blocks' own tensors and temporaries), and from the third such run on repeated with that
        run's tensors in place of the recorded ones.  Runs that fork onto a second stream are left
        alone: their events are no launches."""
        repeat = ops.REPEAT_LAYERS and getattr(ctx, "side_stream", None) is None and stop - start > 2
        kinds: List[list] = []            # [block, (writes, view type, how it hands on), tape, pointers, state, tries]
        for i in range(start, stop):
            e = self.spec.schedule[i]
            view = cache.view(e.cache, e.writes) if e.cache is not None else None
            block = self.blocks[e.layer]
            after = None
            if self.spec.streams:                 # a block of several streams reads them for the run behind it
                nxt = self.spec.schedule[i + 1].layer if i + 1 < len(self.spec.schedule) else None
                ctx.next_block = self.blocks[nxt] if nxt is not None else None
                after = None if nxt is None else (nxt == e.layer, ctx.next_block.opening()[2])
            if not getattr(block, "takes_rounded_stream", False) or e.enter is not None:
                ctx.scratch.pop("stream_rounded", None)      # (a rounded copy of the stream a layer left for the next one)
            if e.enter is not None:
                ops.enter_pass(x, ctx.scratch["embedding_output"] if e.enter.add_embedding else None,
                               self.pass_vectors, e.enter.index)
            if not repeat or not getattr(block, "launches_only", False):
                block.forward(x, ctx, view)
                continue
            ptrs = self._pointers(e.layer, view)
            if after is not None:
                opening = ctx.next_block.opening()
                ptrs = dict(ptrs, **{"next/in": opening[0].data_ptr(), "next/gamma": opening[1].data_ptr()})
            how = (e.writes, type(view), after)
            kind = next((k for k in kinds if type(k[0]) is type(block) and k[0].spec == block.spec and k[1] == how), None)
            if kind is not None and kind[4] == "repeat":
                kind[2].repeat(ptrs)
                continue
            if kind is not None and kind[4] == "own":
                block.forward(x, ctx, view)
                continue
            tape = ops.LaunchTape().start()
            try:
                block.forward(x, ctx, view)
            finally:
                tape.stop()
            if kind is None:
                kinds.append([block, how, tape, ptrs, "recorded", 0])
            elif kind[2].same_as(tape, kind[3], ptrs):
                kind[2].bind(kind[3])
                kind[4] = "repeat"
            else:
                # (the first run of a step may do what later ones find done: tables of the step's
                # positions, say; so the later run becomes the one to compare with, a few times)
                kind[2], kind[3], kind[5] = tape, ptrs, kind[5] + 1
                if kind[5] >= 3:
                    kind[4] = "own"

    def _pointers(self, layer: int, view) -> Dict[str, int]:
        """name -> address of every tensor block ``layer`` holds, and of the cache entry it runs on."""
        held = self._held.get(layer)
        if held is None:
            held = self._held[layer] = _tensor_addresses(self.blocks[layer], "")
        if view is None:
            return held
        ptrs = dict(held)
        if isinstance(view, (tuple, list)):            # a mixer made of several keeps several views
            for j, v in enumerate(view):
                ptrs.update(_tensor_addresses(v, f"cache[{j}]/"))
        else:
            ptrs.update(_tensor_addresses(view, "cache/"))
        return ptrs

    def _norm_of_streams(self, x, ctx) -> torch.Tensor:
        """The final norm of the sum of a token's streams, at the wanted places."""
        norm = self.final_norm
        if getattr(norm, "rms", False) and norm.fusable is not None and not norm.spec.bias:
            gamma, _, eps, _ = norm.fusable()
            h = ops.empty((ctx.n_want, self.spec.hidden), ctx.act_dtype, x.device)
            return ops.streams_read(x, self._ones, gamma, eps, h, rows=ctx.want_rows)
        total = ops.empty((ctx.n_want, self.spec.hidden), torch.float32, x.device)
        return norm.forward(ops.streams_read(x, self._ones, None, 0.0, total, rows=ctx.want_rows), ctx.act_dtype)

    def finish(self, x, ctx) -> torch.Tensor:
        s = self.spec
        if ctx.n_want == 0:
            return torch.empty((0, s.vocab), dtype=torch.float32, device=x.device)
        if s.streams:
            xn = self._norm_of_streams(x, ctx)
        else:
            xn = self.final_norm.forward(x, ctx.act_dtype, rows=ctx.want_rows)
        logits = ops.linear(xn, self.head_weight, self.head_bias, out_dtype=torch.float32)
        if s.logit_scale != 1.0 or s.logit_softcap > 0.0:
            ops.scale_softcap(logits, s.logit_scale, s.logit_softcap)
        return logits
