"""The generic decoder: built from a ModelSpec, it knows parts and a run order, not an
architecture."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Mapping

import torch

from ..config.spec import ModelSpec
from .base import BuildEnv, CacheNeed, ResidualStream, WeightDecl, build_part, flat_needs
from .block import build_block


@dataclass(frozen=True)
class EntryCache:
    """Which cache a run entry uses: ``owner`` is the run entry whose cache it is (itself,
    unless the entry reads another's), ``need`` what that owner asked for."""

    owner: int
    need: "CacheNeed | tuple | None"  # one need, or a tuple of needs (a mixer made of several)
    # An entry that owns part of what it uses (a state of its own) and reads the rest from another entry: ``need`` is
    # a tuple with None where it has nothing of its own, and the view it gets has the views of entry ``shares`` there.
    shares: int | None = None


class DecoderModel:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device: torch.device | str):
        self.spec = spec
        self.env = BuildEnv(dtype, torch.device(device))
        self.embedding = build_part("embedding", spec.embedding, self.env)
        self.layers = [build_block(layer, self.env) for layer in spec.layers]
        self.prefixes = [layer.prefix for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, self.env)
        self.final_norm_name = spec.final_norm_prefix
        self.head = build_part("head", spec.head, self.env)
        self.transitions = [build_part("transition", t, self.env) for t in spec.transitions]  # tensors by their full names
        self.entry_caches: list[EntryCache] = []
        for i, e in enumerate(spec.run_order):
            block = self.layers[e.layer]
            mixer = block.mixer
            # a block that keeps something of its own beside the mixer's cache (a token shift's state) says so itself
            need = block.cache_need() if hasattr(block, "cache_need") else mixer.cache_need()
            if e.cache_of is None:
                self.entry_caches.append(EntryCache(i, need))
            elif isinstance(need, tuple) and any(n is None for n in need) and flat_needs(need):
                self.entry_caches.append(EntryCache(i, need, shares=self.entry_caches[e.cache_of].owner))
            else:
                if need is not None:
                    raise ValueError(f"run_order[{i}] reads the cache of entry {e.cache_of}, but its mixer "
                                     f"({mixer.spec.kind}) wants a cache of its own")
                owner = self.entry_caches[e.cache_of]
                self.entry_caches.append(EntryCache(owner.owner, owner.need))
        # an embedding that keeps something per request (the token before) comes behind the run entries
        need = self.embedding.cache_need() if hasattr(self.embedding, "cache_need") else None
        self.embedding_entry: int | None = None
        if need is not None:
            self.embedding_entry = len(self.entry_caches)
            self.entry_caches.append(EntryCache(self.embedding_entry, need))
        self.bound = False

    def embed(self, ctx, caches) -> torch.Tensor:
        """The stream's first value, float32 [T, hidden]."""
        if self.embedding_entry is None:
            return self.embedding.forward(ctx)
        return self.embedding.forward(ctx, caches[self.embedding_entry])

    @property
    def shape_static(self) -> bool:
        """Whether every part says that its launches follow from the step's token count alone
        (``Part.shape_static``): then a pass can be captured into CUDA graphs and replayed for
        later steps of the same shape."""

        def ok(part) -> bool:
            subs = list(part.sub_parts().values())
            pos = getattr(part, "position", None)
            if pos is not None:
                subs.append(pos)
            return bool(getattr(part, "shape_static", False)) and all(ok(p) for p in subs)

        return all(ok(p) for p in [self.embedding, self.final_norm, self.head, *self.layers, *self.transitions])

    @property
    def dtype(self) -> torch.dtype:
        return self.env.dtype

    @property
    def device(self) -> torch.device:
        return self.env.device

    # ------------------------------------------------------------------ weights
    def weight_decls(self) -> dict[str, WeightDecl]:
        out = dict(self.embedding.all_weights())
        for prefix, layer in zip(self.prefixes, self.layers):
            out.update(layer.all_weights(prefix))
        out.update(self.final_norm.all_weights(self.final_norm_name))
        out.update(self.head.all_weights())
        for part in self.transitions:
            out.update(part.all_weights())
        return out

    def weight_stacks(self) -> dict[str, tuple[str, ...]]:
        """Tensors that parts want joined (``Part.stacks``), by full name."""
        out: dict[str, tuple[str, ...]] = {}
        for prefix, layer in zip(self.prefixes, self.layers):
            out.update(layer.all_stacks(prefix))
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.embedding.bind_all(tensors)
        for prefix, layer in zip(self.prefixes, self.layers):
            layer.bind_all(tensors, prefix)
        self.final_norm.bind_all(tensors, self.final_norm_name)
        self.head.bind_all(tensors)
        for part in self.transitions:
            part.bind_all(tensors)
        if getattr(self.head, "tied", False):
            self.head.weight = self.embedding.table
        self.bound = True

    def weight_bytes(self) -> int:
        """Bytes of every distinct weight tensor a step reads once (a tied head counts once;
        of the embedding table only the gathered rows are read, so an untied table is left out)."""
        seen, total = set(), 0

        def add(t):
            nonlocal total
            if isinstance(t, torch.Tensor) and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()

        def walk(part):
            for v in vars(part).values():
                if isinstance(v, torch.Tensor) and v.dim() >= 1 and v.is_floating_point():
                    add(v)
            for sub in part.sub_parts().values():
                walk(sub)
            pos = getattr(part, "position", None)
            if pos is not None:
                walk(pos)

        for layer in self.layers:
            walk(layer)
        for part in self.transitions:
            walk(part)
        walk(self.final_norm)
        add(self.head.weight)
        return total

    # ------------------------------------------------------------------ forward
    def forward(self, ctx, caches) -> torch.Tensor:
        """Run the tokens of ``ctx`` through every run entry; ``caches[i]`` is the cache view
        of run entry i (and one more behind them for an embedding with state). Returns float32 logits at ``ctx.logit_rows``: [wanted, vocab]."""
        if not self.bound:
            raise RuntimeError("the model has no weights yet (bind() was not called)")
        # What parts share within one pass is made anew by every pass. That holds for the activation
        # buffers too: a pass that is captured into a CUDA graph must allocate them itself (from the
        # graph's memory pool); tensors left by an earlier pass over the same context are ordinary
        # memory that goes back to the allocator while the graph still holds their addresses.
        ctx.step_cache.clear()
        ctx.buffers.clear()
        stream = ResidualStream(self.embed(ctx, caches))
        for i, entry in enumerate(self.spec.run_order):
            if entry.transition is not None:
                stream = self.transitions[entry.transition].forward(stream, ctx, self.embedding, entry.transition_arg)
            stream = self.layers[entry.layer].forward(stream, ctx, caches[i])
        if stream.links is not None:  # several streams: the head reads their sum
            x = self.final_norm.forward_streams(stream, ctx, None, stream.stream_count, rows=ctx.logit_rows, num_rows=ctx.num_logit_rows, write=False)
            return self.head.forward(x, ctx)
        extra = {"delta_scale": stream.pending_scale} if stream.pending_scale != 1.0 else {}
        if stream.pending_norm is not None:
            extra["delta_norm"] = stream.pending_norm
        x = self.final_norm.forward(stream.total, stream.pending, ctx, rows=ctx.logit_rows,
                                    num_rows=ctx.num_logit_rows, write_residual=False, **extra)
        return self.head.forward(x, ctx)
