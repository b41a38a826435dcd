"""A decoder model put together from a ``ModelSpec``: an embedding part, blocks in their run
order, a head part.  It names no architecture and knows no part's kind."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..parts.base import CacheView, ParamSpec, ResidualStream, Runtime, StreamBundle, build_part, join_cache_specs
from ..parts.specs import ModelSpec
from ..weights.loader import WeightSource, check_against, load_report


class DecoderModel:
    """The model of vt-transformer's ``gpu_main`` (v1/models/qwen2-7b/inference_fp16.dag:368-396):
    embed the tokens, run the layers, norm, logits at the wanted rows only.

    ``order`` is data: ``spec.order[n] = RunSpec(block, cache, writes)``.  The cache slots
    that the runs name are declared by ``cache_slots()``: slot id -> the cache spec of the
    block whose run writes it, under the widest window of the runs that read it."""

    def __init__(self, spec: ModelSpec, rt: Runtime):
        self.spec = spec
        self.rt = rt
        self.embedding = build_part("embedding", spec.embedding, spec.embedding.name, rt)
        self.blocks = [build_part("block", b, b.prefix, rt) for b in spec.blocks]
        self.head = build_part("head", spec.head, spec.head.name, rt)
        self.load_info, self.load_warnings = [], []
        self._check_order()

    # ---- structure -----------------------------------------------------------------
    def _check_order(self) -> None:
        slots: Dict[int, object] = {}
        for n, run in enumerate(self.spec.order):
            if not 0 <= run.block < len(self.blocks):
                raise ValueError(f"run {n} names block {run.block}; the model has {len(self.blocks)}")
            need = self.blocks[run.block].cache_spec()
            if need is None:
                continue
            if run.cache is None:
                raise ValueError(f"run {n}: block {run.block} keeps a cache but the run names no slot")
            # a mixer that keeps several things names a spec for each, and the run a slot for each
            needs = tuple(need) if isinstance(need, (tuple, list)) else (need,)
            named = tuple(run.cache) if isinstance(run.cache, (tuple, list)) else (run.cache,)
            if len(needs) != len(named):
                raise ValueError(f"run {n}: block {run.block} keeps {len(needs)} caches but the run names {len(named)} slots")
            for slot, spec in zip(named, needs):
                if run.writes:
                    if slot in slots:
                        raise ValueError(f"run {n}: cache slot {slot} is written by an earlier run already")
                    slots[slot] = spec
                else:
                    if slot not in slots:
                        raise ValueError(f"run {n} reads cache slot {slot} before any run wrote it")
                    try:
                        slots[slot] = join_cache_specs(slots[slot], spec)
                    except ValueError:
                        raise ValueError(f"run {n}: cache slot {slot} has another layout than block {run.block} reads") from None
        need = self.embedding.cache_spec()
        if need is not None:
            slot = self.spec.embedding_cache
            if slot is None or slot in slots:
                raise ValueError(f"the embedding keeps something of a request and needs a cache slot of its own; the model names {slot}")
            slots[slot] = need
        if any(bool(getattr(b, "streams", 0)) != bool(self.spec.streams) or (self.spec.streams and b.streams != self.spec.streams)
               for b in (*self.spec.blocks, self.spec.embedding)):
            raise ValueError(f"every block and the embedding of a model of {self.spec.streams} streams must be made for that many")
        if (self.spec.streams or need is not None) and any(run.add_embedding for run in self.spec.order):
            raise ValueError("adding the embedding's output again is built for one stream and an embedding that keeps nothing")
        self._slots = slots

    def cache_slots(self) -> Dict[int, object]:
        return dict(self._slots)

    def graph_safe(self) -> bool:
        """True if a step of this model may be captured as a CUDA graph and replayed."""
        return all(p.graph_safe for p in (self.embedding, *self.blocks, self.head))

    def param_specs(self) -> Dict[str, ParamSpec]:
        out = dict(self.embedding.param_specs())
        for b in self.blocks:
            out.update(b.param_specs())
        for name, spec in self.head.param_specs().items():
            out.setdefault(name, spec)          # a head tied to the embedding names the same tensor
        return out

    # ---- weights -------------------------------------------------------------------
    def load(self, source: WeightSource) -> None:
        """Checks the source against the parameter table (one error for all differences),
        then hands each part its tensors."""
        aside = check_against(source, self.param_specs(), self.spec.ignored)
        self.rt.notes.clear()
        for part in (self.embedding, *self.blocks, self.head):
            part.load(source.get)
        self.rt.loaded.clear()                  # the parts hold what they share; nothing else needs the table
        self.load_info, self.load_warnings = load_report(source, self.rt.notes, aside)
        self._link_runs()

    def _link_runs(self) -> None:
        """Tells every run's block which matrix the step streams after it: the first product of the block of the
        next run, of the head after the last.  (A block that runs twice keeps what follows its last run.)"""
        runs = self.spec.order
        for n, run in enumerate(runs):
            after = self.blocks[runs[n + 1].block] if n + 1 < len(runs) else self.head
            self.blocks[run.block].link(after.first_product())

    def weight_bytes(self, n_tokens: int = 1) -> int:
        """Bytes of weights a step reads: every block's weights once for each of its runs,
        the head with its norm, and the embedding rows of the step's tokens."""
        n = sum(self.blocks[r.block].weight_bytes() for r in self.spec.order)
        return n + self.head.weight_bytes() + self.embedding.step_bytes(n_tokens)

    # ---- forward -------------------------------------------------------------------
    @staticmethod
    def _view(views: Dict[int, CacheView], slot, writes: bool) -> Optional[CacheView]:
        view = views.get(slot)
        if view is not None and view.writes != writes:
            view = CacheView(**{**view.__dict__, "writes": writes})
        return view

    def forward(self, ctx, views: Dict[int, CacheView]) -> torch.Tensor:
        """Runs the step's tokens and returns float32 logits [wanted rows, vocab].
        ``views[slot]`` is the cache view of a slot for this step."""
        if self.spec.embedding_cache is None:
            x = self.embedding.forward(ctx)
        else:
            x = self.embedding.forward(ctx, self._view(views, self.spec.embedding_cache, True))
        stream = StreamBundle(x, status=ctx.status) if self.spec.streams else ResidualStream(x, status=ctx.status)
        # a run that adds the embedding's output once more reads a second copy of it (the stream itself moves on)
        first = self.embedding.forward(ctx) if any(run.add_embedding for run in self.spec.order) else None
        for run in self.spec.order:
            if run.add_embedding:
                self.rt.ops.add_rows(stream.x, first)
            view = None
            if isinstance(run.cache, (tuple, list)):
                view = tuple(self._view(views, slot, run.writes) for slot in run.cache)
            elif run.cache is not None:
                view = self._view(views, run.cache, run.writes)
            self.blocks[run.block].forward(stream, ctx, view)
        return self.head.forward(stream, ctx)
