"""The two ends of a model: token ids into the residual stream, and the stream's wanted rows into logits."""
from __future__ import annotations

import torch

from .base import Embedding, Head, ParamSpec, StateSpec, build_part, register_part


@register_part("embedding", "table")
class TableEmbedding(Embedding):
    """x[t,:] = scale * table[id[t],:] as a copy of rows into 32-bit (v1/tensortype/host_tensor.cpp:189-198 has no
    scale: ``scale`` is 1 there).  ``prefix`` is the table's tensor name."""

    graph_safe = True

    def param_specs(self):
        return {self.prefix: ParamSpec((self.spec.vocab, self.spec.hidden))}

    def load(self, get) -> None:
        self.table = self.rt.load(get, self.prefix)

    def step_bytes(self, n_tokens: int) -> int:
        return n_tokens * self.spec.hidden * self.table.element_size()

    def forward(self, ctx, cache=None):
        x = torch.empty((ctx.n_tokens, self.spec.hidden), dtype=torch.float32, device=self.rt.device)
        self.rt.ops.embedding(self.table, ctx.token_ids, x, status=ctx.status, scale=self.spec.scale)
        return x


@register_part("embedding", "pair")
class PairEmbedding(Embedding):
    """See ``EmbeddingSpec``: a token's row plus a row of a second table that the pair (token before, token) picks, normed
    where a norm is given, in every stream of the residual; one kernel.  A request keeps its last token (a state slot)."""

    graph_safe = True

    def __init__(self, spec, prefix, rt):
        super().__init__(spec, prefix, rt)
        if spec.pair is None:
            raise ValueError("pair embedding: 'pair' = (buckets, factor of the token before, factor of the token)")
        if spec.scale != 1.0:
            raise ValueError("pair embedding: a scale is not built")
        if spec.norm is not None and (spec.norm.kind != "rmsnorm" or spec.norm.groups != 1):
            raise ValueError("pair embedding: its norm is a root-mean-square norm without groups")
        self.norm = build_part("norm", spec.norm, spec.norm_name, rt) if spec.norm is not None else None

    def cache_spec(self):
        return StateSpec((1,), torch.int32)

    def param_specs(self):
        s = self.spec
        out = {self.prefix: ParamSpec((s.vocab, s.hidden)), s.pair_name: ParamSpec((s.pair[0] + 1, s.hidden))}
        if self.norm is not None:
            out.update(self.norm.param_specs())
        return out

    def load(self, get) -> None:
        self.table, self.second = self.rt.load(get, self.prefix), self.rt.load(get, self.spec.pair_name)
        if self.table.dtype != self.second.dtype:
            self.table, self.second = self.table.float(), self.second.float()
        if self.norm is not None:
            self.norm.load(get)

    def step_bytes(self, n_tokens: int) -> int:
        return 2 * n_tokens * self.spec.hidden * self.table.element_size()

    def forward(self, ctx, cache=None):
        s = self.spec
        x = torch.empty((ctx.n_tokens, max(1, s.streams), s.hidden), dtype=torch.float32, device=self.rt.device)
        weight, eps = (None, 0.0) if self.norm is None else (self.norm.weighted(), s.norm.eps)
        self.rt.ops.embedding_pair(self.table, self.second, ctx, cache.state, x, s.pair[1], s.pair[2], weight=weight, eps=eps,
                                   status=ctx.status)
        return x if s.streams else x.view(ctx.n_tokens, s.hidden)


@register_part("head", "linear")
class LinearHead(Head):
    """Norm of the wanted rows only, then their product with the [vocab, hidden] matrix into float32 logits
    (v1/models/qwen2-7b/inference_fp16.dag:383-384, v1/tensortype/cuda_tensor.cpp:946-992: logits for the selected
    positions only), then the optional scale and soft cap.  ``prefix`` is unused: the names are the spec's."""

    def __init__(self, spec, prefix, rt):
        super().__init__(spec, prefix, rt)
        self.norm = build_part("norm", spec.norm, spec.norm_name, rt)

    @property
    def graph_safe(self):
        return self.norm.graph_safe

    def param_specs(self):
        s = self.spec
        out = {s.name: ParamSpec((s.vocab, s.hidden), optional=s.tied_to is not None)}
        out.update(self.norm.param_specs())
        return out

    def load(self, get) -> None:
        s = self.spec
        self.weight = self.rt.load(get, s.tied_to if s.tied_to is not None else s.name)
        self.norm.load(get)

    def weight_bytes(self) -> int:
        return self.weight.numel() * self.weight.element_size() + self.norm.weight_bytes()

    def first_product(self):
        return self.rt.ops.product_hint(self.weight, "linear")

    def forward(self, stream, ctx):
        s, ops = self.spec, self.rt.ops
        n_want = ctx.want_rows.numel()
        logits = torch.empty((n_want, s.vocab), dtype=torch.float32, device=self.rt.device)
        if n_want == 0:
            return logits
        h = stream.normed(self.norm, rows=ctx.want_rows)
        ops.linear(h, self.weight, None, logits)
        if s.logit_scale != 1.0 or s.logit_cap > 0.0:
            ops.logits_scale_cap(logits, s.logit_scale, s.logit_cap)
        return logits
