"""Gedulorn as a ``ModelSpec``: a decoder whose sublayers read the residual as it is and whose results are normed before they
join it.  The mixers are grouped-query softmax attention under a window (queries and keys normed head by head, values that are the
keys' projections, capped scores), softmax attention under a window over a narrow latent a token with a sink a head, where a
layer may read the latent that an earlier one keeps, and a state-space recurrence behind a short convolution with a gated norm in
groups; the feed-forward is a mixture of gated experts with a bias of the router and a shared expert; the embedding is scaled.

Tensor names: ``embed``, ``final.norm``, ``head``, and for layer i ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` and ``l<i>.mlp.*``."""
from __future__ import annotations

from ..config.gedulorn import GedulornAttention, GedulornConfig, GedulornLatentAttention, GedulornRotation
from ..config.registry import register_architecture
from ..parts.specs import (AttentionSpec, BlockSpec, EmbeddingSpec, ExpertsSpec, HeadSpec, LatentAttentionSpec, ModelSpec, NormSpec,
                           PositionSpec, RunSpec, StateSpaceSpec)


def _position(rot: GedulornRotation) -> PositionSpec:
    if not rot.dims:
        return PositionSpec(kind="none")
    return PositionSpec(kind="rotary_computed", dim=rot.dims, base=rot.base, factor=rot.factor)


def _mixer(cfg: GedulornConfig, m):
    if isinstance(m, GedulornAttention):
        return AttentionSpec(hidden=cfg.width, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, qkv_bias=False, out_bias=False,
                             window=m.window, scale=m.scale, position=_position(m.rot), names=("q", "k", "v", "o"), weight_suffix="",
                             head_norm_eps=cfg.norm_eps, values_from_keys=True, softcap=m.softcap)
    if isinstance(m, GedulornLatentAttention):
        return LatentAttentionSpec(hidden=cfg.width, heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, v_dim=m.vdim, q_rank=m.q_rank,
                                   kv_rank=m.kv_rank, scale=m.scale, sink=True, window=m.window, own_latent=m.kv_from is None,
                                   norm_eps=cfg.norm_eps, position=_position(m.rot))
    return StateSpaceSpec(hidden=cfg.width, heads=m.heads, groups=m.groups, dim=m.state, v_dim=m.vdim, taps=m.conv,
                          norm_groups=m.norm_groups, norm_eps=cfg.norm_eps)


def gedulorn_model_spec(cfg: GedulornConfig) -> ModelSpec:
    norm = NormSpec(size=cfg.width, eps=cfg.norm_eps, kind="rmsnorm", weight_suffix="")
    blocks, order, slots, free = [], [], [], 0
    for i, layer in enumerate(cfg.layers):
        m, f = layer.mixer, layer.mlp
        ffn = None
        if f is not None:
            ffn = ExpertsSpec(hidden=cfg.width, experts=f.experts, top=f.top, inter=f.ff, shared_inter=f.shared_ff, router_bias_name="router.b")
        blocks.append(BlockSpec(mixer=_mixer(cfg, m), ffn=ffn, norm1=norm, norm2=None if ffn is None else norm, prefix=f"l{i}.",
                                mixer_prefix="mix.", ffn_prefix="mlp.", norm1_name="norm1", norm2_name="norm2", kind="outnorm"))
        source = getattr(m, "kv_from", None)
        if source is not None:                       # the pages of the layer whose latent it reads
            slots.append(slots[source])
        else:                                        # pages of its own; a state-space layer: the state and the convolution's inputs
            n = 2 if layer.type == "mamba2" and m.conv > 1 else 1
            slots.append(free if n == 1 else tuple(range(free, free + n)))
            free += n
        order.append(RunSpec(block=i, cache=slots[i], writes=source is None))
    embedding = EmbeddingSpec(vocab=cfg.vocab, hidden=cfg.width, name="embed", scale=cfg.embedding_scale)
    head = HeadSpec(vocab=cfg.vocab, hidden=cfg.width, norm=norm, norm_name="final.norm", name="head")
    return ModelSpec(vocab=cfg.vocab, hidden=cfg.width, blocks=tuple(blocks), order=tuple(order), embedding=embedding, head=head, max_positions=0)


register_architecture("Gedulorn", GedulornConfig, gedulorn_model_spec, replace=True)
