"""Laposun as a ``ModelSpec``: a decoder whose residual is several streams that every sublayer reads as one vector and writes
all at once; the embedding is a token's row plus a row picked by the pair of tokens, normed; every sublayer reads its
normed input through a short causal convolution with a skip; the mixers are softmax attention under a window over a
narrow latent a token, with one output gate a head; the feed-forward is a dense gated one or a mixture of experts (square
of relu) with softmax scores and a gated shared expert; the output head is the embedding table.

Tensor names: ``embed``, ``bigram``, ``embed.norm``, ``final.norm``, and for layer i ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.canon1``,
``l<i>.canon2``, ``l<i>.hc1.in|out|mix``, ``l<i>.hc2.in|out|mix``, ``l<i>.mix.*`` and ``l<i>.mlp.*``."""
from __future__ import annotations

from ..config.laposun import LaposunConfig, LaposunDense, LaposunExperts
from ..config.registry import register_architecture
from ..parts.specs import (BlockSpec, EmbeddingSpec, ExpertsSpec, GatedMLPSpec, HeadSpec, LatentAttentionSpec, ModelSpec, NormSpec,
                           PositionSpec, RunSpec)


def _block(cfg: LaposunConfig, i: int, norm: NormSpec) -> BlockSpec:
    layer = cfg.layers[i]
    m, f = layer.mixer, layer.mlp
    position = PositionSpec(kind="rotary_interleaved", dim=m.rot_dims, base=m.rot_base) if m.rot_dims else PositionSpec(kind="none")
    mixer = LatentAttentionSpec(hidden=cfg.width, heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, v_dim=m.vdim, q_rank=m.q_rank,
                                kv_rank=m.kv_rank, scale=m.scale, gate="head", window=m.window, norm_eps=cfg.norm_eps, position=position)
    ffn = None
    if isinstance(f, LaposunDense):
        ffn = GatedMLPSpec(hidden=cfg.width, inter=f.ff, names=("gate", "up", "down"), weight_suffix="")
    elif isinstance(f, LaposunExperts):
        ffn = ExpertsSpec(hidden=cfg.width, experts=f.experts, top=f.top, inter=f.ff, shared_inter=f.shared_ff, activation="relu_square",
                          router_weights="softmax", router_scale=f.scale, shared_gate_name=None if f.shared_ff is None else "shared.sg")
    return BlockSpec(mixer=mixer, ffn=ffn, norm1=norm, norm2=None if ffn is None else norm, prefix=f"l{i}.", mixer_prefix="mix.",
                     ffn_prefix="mlp.", norm1_name="norm1", norm2_name="norm2", kind="streams", streams=cfg.streams, conv_taps=cfg.taps)


def laposun_model_spec(cfg: LaposunConfig) -> ModelSpec:
    norm = NormSpec(size=cfg.width, eps=cfg.norm_eps, kind="rmsnorm", weight_suffix="")
    blocks = tuple(_block(cfg, i, norm) for i in range(len(cfg.layers)))
    # cache slots: the embedding's last token first, then for every layer the rows its convolutions keep (one slot a sublayer;
    # none with one tap) and its attention's pages
    order, slot = [], 1
    for i, b in enumerate(blocks):
        n = 1 + ((1 if b.ffn is None else 2) if cfg.taps > 1 else 0)
        order.append(RunSpec(block=i, cache=slot if n == 1 else tuple(range(slot, slot + n))))
        slot += n
    embedding = EmbeddingSpec(vocab=cfg.vocab, hidden=cfg.width, name="embed", kind="pair", pair=(cfg.buckets, cfg.mul_prev, cfg.mul_cur),
                              pair_name="bigram", norm=norm, norm_name="embed.norm", streams=cfg.streams)
    head = HeadSpec(vocab=cfg.vocab, hidden=cfg.width, norm=norm, norm_name="final.norm", name="head", tied_to="embed")
    return ModelSpec(vocab=cfg.vocab, hidden=cfg.width, blocks=blocks, order=tuple(order), embedding=embedding, head=head, max_positions=0,
                     streams=cfg.streams, embedding_cache=0)


register_architecture("Laposun", LaposunConfig, laposun_model_spec, replace=True)
