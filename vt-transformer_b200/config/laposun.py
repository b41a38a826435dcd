"""Configuration of the Laposun decoder ("Laposun").

Its config.json is nested: ``layers`` lists the layers one by one, each with the ``type`` of its mixer ("latent_attention":
softmax attention under a window over a narrow latent a token, with one output gate a head), the mixer's sizes and
constants under ``mixer``, and its feed-forward under ``mlp`` (dense, a mixture of experts, or null).  The residual is
``streams`` streams; ``canon.taps`` are the taps of the convolution in front of every sublayer; ``embedding.bigram`` says how a
pair of tokens picks a row of the second embedding table.  Every size and every constant that can differ between two
models of the design is read from there.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, KeyReader, ModelConfig, architecture_name


@dataclass(frozen=True)
class LaposunLatentAttention:
    """``heads`` heads with ``dim`` plain and ``rot_dim`` rotated query/key dimensions and values of ``vdim``; queries
    through a latent of ``q_rank``, keys and values from a latent of ``kv_rank``; the first ``rot_dims`` of the rotated
    dimensions turn by base^(-2i/dims) a position; ``window``: how many tokens a token sees, itself included (None: all)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    window: Optional[int]


@dataclass(frozen=True)
class LaposunDense:
    ff: int


@dataclass(frozen=True)
class LaposunExperts:
    """``experts`` feed-forwards of inner size ``ff`` (square of relu, no gate) of which a token uses ``top``, weighted by
    their softmax scores over the chosen ones' sum, times ``scale``; ``shared_ff``: the inner size of the expert every token
    uses under a gate of its own (None: there is none)."""
    experts: int
    top: int
    scale: float
    ff: int
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LaposunLayer:
    type: str
    mixer: LaposunLatentAttention
    mlp: Any                            # LaposunDense, LaposunExperts or None


@dataclass(frozen=True)
class LaposunConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    taps: int
    buckets: int
    mul_prev: int
    mul_cur: int
    norm_eps: float
    layers: Tuple[LaposunLayer, ...]

    # ---- reading -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, data: Dict[str, Any], where: str = "config.json") -> "LaposunConfig":
        r = KeyReader(data, where)
        arch = architecture_name(data, where)
        layers_raw = r.raw("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: key 'layers' must be a list with one entry for each layer")
        layers = tuple(_layer(entry, f"{where}: layers[{i}]") for i, entry in enumerate(layers_raw))
        norm = _reader(r.raw("norm"), f"{where}: norm")
        canon = _reader(r.raw("canon"), f"{where}: canon")
        bigram = _reader(_reader(r.raw("embedding"), f"{where}: embedding").raw("bigram"), f"{where}: embedding.bigram")
        cfg = cls(architecture=arch, vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                  streams=r.integer("streams", minimum=1), taps=canon.integer("taps", minimum=1),
                  buckets=bigram.integer("buckets", minimum=1), mul_prev=bigram.integer("mul_prev", minimum=0),
                  mul_cur=bigram.integer("mul_cur", minimum=0), norm_eps=norm.number("eps", positive=True), layers=layers)
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config.json") -> None:
        if self.width % 8:
            raise ConfigError(f"{where}: 'width' {self.width} is not supported: the matrix kernels read rows in "
                              f"16-byte pieces, so it must be a multiple of 8")
        if self.width > 12288:
            raise ConfigError(f"{where}: 'width' above 12288 is not supported by the streams' kernel")
        if self.streams > 16:
            raise ConfigError(f"{where}: more than 16 'streams' are not supported by the streams' kernel")
        if self.taps > 16:
            raise ConfigError(f"{where}: canon 'taps' above 16 are not supported by the convolution's kernel")
        if max(self.mul_prev, self.mul_cur) >= 1 << 31:
            raise ConfigError(f"{where}: embedding.bigram 'mul_prev' and 'mul_cur' must lie below 2^31")
        for i, layer in enumerate(self.layers):
            at = f"{where}: layers[{i}]"
            m, f = layer.mixer, layer.mlp
            if m.rot_dims % 2 or m.rot_dims > m.rot_dim:
                raise ConfigError(f"{at}: 'rot.dims' {m.rot_dims} must be even and at most 'rot_dim' {m.rot_dim}")
            if m.kv_rank + m.rot_dim > 2048 or m.kv_rank > 1024:
                raise ConfigError(f"{at}: 'kv_rank' above 1024 (or with 'rot_dim' above 2048) is not supported by the "
                                  f"attention kernel")
            if max(m.dim, m.kv_rank) > 1536:
                raise ConfigError(f"{at}: 'dim' above 1536 is not supported by the heads' products")
            if isinstance(f, LaposunExperts):
                if not 1 <= f.top <= f.experts:
                    raise ConfigError(f"{at}: router 'top' {f.top} must lie between 1 and 'experts' {f.experts}")
                if f.experts > 1024:
                    raise ConfigError(f"{at}: more than 1024 experts are not supported by the routing kernel")

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "canon": {"taps": self.taps}, "norm": {"eps": self.norm_eps},
                "embedding": {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}},
                "layers": [_layer_dict(layer) for layer in self.layers]}


def _reader(v, where: str) -> KeyReader:
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: expected an object")
    return KeyReader(v, where)


def _layer(entry, where: str) -> LaposunLayer:
    r = _reader(entry, where)
    kind = r.string("type")
    if kind != "latent_attention":
        raise ConfigError(f"{where}: layer type '{kind}' is not known; known is 'latent_attention'")
    mw = f"{where}.mixer"
    m = _reader(r.raw("mixer"), mw)
    dim, rot_dim = m.integer("dim", minimum=1), m.integer("rot_dim", minimum=0)
    rot_dims, rot_base = 0, 10000.0
    rot_raw = m.raw("rot", default=None)
    if rot_raw is not None:
        rot = _reader(rot_raw, mw + ".rot")
        rot_dims, rot_base = rot.integer("dims", default=rot_dim, minimum=0), rot.number("base", positive=True)
    window = None
    mask_raw = m.raw("mask", default=None)
    if mask_raw is not None:
        window = _reader(mask_raw, mw + ".mask").integer("size", minimum=1)
    mixer = LaposunLatentAttention(heads=m.integer("heads", minimum=1), dim=dim, rot_dim=rot_dim,
                                   vdim=m.integer("vdim", default=dim, minimum=1), q_rank=m.integer("q_rank", minimum=1),
                                   kv_rank=m.integer("kv_rank", minimum=1), scale=m.number("scale", default=(dim + rot_dim) ** -0.5),
                                   rot_dims=rot_dims, rot_base=rot_base, window=window)
    mlp_raw = r.raw("mlp", default=None)
    mlp = None
    if mlp_raw is not None:
        fw = f"{where}.mlp"
        f = _reader(mlp_raw, fw)
        ff_kind = f.string("kind")
        if ff_kind == "dense":
            mlp = LaposunDense(ff=f.integer("ff", minimum=1))
        elif ff_kind == "moe":
            router = _reader(f.raw("router"), fw + ".router")
            shared_raw = f.raw("shared", default=None)
            mlp = LaposunExperts(experts=router.integer("experts", minimum=1), top=router.integer("top", minimum=1),
                                 scale=router.number("scale", default=1.0), ff=_reader(f.raw("expert"), fw + ".expert").integer("ff", minimum=1),
                                 shared_ff=None if shared_raw is None else _reader(shared_raw, fw + ".shared").integer("ff", minimum=1))
        else:
            raise ConfigError(f"{fw}: feed-forward kind '{ff_kind}' is not known; known are 'dense' and 'moe'")
    return LaposunLayer(type=kind, mixer=mixer, mlp=mlp)


def _layer_dict(layer: LaposunLayer) -> Dict[str, Any]:
    m, f = layer.mixer, layer.mlp
    mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
             "scale": m.scale, "rot": {"dims": m.rot_dims, "base": m.rot_base}, "mask": None if m.window is None else {"size": m.window}}
    mlp = None
    if isinstance(f, LaposunDense):
        mlp = {"kind": "dense", "ff": f.ff}
    elif isinstance(f, LaposunExperts):
        mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top, "scale": f.scale}, "expert": {"ff": f.ff},
               "shared": None if f.shared_ff is None else {"ff": f.shared_ff}}
    return {"type": layer.type, "mixer": mixer, "mlp": mlp}
