"""Configuration of the Gedulorn decoder ("Gedulorn").

Its config.json is nested: ``layers`` lists the layers one by one, each with the ``type`` of its mixer ("attention": grouped-query
softmax attention under a window whose values are its keys' projections; "latent_attention": softmax attention under a window
over a narrow latent a token, which may be another layer's, with a sink a head; "mamba2": a state-space recurrence behind a short
convolution), the mixer's sizes and constants under ``mixer``, and its feed-forward under ``mlp`` (a mixture of experts, or null).
Every size and every constant that can differ between two models of the design is read from there.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, KeyReader, ModelConfig, architecture_name


@dataclass(frozen=True)
class GedulornRotation:
    """The first ``dims`` dimensions turn by base^(-2i/dims) / factor a position, pairs (i, i + dims/2)."""
    dims: int
    base: float
    factor: float = 1.0


@dataclass(frozen=True)
class GedulornAttention:
    """``heads`` query heads over ``kv_heads`` heads of keys of ``dim`` (which are the values too); scores times ``scale``, capped
    at ``softcap`` (None: not); ``window``: how many tokens a token sees, itself included (None: all)."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: Optional[float]
    rot: GedulornRotation
    window: Optional[int]


@dataclass(frozen=True)
class GedulornLatentAttention:
    """``heads`` heads with ``dim`` plain and ``rot_dim`` rotated query/key dimensions and values of ``vdim``; queries through a
    latent of ``q_rank``, keys and values from a latent of ``kv_rank``: the layer's own or, with ``kv_from``, that layer's."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: GedulornRotation
    window: Optional[int]
    kv_from: Optional[int]


@dataclass(frozen=True)
class GedulornStateSpace:
    """``heads`` heads with a state of ``state`` x ``vdim``, B and C of ``groups`` groups, a convolution of ``conv`` taps, a norm in
    ``norm_groups`` parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class GedulornExperts:
    """``experts`` gated feed-forwards of inner size ``ff`` of which a token uses ``top``; ``shared_ff``: the inner size of the expert
    that every token uses (None: there is none)."""
    experts: int
    top: int
    ff: int
    shared_ff: Optional[int]


@dataclass(frozen=True)
class GedulornLayer:
    type: str
    mixer: Any                          # GedulornAttention, GedulornLatentAttention or GedulornStateSpace
    mlp: Optional[GedulornExperts]


@dataclass(frozen=True)
class GedulornConfig(ModelConfig):
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: Tuple[GedulornLayer, ...]

    # ---- reading -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, data: Dict[str, Any], where: str = "config.json") -> "GedulornConfig":
        r = KeyReader(data, where)
        arch = architecture_name(data, where)
        layers_raw = r.raw("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: key 'layers' must be a list with one entry for each layer")
        layers = tuple(_layer(entry, f"{where}: layers[{i}]") for i, entry in enumerate(layers_raw))
        norm = _reader(r.raw("norm"), f"{where}: norm")
        embedding = _reader(r.raw("embedding", default={}), f"{where}: embedding")
        cfg = cls(architecture=arch, vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                  embedding_scale=embedding.number("scale", default=1.0), norm_eps=norm.number("eps", positive=True), layers=layers)
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config.json") -> None:
        if self.width % 8:
            raise ConfigError(f"{where}: 'width' {self.width} is not supported: the matrix kernels read rows in "
                              f"16-byte pieces, so it must be a multiple of 8")
        for i, layer in enumerate(self.layers):
            at = f"{where}: layers[{i}]"
            m, f = layer.mixer, layer.mlp
            if isinstance(m, GedulornAttention):
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: 'heads' {m.heads} is not a multiple of 'kv_heads' {m.kv_heads}")
                if m.rot.dims % 2 or m.rot.dims > m.dim:
                    raise ConfigError(f"{at}: 'rot.dims' {m.rot.dims} must be even and at most 'dim' {m.dim}")
                if m.dim > 256:
                    raise ConfigError(f"{at}: 'dim' above 256 is not supported by the attention kernel")
            elif isinstance(m, GedulornLatentAttention):
                if m.rot.dims % 2 or m.rot.dims > m.rot_dim:
                    raise ConfigError(f"{at}: 'rot.dims' {m.rot.dims} must be even and at most 'rot_dim' {m.rot_dim}")
                if m.kv_rank + m.rot_dim > 2048 or m.kv_rank > 1024:
                    raise ConfigError(f"{at}: 'kv_rank' above 1024 (or with 'rot_dim' above 2048) is not supported by the "
                                      f"attention kernel")
                if max(m.dim, m.kv_rank) > 1536:
                    raise ConfigError(f"{at}: 'dim' above 1536 is not supported by the heads' products")
                if m.kv_from is not None:
                    j = m.kv_from
                    owner = self.layers[j].mixer if 0 <= j < i else None
                    if not isinstance(owner, GedulornLatentAttention) or owner.kv_from is not None:
                        raise ConfigError(f"{at}: 'kv_from' {j} must name an earlier latent_attention layer with a latent of its own")
                    if (owner.kv_rank, owner.rot_dim, owner.rot) != (m.kv_rank, m.rot_dim, m.rot):
                        raise ConfigError(f"{at}: 'kv_rank', 'rot_dim' and 'rot' must equal those of layer {j}, whose latent it reads")
            else:
                if m.heads % m.groups:
                    raise ConfigError(f"{at}: 'heads' {m.heads} is not a multiple of 'groups' {m.groups}")
                if (m.heads * m.vdim) % m.norm_groups:
                    raise ConfigError(f"{at}: 'heads' * 'vdim' {m.heads * m.vdim} is not a multiple of 'norm_groups' {m.norm_groups}")
                if m.conv > 16:
                    raise ConfigError(f"{at}: 'conv' above 16 taps is not supported by the convolution's kernel")
                if m.state > 512:
                    raise ConfigError(f"{at}: 'state' above 512 is not supported by the scan kernel")
            if f is not None:
                if not 1 <= f.top <= f.experts:
                    raise ConfigError(f"{at}: router 'top' {f.top} must lie between 1 and 'experts' {f.experts}")
                if f.experts > 1024:
                    raise ConfigError(f"{at}: more than 1024 experts are not supported by the routing kernel")

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
                "norm": {"eps": self.norm_eps}, "layers": [_layer_dict(layer) for layer in self.layers]}


def _reader(v, where: str) -> KeyReader:
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: expected an object")
    return KeyReader(v, where)


def _rotation(m: KeyReader, where: str, dims: int) -> GedulornRotation:
    raw = m.raw("rot", default=None)
    if raw is None:
        return GedulornRotation(0, 10000.0)
    rot = _reader(raw, where + ".rot")
    scaling = rot.raw("scaling", default=None)
    factor = 1.0 if scaling is None else _reader(scaling, where + ".rot.scaling").number("factor", positive=True)
    return GedulornRotation(rot.integer("dims", default=dims, minimum=0), rot.number("base", positive=True), factor)


def _window(m: KeyReader, where: str) -> Optional[int]:
    raw = m.raw("mask", default=None)
    return None if raw is None else _reader(raw, where + ".mask").integer("size", minimum=1)


def _layer(entry, where: str) -> GedulornLayer:
    r = _reader(entry, where)
    kind = r.string("type")
    mw = f"{where}.mixer"
    m = _reader(r.raw("mixer"), mw)
    heads = m.integer("heads", minimum=1)
    if kind == "attention":
        dim = m.integer("dim", minimum=1)
        if m.integer("vdim", default=dim) != dim:
            raise ConfigError(f"{mw}: 'vdim' must equal 'dim': the values are the keys' projections")
        mixer = GedulornAttention(heads=heads, kv_heads=m.integer("kv_heads", default=heads, minimum=1), dim=dim,
                                  scale=m.number("scale", default=dim ** -0.5), softcap=m.number("softcap", default=None, positive=True),
                                  rot=_rotation(m, mw, dim), window=_window(m, mw))
    elif kind == "latent_attention":
        dim, rot_dim = m.integer("dim", minimum=1), m.integer("rot_dim", minimum=0)
        mixer = GedulornLatentAttention(heads=heads, dim=dim, rot_dim=rot_dim, vdim=m.integer("vdim", default=dim, minimum=1),
                                        q_rank=m.integer("q_rank", minimum=1), kv_rank=m.integer("kv_rank", minimum=1),
                                        scale=m.number("scale", default=(dim + rot_dim) ** -0.5), rot=_rotation(m, mw, rot_dim),
                                        window=_window(m, mw), kv_from=m.integer("kv_from", default=None, minimum=0))
    elif kind == "mamba2":
        mixer = GedulornStateSpace(heads=heads, vdim=m.integer("vdim", minimum=1), state=m.integer("state", minimum=1),
                                   groups=m.integer("groups", default=1, minimum=1), conv=m.integer("conv", minimum=1),
                                   norm_groups=m.integer("norm_groups", default=1, minimum=1))
    else:
        raise ConfigError(f"{where}: layer type '{kind}' is not known; known are 'attention', 'latent_attention' and 'mamba2'")
    mlp_raw = r.raw("mlp", default=None)
    mlp = None
    if mlp_raw is not None:
        fw = f"{where}.mlp"
        f = _reader(mlp_raw, fw)
        ff_kind = f.string("kind")
        if ff_kind != "moe":
            raise ConfigError(f"{fw}: feed-forward kind '{ff_kind}' is not known; known is 'moe'")
        router = _reader(f.raw("router"), fw + ".router")
        shared_raw = f.raw("shared", default=None)
        mlp = GedulornExperts(experts=router.integer("experts", minimum=1), top=router.integer("top", minimum=1),
                              ff=_reader(f.raw("expert"), fw + ".expert").integer("ff", minimum=1),
                              shared_ff=None if shared_raw is None else _reader(shared_raw, fw + ".shared").integer("ff", minimum=1))
    return GedulornLayer(type=kind, mixer=mixer, mlp=mlp)


def _layer_dict(layer: GedulornLayer) -> Dict[str, Any]:
    m, f = layer.mixer, layer.mlp
    if isinstance(m, GedulornStateSpace):
        mixer = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups}
    else:
        rot = {"dims": m.rot.dims, "base": m.rot.base}
        if m.rot.factor != 1.0:
            rot["scaling"] = {"factor": m.rot.factor}
        mixer = {"heads": m.heads, "dim": m.dim, "scale": m.scale, "rot": rot, "mask": None if m.window is None else {"size": m.window}}
        if isinstance(m, GedulornAttention):
            mixer.update(kv_heads=m.kv_heads, vdim=m.dim, softcap=m.softcap)
        else:
            mixer.update(rot_dim=m.rot_dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank)
            if m.kv_from is not None:
                mixer["kv_from"] = m.kv_from
    mlp = None
    if f is not None:
        mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff},
               "shared": None if f.shared_ff is None else {"ff": f.shared_ff}}
    return {"type": layer.type, "mixer": mixer, "mlp": mlp}
