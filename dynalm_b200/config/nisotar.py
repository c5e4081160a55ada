"""The Nisotar configuration: config.json -> NisotarConfig.

A Nisotar config.json lists its layers one by one. A layer's mixer is windowed attention ("attention"), latent attention
with a window ("latent_attention"), or two mixers side by side that read the same input ("parallel": attention inside
chunks whose values are its keys on the left, a gated delta rule with a decay per key channel on the right); its
feed-forward is a dense gated one with clamped halves, a mixture of experts, or absent:

    {"architecture": "Nisotar", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                                                 "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}},
                {"type": "latent_attention", "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask": {"size"},
                                                        "rot": {"base", "dims"}},
                 "mlp": {"kind": "dense", "ff", "limit"} or null},
                {"type": "parallel", "mixer": {"left": {the keys of attention}, "right": {"heads", "kv_heads", "dim", "vdim",
                                                                                           "conv"}}, ...}]}

Where a key may be left out its mechanism is switched off (no window or chunks without `mask`, no rotation without `rot`,
no stretching without `scaling`); no default stands for a model's value. The inner sizes of the delta rule's two-step
projections are read from the model's tensors; a configuration without tensors (random weights) gives them as `decay_rank`
and `gate_rank` beside the delta rule's other sizes.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import InvalidArgument, NotFound, Unsupported
from .reader import KeyReader
from .yarn import YarnStretch

DEFAULT_CONTEXT = 131072      # the design has no positional limit; block tables are sized for this unless told otherwise


@dataclass(frozen=True)
class NisotarRotation:
    dims: int                    # how many of a vector's first numbers are turned (0: none)
    base: float
    stretch: Optional[YarnStretch]


@dataclass(frozen=True)
class NisotarAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    size: int                    # of the window, or of the chunks for the left side of a pair; 0: all earlier keys
    rot: NisotarRotation


@dataclass(frozen=True)
class NisotarLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int                  # 0: all earlier keys
    rot: NisotarRotation


@dataclass(frozen=True)
class NisotarDelta:
    heads: int                   # value heads, each with a matrix state dim x vdim
    kv_heads: int                # query/key heads, each shared by heads / kv_heads value heads
    dim: int
    vdim: int
    taps: int                    # of the short convolutions
    decay_rank: int              # inner sizes of the two-step projections; 0: told by the tensors
    gate_rank: int


@dataclass(frozen=True)
class NisotarPair:
    left: NisotarAttention       # inside chunks; its values are its keys before norm and rotation
    right: NisotarDelta


@dataclass(frozen=True)
class NisotarDense:
    ff: int
    limit: float


@dataclass(frozen=True)
class NisotarMoE:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class NisotarLayer:
    type: str
    mixer: Union[NisotarAttention, NisotarLatent, NisotarPair]
    mlp: Optional[Union[NisotarDense, NisotarMoE]]


def _positive(where: str, **sizes) -> None:
    for name, value in sizes.items():
        if not value > 0:
            raise InvalidArgument(f"{where}: '{name}' must be positive")


def _divide(where: str, heads: int, kv_heads: int) -> None:
    if heads % kv_heads:
        raise InvalidArgument(f"{where}: {heads} heads do not divide into {kv_heads} key/value heads")


def _read_rotation(mr: KeyReader, size: int, room: str) -> NisotarRotation:
    """`size`: how many numbers there are to turn, the value of the key named `room`."""
    rot = mr.object_or_none("rot")
    if rot is None:
        return NisotarRotation(0, 10000.0, None)
    dims, base = rot.int_or("dims", size), rot.float_or("base", 10000.0)
    _positive(rot.where, base=base)
    if dims < 0 or dims > size or dims % 2:
        raise InvalidArgument(f"{rot.where}: 'dims' {dims} must be even and at most {room} {size}")
    sc = rot.object_or_none("scaling")
    return NisotarRotation(dims, base, YarnStretch.read(sc, base) if sc is not None else None)


def _read_mask(mr: KeyReader) -> int:
    mask = mr.object_or_none("mask")
    if mask is None:
        return 0
    size = mask.int("size")
    _positive(mask.where, size=size)
    return size


def _read_attention(mr: KeyReader, values_are_keys: bool) -> NisotarAttention:
    heads, dim = mr.int("heads"), mr.int("dim")
    m = NisotarAttention(heads, mr.int_or("kv_heads", heads), dim, mr.int_or("vdim", dim), mr.float_or("scale", dim ** -0.5),
                         _read_mask(mr), _read_rotation(mr, dim, "dim"))
    _positive(mr.where, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale)
    _divide(mr.where, m.heads, m.kv_heads)
    if values_are_keys and m.vdim != m.dim:
        raise InvalidArgument(f"{mr.where}: values that are the keys have 'vdim' {m.vdim} = 'dim' {m.dim}")
    return m


def _read_latent(mr: KeyReader) -> NisotarLatent:
    dim, rot_dim = mr.int("dim"), mr.int_or("rot_dim", 0)
    m = NisotarLatent(mr.int("heads"), dim, rot_dim, mr.int_or("vdim", dim), mr.int("kv_rank"),
                      mr.float_or("scale", (dim + rot_dim) ** -0.5), _read_mask(mr), _read_rotation(mr, rot_dim, "rot_dim"))
    _positive(mr.where, heads=m.heads, dim=m.dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale)
    if rot_dim < 0:
        raise InvalidArgument(f"{mr.where}: 'rot_dim' must not be negative")
    return m


def _read_delta(mr: KeyReader) -> NisotarDelta:
    heads, dim = mr.int("heads"), mr.int("dim")
    m = NisotarDelta(heads, mr.int_or("kv_heads", heads), dim, mr.int_or("vdim", dim), mr.int("conv"),
                     mr.int_or("decay_rank", 0), mr.int_or("gate_rank", 0))
    _positive(mr.where, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, conv=m.taps)
    _divide(mr.where, m.heads, m.kv_heads)
    return m


def _read_mlp(pr: KeyReader) -> Union[NisotarDense, NisotarMoE]:
    kind = pr.str_or("kind", None)
    if kind == "dense":
        f = NisotarDense(pr.int("ff"), pr.float_or("limit", 0.0))
        _positive(pr.where, ff=f.ff, limit=f.limit)
        return f
    if kind != "moe":
        raise Unsupported(f"{pr.where}: a feed-forward of kind '{kind}'; this design has 'dense' and 'moe'")
    expert, router = pr.object_or_none("expert"), pr.object_or_none("router")
    if expert is None or router is None:
        raise NotFound(f"{pr.where}: needs 'expert' and 'router'")
    m = NisotarMoE(expert.int("ff"), router.int("experts"), router.int("top"))
    _positive(pr.where, ff=m.ff, experts=m.experts, top=m.top)
    if m.top > m.experts:
        raise InvalidArgument(f"{pr.where}: {m.top} of {m.experts} experts a token")
    return m


@dataclass(frozen=True)
class NisotarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[NisotarLayer, ...]
    context: int = DEFAULT_CONTEXT

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def max_position_embeddings(self) -> int:
        return self.context

    @classmethod
    def from_dict(cls, obj: Mapping[str, Any]) -> "NisotarConfig":
        top = KeyReader(obj)
        vocab, width = top.int("vocab"), top.int("width")
        _positive("config.json", vocab=vocab, width=width)
        norm, emb = top.object_or_none("norm"), top.object_or_none("embedding")
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise NotFound("config.json: missing 'layers' (a list with one entry per layer)")
        layers = []
        for i, raw in enumerate(raw_layers):
            lr = KeyReader(raw, f"config.json: layers[{i}]")
            kind = lr.str_or("type", None)
            mr = lr.object_or_none("mixer")
            if mr is None:
                raise NotFound(f"config.json: layers[{i}] has no 'mixer'")
            if kind == "attention":
                mixer = _read_attention(mr, values_are_keys=False)
            elif kind == "latent_attention":
                mixer = _read_latent(mr)
            elif kind == "parallel":
                left, right = mr.object_or_none("left"), mr.object_or_none("right")
                if left is None or right is None:
                    raise NotFound(f"{mr.where}: needs 'left' and 'right'")
                mixer = NisotarPair(_read_attention(left, values_are_keys=True), _read_delta(right))
            else:
                raise Unsupported(f"config.json: layers[{i}] has a mixer of type '{kind}'; this design has 'attention', "
                                  f"'latent_attention' and 'parallel'")
            pr = lr.object_or_none("mlp")
            layers.append(NisotarLayer(kind, mixer, _read_mlp(pr) if pr is not None else None))
        return cls(vocab, width, norm.float_or("eps", 1e-6) if norm is not None else 1e-6,
                   emb.float_or("scale", 1.0) if emb is not None else 1.0, tuple(layers),
                   top.int_or("context", DEFAULT_CONTEXT))
