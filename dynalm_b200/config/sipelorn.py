"""The Sipelorn configuration: config.json -> SipelornConfig.

A Sipelorn config.json lists its layers one by one. A layer's mixer is windowed attention without a rotation (short
convolutions over queries, keys and values, a distance bias on the scores, an output gate; it may read the keys and values
of an earlier layer) or latent attention with stretched rotary positions; its feed-forward is dense, a mixture of experts
with a shared expert, or absent:

    {"architecture": "Sipelorn", "vocab": V, "width": W, "norm": {"eps": e},
     "embedding": {"scale": s, "bigram": {"buckets", "mul_prev", "mul_cur"}}, "token_side": {"dim": n},
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "conv", "mask": {"size"},
                                                 "kv_from": j},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups": {"count", "keep"}},
                         "shared": {"ff"}}},
                {"type": "latent_attention", "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
                                                        "rot": {"base", "dims", "scaling": {"factor", "original", "fast",
                                                                                            "slow"}}},
                 "mlp": {"kind": "dense", "ff"} or null}]}

Where a key may be left out its mechanism is switched off (no bigram table without `bigram`, no per-layer token input
without `token_side`, no window without `mask`, no convolutions without `conv`, no stretching without `scaling`, no groups
of experts without `groups`, no shared expert without `shared`); no default stands for a model's value.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import InvalidArgument, NotFound, Unsupported
from .reader import KeyReader
from .yarn import YarnStretch

DEFAULT_CONTEXT = 131072      # the design has no positional limit; block tables are sized for this unless told otherwise


@dataclass(frozen=True)
class SipelornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    taps: int                    # of the short convolutions over q, k and v; 0: none
    window: int                  # 0: all earlier keys
    kv_from: Optional[int]       # the layer whose keys and values are read instead of own ones


@dataclass(frozen=True)
class SipelornLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int                # 0: no rotation
    rot_base: float
    stretch: Optional[YarnStretch]


@dataclass(frozen=True)
class SipelornDense:
    ff: int


@dataclass(frozen=True)
class SipelornMoE:
    ff: int
    experts: int
    top: int
    groups: int                  # 1: no groups
    keep_groups: int
    shared_ff: int               # 0: no shared expert


@dataclass(frozen=True)
class SipelornLayer:
    type: str
    mixer: Union[SipelornAttention, SipelornLatent]
    mlp: Optional[Union[SipelornDense, SipelornMoE]]


@dataclass(frozen=True)
class SipelornBigram:
    buckets: int
    mul_prev: int
    mul_cur: int


def _positive(where: str, **sizes) -> None:
    for name, value in sizes.items():
        if not value > 0:
            raise InvalidArgument(f"{where}: '{name}' must be positive")


def _read_attention(mr: KeyReader) -> SipelornAttention:
    heads, dim = mr.int("heads"), mr.int("dim")
    mask = mr.object_or_none("mask")
    m = SipelornAttention(heads, mr.int_or("kv_heads", heads), dim, mr.int_or("vdim", dim), mr.float_or("scale", dim ** -0.5),
                          mr.int_or("conv", 0), mask.int("size") if mask is not None else 0,
                          mr.int("kv_from") if mr.has("kv_from") else None)
    _positive(mr.where, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim)
    if mask is not None:
        _positive(mask.where, size=m.window)
    if m.heads % m.kv_heads:
        raise InvalidArgument(f"{mr.where}: {m.heads} heads do not divide into {m.kv_heads} key/value heads")
    if m.taps < 0:
        raise InvalidArgument(f"{mr.where}: 'conv' must not be negative")
    return m


def _read_latent(mr: KeyReader) -> SipelornLatent:
    dim, rot_dim = mr.int("dim"), mr.int_or("rot_dim", 0)
    rot = mr.object_or_none("rot")
    stretch, dims, base = None, 0, 10000.0
    if rot is not None:
        dims, base = rot.int_or("dims", rot_dim), rot.float_or("base", 10000.0)
        sc = rot.object_or_none("scaling")
        if sc is not None:
            stretch = YarnStretch.read(sc, base)
    m = SipelornLatent(mr.int("heads"), dim, rot_dim, mr.int_or("vdim", dim), mr.int("kv_rank"),
                       mr.float_or("scale", (dim + rot_dim) ** -0.5), dims, base, stretch)
    _positive(mr.where, heads=m.heads, dim=m.dim, vdim=m.vdim, kv_rank=m.kv_rank, rot_base=m.rot_base)
    if m.rot_dim < 0 or m.rot_dims < 0 or m.rot_dims > m.rot_dim or m.rot_dims % 2:
        raise InvalidArgument(f"{mr.where}: rot.dims {m.rot_dims} must be even and at most rot_dim {m.rot_dim}")
    return m


def _read_mlp(pr: KeyReader) -> Union[SipelornDense, SipelornMoE]:
    kind = pr.str_or("kind", None)
    if kind == "dense":
        f = SipelornDense(pr.int("ff"))
        _positive(pr.where, ff=f.ff)
        return f
    if kind != "moe":
        raise Unsupported(f"{pr.where}: a feed-forward of kind '{kind}'; this design has 'dense' and 'moe'")
    expert, router = pr.object_or_none("expert"), pr.object_or_none("router")
    if expert is None or router is None:
        raise NotFound(f"{pr.where}: needs 'expert' and 'router'")
    groups, shared = router.object_or_none("groups"), pr.object_or_none("shared")
    m = SipelornMoE(expert.int("ff"), router.int("experts"), router.int("top"),
                    groups.int_or("count", 1) if groups is not None else 1,
                    groups.int_or("keep", 1) if groups is not None else 1, shared.int("ff") if shared is not None else 0)
    _positive(pr.where, ff=m.ff, experts=m.experts, top=m.top, groups=m.groups, keep=m.keep_groups)
    if shared is not None:
        _positive(shared.where, ff=m.shared_ff)
    if m.experts % m.groups:
        raise InvalidArgument(f"{pr.where}: {m.experts} experts do not divide into {m.groups} groups")
    if m.keep_groups > m.groups:
        raise InvalidArgument(f"{pr.where}: keeps {m.keep_groups} of {m.groups} groups")
    if m.top > m.keep_groups * (m.experts // m.groups):
        raise InvalidArgument(f"{pr.where}: {m.top} experts a token cannot come from {m.keep_groups} groups of "
                              f"{m.experts // m.groups}")
    return m


@dataclass(frozen=True)
class SipelornConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Optional[SipelornBigram]
    side_dim: int                # size of the per-layer token input; 0: none
    layers: Tuple[SipelornLayer, ...]
    context: int = DEFAULT_CONTEXT

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def max_position_embeddings(self) -> int:
        return self.context

    @classmethod
    def from_dict(cls, obj: Mapping[str, Any]) -> "SipelornConfig":
        top = KeyReader(obj)
        vocab, width = top.int("vocab"), top.int("width")
        _positive("config.json", vocab=vocab, width=width)
        norm, emb, side = top.object_or_none("norm"), top.object_or_none("embedding"), top.object_or_none("token_side")
        bigram = emb.object_or_none("bigram") if emb is not None else None
        pairs = None
        if bigram is not None:
            pairs = SipelornBigram(bigram.int("buckets"), bigram.int("mul_prev"), bigram.int("mul_cur"))
            _positive(bigram.where, buckets=pairs.buckets)
            if pairs.mul_prev < 0 or pairs.mul_cur < 0 or (pairs.mul_prev + pairs.mul_cur) * vocab >= 1 << 62:
                raise InvalidArgument(f"{bigram.where}: the multipliers must not be negative nor overflow 64 bits")
        side_dim = side.int("dim") if side is not None else 0
        if side is not None:
            _positive(side.where, dim=side_dim)
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise NotFound("config.json: missing 'layers' (a list with one entry per layer)")
        layers: list = []
        for i, raw in enumerate(raw_layers):
            lr = KeyReader(raw, f"config.json: layers[{i}]")
            kind = lr.str_or("type", None)
            mr = lr.object_or_none("mixer")
            if mr is None:
                raise NotFound(f"config.json: layers[{i}] has no 'mixer'")
            if kind == "attention":
                mixer = _read_attention(mr)
                j = mixer.kv_from
                if j is not None:
                    source = layers[j].mixer if 0 <= j < i else None
                    if not isinstance(source, SipelornAttention) or source.kv_from is not None:
                        raise InvalidArgument(f"{mr.where}: kv_from {j} names no earlier attention layer with keys of its own")
                    if (source.kv_heads, source.dim, source.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                        raise InvalidArgument(f"{mr.where}: the keys and values of layer {j} have other sizes")
            elif kind == "latent_attention":
                mixer = _read_latent(mr)
            else:
                raise Unsupported(f"config.json: layers[{i}] has a mixer of type '{kind}'; this design has 'attention' and "
                                  f"'latent_attention'")
            pr = lr.object_or_none("mlp")
            layers.append(SipelornLayer(kind, mixer, _read_mlp(pr) if pr is not None else None))
        return cls(vocab, width, norm.float_or("eps", 1e-5) if norm is not None else 1e-5,
                   emb.float_or("scale", 1.0) if emb is not None else 1.0, pairs, side_dim, tuple(layers),
                   top.int_or("context", DEFAULT_CONTEXT))
