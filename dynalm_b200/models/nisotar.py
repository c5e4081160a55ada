"""The Nisotar architecture: config.json -> NisotarConfig -> ModelPlan.

A pre-norm decoder with layer norms without bias ("pre_norm", parts/block.py). The mixer of a layer is windowed attention
(parts/attention.py, kind "gated_attention": queries and keys normed head by head with one weight, then turned, YaRN
frequencies where the layer has them, one more term of score 0 in the softmax's denominator), latent attention with a window
and an ordinary softmax (parts/latent_attention.py), or two mixers side by side (parts/side_by_side.py): attention inside
chunks of the sequence whose values are its keys as projected, beside a gated delta rule with a decay per key channel whose
decay and output gate come from two-step projections (parts/delta_rule.py); the two results are normed, each with a weight
of its own, and half their sum is the pair's. The feed-forward is a gated one with biases whose halves are clamped
(parts/mlp.py), a mixture of gated experts chosen by biased logits (parts/moe.py), or absent. The head has a matrix of its
own.
Tensor names: `embed`, `l<i>.norm{1,2}`, `l<i>.mix.{q,k,v,o}` with `.q.norm` and `.k.norm`,
`l<i>.mix.{q,dkv,dkv.norm,uk,uv,o}`, `l<i>.mix.left.{q,k,o,q.norm,k.norm,out}` with
`l<i>.mix.right.{q,k,v,b,a1,a2,A_log,dt_bias,g1,g2,norm,o,out}` (+ `.conv` for q, k and v),
`l<i>.mlp.{gate,up,down}` (+ `.b`), `l<i>.mlp.router` (+ `.b`), `l<i>.mlp.e<j>.{gate,up,down}`, `final.norm`, `head`.
"""

from __future__ import annotations

from typing import Any, Dict, Mapping, Optional, Tuple

from ..config.nisotar import (NisotarAttention, NisotarConfig, NisotarDelta, NisotarDense, NisotarLatent, NisotarPair,
                              NisotarRotation)
from ..config.plan import (BlockSpec, EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerRun, MixerSpec, ModelPlan, NormSpec,
                           PositionSpec)
from ..errors import NotFound
from ..registry import register_architecture

_ATTENTION = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"))
_LATENT = (("q", "q"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"), ("uk", "uk"), ("uv", "uv"), ("o", "o"))
_DELTA = (("q", "q"), ("q_conv", "q.conv"), ("k", "k"), ("k_conv", "k.conv"), ("v", "v"), ("v_conv", "v.conv"), ("b", "b"),
          ("decay_in", "a1"), ("decay_out", "a2"), ("a_log", "A_log"), ("dt_bias", "dt_bias"), ("gate_in", "g1"),
          ("gate_out", "g2"), ("norm", "norm"), ("o", "o"))


def _position(rot: NisotarRotation, size: int) -> Optional[PositionSpec]:
    if rot.dims == 0:
        return None
    return PositionSpec("rotary_halves", head_dim=size, rotary_dim=rot.dims, theta=rot.base,
                        factors=rot.stretch.divisors(rot.base, rot.dims) if rot.stretch is not None else None,
                        magnitude=rot.stretch.magnitude if rot.stretch is not None else 1.0)


def _attention(m: NisotarAttention, eps: float, chunked: bool) -> Dict[str, Any]:
    return dict(num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale,
                window=0 if chunked else m.size, chunk=m.size if chunked else 0, eps=eps, qk_norm="head_first", sink="zero",
                gated=False, values="keys" if chunked else "own", position=_position(m.rot, m.dim))


class NisotarArchitecture:
    name = "Nisotar"
    model_types = ("nisotar",)

    def read_config(self, obj: Mapping[str, Any]) -> NisotarConfig:
        return NisotarConfig.from_dict(obj)

    @staticmethod
    def _ranks(m: NisotarDelta, p: str, present: Optional[Any]) -> Tuple[int, int]:
        ranks = []
        for name, told, key in (("a1", m.decay_rank, "decay_rank"), ("g1", m.gate_rank, "gate_rank")):
            r = int(present[p + name][0]) if isinstance(present, Mapping) and p + name in present else told
            if r <= 0:
                raise NotFound(f"config.json: an inner size of a two-step projection is given neither by a tensor '{p}{name}' "
                               f"nor by '{key}'")
            ranks.append(r)
        return ranks[0], ranks[1]

    def _mixer(self, m, width: int, eps: float, p: str, present: Optional[Any]) -> MixerSpec:
        if isinstance(m, NisotarAttention):
            return MixerSpec("gated_attention", width, {k: p + f for k, f in _ATTENTION}, **_attention(m, eps, chunked=False))
        if isinstance(m, NisotarLatent):
            return MixerSpec("latent_attention", width, {k: p + f for k, f in _LATENT}, num_heads=m.heads, head_dim=m.dim,
                             rot_dim=m.rot_dim, value_dim=m.vdim, q_rank=0, kv_rank=m.kv_rank, scale=m.scale,
                             window=m.window, eps=eps, position=_position(m.rot, m.rot_dim))
        assert isinstance(m, NisotarPair)
        decay_rank, gate_rank = self._ranks(m.right, p + "right.", present)
        left = MixerSpec("gated_attention", width, None, **_attention(m.left, eps, chunked=True))
        r = m.right
        right = MixerSpec("gated_delta", width, None, num_heads=r.heads, num_kv_heads=r.kv_heads, head_dim=r.dim,
                          value_dim=r.vdim, taps=r.taps, eps=eps, decay="channel", decay_rank=decay_rank, gate="sigmoid",
                          gate_rank=gate_rank)
        names = {f"left.{k}": f"{p}left.{f}" for k, f in _ATTENTION if k != "v"}
        names.update({f"right.{k}": f"{p}right.{f}" for k, f in _DELTA})
        names.update(left_norm=p + "left.out", right_norm=p + "right.out")
        return MixerSpec("side_by_side", width, names, left=left, right=right, left_scale=0.5, right_scale=0.5, normed=True,
                         eps=eps)

    def plan(self, cfg: NisotarConfig, present: Optional[Any] = None) -> ModelPlan:
        """`present`: the tensors of the model folder, when known; where it also gives their shapes (a mapping), the inner
        sizes of the delta rule's two-step projections are read from there."""
        W, eps = cfg.width, cfg.norm_eps
        layers, order, ignorable = [], [], []
        for i, layer in enumerate(cfg.layers):
            p = f"l{i}."
            parts: Dict[str, Any] = dict(mixer_norm=NormSpec("layer", W, eps, {"weight": p + "norm1"}),
                                         mixer=self._mixer(layer.mixer, W, eps, p + "mix.", present))
            f = layer.mlp
            if f is None:
                ignorable.append(p + "norm2")          # a layer without a feed-forward may still carry its norm
            else:
                parts["ffn_norm"] = NormSpec("layer", W, eps, {"weight": p + "norm2"})
            if isinstance(f, NisotarDense):
                names = {k: f"{p}mlp.{k}" for k in ("gate", "up", "down")}
                names.update({k + "_bias": f"{p}mlp.{k}.b" for k in ("gate", "up", "down")})
                parts["ffn"] = FeedForwardSpec("gated_mlp", W, names, inner=f.ff, activation="clamped_swiglu", limit=f.limit,
                                               gate_scale=1.702)
            elif f is not None:
                names = {"router": p + "mlp.router", "router_bias": p + "mlp.router.b"}
                for j in range(f.experts):
                    names.update({f"{k}{j}": f"{p}mlp.e{j}.{k}" for k in ("gate", "up", "down")})
                # a softmax over the chosen logits alone is the chosen part of one over all experts, over its sum
                parts["ffn"] = FeedForwardSpec("routed_mlp", W, names, inner=f.ff, experts=f.experts, top=f.top, groups=1,
                                               keep_groups=1, weight_scale=1.0, activation="swiglu", scores="softmax",
                                               renormalize=True, biased=True)
            layers.append(BlockSpec("pre_norm", **parts))
            order.append(LayerRun(i))
        plan = ModelPlan(
            embedding=EmbeddingSpec(cfg.vocab, W, cfg.embedding_scale, {"weight": "embed"}),
            layers=layers, order=order, final_norm=NormSpec("layer", W, eps, {"weight": "final.norm"}),
            head=HeadSpec(cfg.vocab, W, False, 1.0, {"weight": "head"}),
            context_length=cfg.context, ignorable=tuple(ignorable))
        plan.validate()
        return plan


register_architecture(NisotarArchitecture())
