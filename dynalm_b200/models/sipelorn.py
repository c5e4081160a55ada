"""The Sipelorn architecture: config.json -> SipelornConfig -> ModelPlan.

A pre-norm decoder with layer norms (weight and bias) whose sublayers join the stream through a gate, x <- x +
sigmoid(W h + b) * sublayer(h), and whose layers end with a small input that depends on the token alone
("gated_pre_norm", parts/block.py). The mixer of a layer is windowed attention without a rotation (parts/attention.py, kind
"gated_attention": short convolutions over queries, keys and values, a logarithmic distance bias, an output gate; a layer
may read the cache of an earlier one and then makes queries only) or latent attention without a query latent
(parts/latent_attention.py). The feed-forward is dense with xIELU (parts/mlp.py), a mixture of gated experts chosen by
corrected sigmoid scores with a gated shared expert (parts/moe.py), or absent. The embedding adds a row of a table of
token pairs (parts/embedding.py), so the last token is part of a request's state. The head has a matrix of its own.
Tensor names: `embed`, `bigram`, `side.embed`, `l<i>.norm{1,2}` (+ `.b`), `l<i>.rg{1,2}` (+ `.b`),
`l<i>.side.{gate,proj,norm}`, `l<i>.mix.{q,k,v,g,o,r1,r2}` (+ `.b` and `.conv` for q, k and v),
`l<i>.mix.{q,dkv,dkv.norm,uk,uv,o}`, `l<i>.mlp.{up,down,act}`, `l<i>.mlp.{router,correction}`,
`l<i>.mlp.e<j>.{gate,up,down}`, `l<i>.mlp.shared.{gate,up,down,sg}`, `final.norm` (+ `.b`), `head`.
"""

from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

from ..config.plan import (BlockSpec, ConnectionSpec, EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerRun, MixerSpec, ModelPlan,
                           NormSpec, PositionSpec)
from ..config.sipelorn import SipelornAttention, SipelornConfig, SipelornDense, SipelornLatent
from ..registry import register_architecture


def _attention(m: SipelornAttention, width: int, eps: float, p: str, cache_window: int) -> MixerSpec:
    own = m.kv_from is None
    projected = ("q", "k", "v") if own else ("q",)
    names = {k: p + "mix." + k for k in projected + ("o",)}
    names.update({k + "_bias": p + "mix." + k + ".b" for k in projected})
    if m.taps > 0:
        names.update({k + "_conv": p + "mix." + k + ".conv" for k in projected})
    names.update(gate=p + "mix.g", distance_rate=p + "mix.r1", distance_step=p + "mix.r2")
    return MixerSpec("gated_attention", width, names, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                     value_dim=m.vdim, scale=m.scale, window=m.window, cache_window=cache_window, keep_first=0, eps=eps,
                     qk_norm="none", sink="none", gated=True, conv=m.taps, distance_bias="log", own_kv=own, position=None)


def _latent(m: SipelornLatent, width: int, eps: float, p: str) -> MixerSpec:
    position = None
    if m.rot_dims > 0:
        position = PositionSpec("rotary_interleaved", head_dim=m.rot_dim, rotary_dim=m.rot_dims, theta=m.rot_base,
                                factors=m.stretch.divisors(m.rot_base, m.rot_dims) if m.stretch is not None else None,
                                magnitude=m.stretch.magnitude if m.stretch is not None else 1.0)
    names = {"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"}
    return MixerSpec("latent_attention", width, {k: p + "mix." + f for k, f in names.items()}, num_heads=m.heads,
                     head_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim, q_rank=0, kv_rank=m.kv_rank, scale=m.scale,
                     window=0, eps=eps, position=position)


def _feed_forward(f, width: int, p: str) -> FeedForwardSpec:
    if isinstance(f, SipelornDense):
        return FeedForwardSpec("mlp", width, {k: f"{p}mlp.{k}" for k in ("up", "down", "act")}, inner=f.ff, activation="xielu")
    names = {"router": p + "mlp.router", "correction": p + "mlp.correction"}
    for j in range(f.experts):
        names.update({f"{k}{j}": f"{p}mlp.e{j}.{k}" for k in ("gate", "up", "down")})
    if f.shared_ff > 0:
        names.update({"shared_" + k: f"{p}mlp.shared.{k}" for k in ("gate", "up", "down", "sg")})
    return FeedForwardSpec("routed_mlp", width, names, inner=f.ff, experts=f.experts, top=f.top, groups=f.groups,
                           keep_groups=f.keep_groups, weight_scale=1.0, activation="swiglu", scores="sigmoid",
                           group_score="top2", renormalize=False, corrected=True, shared_inner=f.shared_ff)


class SipelornArchitecture:
    name = "Sipelorn"
    model_types = ("sipelorn",)

    def read_config(self, obj: Mapping[str, Any]) -> SipelornConfig:
        return SipelornConfig.from_dict(obj)

    def plan(self, cfg: SipelornConfig, present: Optional[Any] = None) -> ModelPlan:
        W, eps = cfg.width, cfg.norm_eps
        # what a layer's cache must still hold is decided by the widest window of those that read it
        reach = {}
        for i, layer in enumerate(cfg.layers):
            if isinstance(layer.mixer, SipelornAttention):
                j = i if layer.mixer.kv_from is None else layer.mixer.kv_from
                reach.setdefault(j, []).append(layer.mixer.window)
        layers, order, ignorable = [], [], []
        for i, layer in enumerate(cfg.layers):
            p, m = f"l{i}.", layer.mixer
            if isinstance(m, SipelornAttention):
                windows = reach.get(i, [m.window])
                mixer = _attention(m, W, eps, p, 0 if min(windows) == 0 else max(windows))
            else:
                assert isinstance(m, SipelornLatent)
                mixer = _latent(m, W, eps, p)

            def norm(name: str) -> NormSpec:
                return NormSpec("layer", W, eps, {"weight": p + name, "bias": p + name + ".b"})

            def gate(name: str) -> ConnectionSpec:
                return ConnectionSpec("sigmoid_gate", W, {"weight": p + name, "bias": p + name + ".b"})

            parts: Dict[str, Any] = dict(mixer_norm=norm("norm1"), mixer=mixer, mixer_gate=gate("rg1"))
            if layer.mlp is not None:
                parts.update(ffn_norm=norm("norm2"), ffn=_feed_forward(layer.mlp, W, p), ffn_gate=gate("rg2"))
            else:                          # a layer without a feed-forward may still carry its norm and its gate
                ignorable += [f"{p}norm2", f"{p}norm2.b", f"{p}rg2", f"{p}rg2.b"]
            if cfg.side_dim > 0:
                parts["side"] = FeedForwardSpec("token_side", W, {"table": "side.embed", "gate": p + "side.gate",
                                                                  "proj": p + "side.proj", "norm": p + "side.norm"},
                                                index=i, inner=cfg.side_dim, vocab=cfg.vocab, layers=len(cfg.layers), eps=eps,
                                                activation="gelu_tanh")
            layers.append(BlockSpec("gated_pre_norm", **parts))
            order.append(LayerRun(i, m.kv_from if isinstance(m, SipelornAttention) else None))
        pairs = cfg.bigram
        plan = ModelPlan(
            embedding=EmbeddingSpec(cfg.vocab, W, cfg.embedding_scale, {"weight": "embed", "pairs": "bigram"},
                                    pair_rows=pairs.buckets if pairs else 0, pair_previous=pairs.mul_prev if pairs else 0,
                                    pair_current=pairs.mul_cur if pairs else 0),
            layers=layers, order=order,
            final_norm=NormSpec("layer", W, eps, {"weight": "final.norm", "bias": "final.norm.b"}),
            head=HeadSpec(cfg.vocab, W, False, 1.0, {"weight": "head"}),
            context_length=cfg.context, ignorable=tuple(ignorable))
        plan.validate()
        return plan


register_architecture(SipelornArchitecture())
