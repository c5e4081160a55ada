"""The two ends of the model: token embedding and the projection to logits."""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import linear, ops
from .base import CacheSpec, TensorDecl


def declare_embedding(spec) -> Dict[str, TensorDecl]:
    out = {spec.tensors["weight"]: TensorDecl((spec.vocab, spec.width))}
    if getattr(spec, "pair_rows", 0) > 0:
        out[spec.tensors["pairs"]] = TensorDecl((spec.pair_rows + 1, spec.width))
    return out


def declare_head(spec) -> Dict[str, TensorDecl]:
    return {} if spec.tied else {spec.tensors["weight"]: TensorDecl((spec.vocab, spec.width))}


class TokenEmbedding:
    """x[i, :] = table[token_i, :] * scale into the float32 residual stream
    (dynalm/src/model/transformer.cpp:576-577), plus, when the spec has a table of token pairs, the row of it that this
    token and the one in front of it choose (the last row for a sequence's first token). The last token of every request
    is then part of its state: one int32 word per request slot, read and written by the embedding's own kernel, so that
    it is right also where a step's tokens are chosen on the device."""

    def __init__(self, spec, store, runtime):
        self.spec = spec
        self.rt = runtime
        self.table = store[spec.tensors["weight"]]
        self.pairs = store[spec.tensors["pairs"]] if getattr(spec, "pair_rows", 0) > 0 else None
        self.scale = float(spec.scale)

    def cache_spec(self) -> Optional[CacheSpec]:
        return CacheSpec(kind="state", state_shape=(1,), dtype="int32") if self.pairs is not None else None

    def forward(self, ctx, cache=None) -> torch.Tensor:
        rows = ctx.num_tokens
        x = self.rt.buffer("residual", (rows, self.spec.width), torch.float32)
        if self.pairs is None:
            ops.embed(self.table, ctx.token_ids, x, self.scale)
        else:
            ops.embed_pairs(self.table, self.pairs, ctx.token_ids, ctx.positions, ctx.row_request, ctx.row_slot, ctx.q_start,
                            cache.arrays[0], x, self.scale, self.spec.pair_previous, self.spec.pair_current)
        return x


class LogitsHead:
    """logits = normed rows x head^T / divisor * scale, float32 [rows, vocab]
    (dynalm/src/model/transformer.cpp:703-719), then capped by c * tanh(logits / c) when the spec gives a cap (which
    keeps their order, so the most likely token may still be chosen inside the product). `tied` uses the embedding
    table."""

    def __init__(self, spec, store, runtime, embedding: TokenEmbedding):
        self.spec = spec
        self.rt = runtime
        self.weight = embedding.table if spec.tied else store[spec.tensors["weight"]]
        self.out_scale = 1.0 / float(spec.logit_divisor) if spec.logit_divisor != 1.0 else 1.0
        self.out_scale *= float(getattr(spec, "logit_scale", 1.0))
        self.softcap = float(getattr(spec, "softcap", 0.0))

    def forward(self, normed_rows: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        linear(normed_rows, self.weight, out, None, self.out_scale)
        if self.softcap > 0.0:
            ops.softcap(out, self.softcap)         # c * tanh(logits / c), in place on the float32 logits
        return out

    def choose(self, normed_rows: torch.Tensor, ids: torch.Tensor, status_to=None) -> bool:
        """ids[r] = the most likely token of row r (the lowest id among equals) without the logits being written, when
        the product's kernel can do that in its epilogue; False when it cannot (the caller then takes the logits)."""
        if not ops.gemm_argmax_applies(normed_rows, self.weight) or self.out_scale <= 0:
            return False
        rows = normed_rows.shape[0]
        scratch = self.rt.flat("head_argmax_parts", 2 * 8 * -(-self.spec.vocab // 16))
        ops.gemm_argmax(normed_rows, self.weight, ids, scratch, self.out_scale, status_to)
        return True
