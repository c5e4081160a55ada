"""Mixture-of-experts feed-forward: the "routed_mlp" kind.

Every token uses `top` of `experts` small feed-forward layers without biases, expert j being down_j(act(up_j x))
(activation "relu2") or down_j(silu(gate_j x) * up_j x) (activation "swiglu"). The router's logits z = W_router x are
float32 (with `biased` plus a number per expert); scores are their softmax over ALL experts, or with scores "sigmoid" the sigmoid of each. Choice scores are the
scores, with `corrected` plus a number per expert. Experts form `groups` equal groups of neighbours, a group's score is its
largest choice score, or with group_score "top2" the sum of its two largest, and only experts of the `keep_groups` best
groups can be chosen; of those the `top` with the largest choice scores are. Their weights are their scores (without the
correction), divided by their sum (+ 1e-20) unless `renormalize` is False, times `weight_scale`, and the result is the
weighted sum of the chosen experts' outputs. With shared_inner > 0 a gated expert of that inner size runs for every token
and is added, times sigmoid(W_sg x), one number a token.

On the device: the router product, `moe_route` (one thread a token), `moe_group` (the step's (token, expert) pairs put
in the order of their experts, with the list of row tiles), the two products over those tiles with the matrix of each
tile's expert (`moe_linear`: the activation sits in the first one's epilogue, the second leaves float32), and
`moe_combine`. Nothing comes back to the host, so the launches depend on the number of rows alone.

Another product over the same input can ride with the router's (`join_input`), whose results are float32 then too.

Parameters: inner, experts, top, groups, keep_groups, weight_scale, activation ("relu2", "swiglu"), scores, group_score,
renormalize, corrected, biased, shared_inner. Tensors: router [experts, width], up<j> [inner, width], down<j> [width, inner], and by
the parameters gate<j> [inner, width], correction [experts], router_bias [experts], shared_gate, shared_up [shared_inner, width], shared_down
[width, shared_inner], shared_sg [1, width].
"""

from __future__ import annotations

from typing import Dict

import torch

from ..errors import Unsupported
from ..kernels import linear, ops
from ..kernels.gemm import linear_partial, linear_swiglu
from .base import TensorDecl, register_feed_forward


@register_feed_forward("routed_mlp")
class RoutedMLP:
    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)
    graph_safe = True      # launches depend on row counts only

    @staticmethod
    def declare(spec) -> Dict[str, TensorDecl]:
        out = {"router": TensorDecl((spec.experts, spec.width))}
        if spec.get("corrected", False):
            out["correction"] = TensorDecl((spec.experts,), role="vector", init="bias")
        if spec.get("biased", False):
            out["router_bias"] = TensorDecl((spec.experts,), role="vector", init="bias")
        shared = int(spec.get("shared_inner", 0))
        if shared > 0:
            out.update(shared_gate=TensorDecl((shared, spec.width)), shared_up=TensorDecl((shared, spec.width)),
                       shared_down=TensorDecl((spec.width, shared)), shared_sg=TensorDecl((1, spec.width)))
        for j in range(spec.experts):
            if spec.get("activation", "relu2") == "swiglu":
                out[f"gate{j}"] = TensorDecl((spec.inner, spec.width))
            out[f"up{j}"] = TensorDecl((spec.inner, spec.width))
            out[f"down{j}"] = TensorDecl((spec.width, spec.inner))
        return out

    def __init__(self, spec, tensors: Dict[str, torch.Tensor], runtime):
        E, top = int(spec.experts), int(spec.top)
        groups, keep = int(spec.get("groups", 1)), int(spec.get("keep_groups", 1))
        activation = spec.get("activation", "relu2")
        if activation not in ("relu2", "swiglu"):
            raise Unsupported(f"routed_mlp: activation '{activation}' has no kernel (relu2 and swiglu do)")
        if E > ops.MOE_MAX_EXPERTS or E % groups or not 0 < keep <= groups or not 0 < top <= keep * (E // groups):
            raise Unsupported(f"routed_mlp: {E} experts in {groups} groups, {keep} kept, {top} a token")
        self.spec = spec
        self.rt = runtime
        self.E, self.top, self.groups, self.keep = E, top, groups, keep
        self.scale = float(spec.get("weight_scale", 1.0))
        self.route = dict(scores=spec.get("scores", "softmax"), group_score=spec.get("group_score", "max"),
                          renormalize=bool(spec.get("renormalize", True)))
        self.correction = tensors.get("correction")
        self.router_bias = tensors.get("router_bias")
        self.shared = int(spec.get("shared_inner", 0))
        # everything that wants float32 results of the layer's input in one product: [router | shared expert's gate | rider],
        # padded to a multiple of 8 rows
        self.w_router = self._padded([tensors["router"]] + ([tensors["shared_sg"]] if self.shared else []))
        self.joined_col = self.joined_cols = 0
        self.act = "pairs" if activation == "swiglu" else "relu2"
        if activation == "swiglu":                           # gate and up rows in turn: [E, 2 * inner, width]
            self.w_up = torch.stack([torch.stack([tensors[f"gate{j}"], tensors[f"up{j}"]], dim=1).reshape(2 * spec.inner, spec.width)
                                     for j in range(E)]).contiguous()
        else:
            self.w_up = torch.stack([tensors[f"up{j}"] for j in range(E)]).contiguous()         # [E, inner, width]
        if self.shared:
            self.w_shared = torch.cat([tensors["shared_gate"], tensors["shared_up"]], dim=0).contiguous()
            self.w_shared_down = tensors["shared_down"]
        self.w_down = torch.stack([tensors[f"down{j}"] for j in range(E)]).contiguous()     # [E, width, inner]

    @staticmethod
    def _padded(mats) -> torch.Tensor:
        w = torch.cat(mats, dim=0)
        pad = -w.shape[0] % 8
        return (torch.cat([w, w.new_zeros(pad, w.shape[1])]) if pad else w).contiguous()

    def join_input(self, w: torch.Tensor) -> bool:
        """Takes the rows of another product over the same input into the router's; `joined` gives its result (float32)."""
        self.joined_col, self.joined_cols = self.w_router.shape[0], w.shape[0]
        self.w_router = self._padded([self.w_router, w])
        return True

    def joined(self, rows: int) -> torch.Tensor:
        return self._logits(rows)[:, self.joined_col:self.joined_col + self.joined_cols]

    def _logits(self, rows: int) -> torch.Tensor:
        return self.rt.buffer("moe_logits", (rows, self.w_router.shape[0]), torch.float32)

    def first_weights(self) -> torch.Tensor:
        return self.w_router

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        s, rt = self.spec, self.rt
        rows = x.shape[0]
        E, top = self.E, self.top
        pairs = rows * top
        logits = self._logits(rows)
        linear(x, self.w_router, logits)                                  # float32 accumulation and result
        ids = rt.buffer("moe_ids", (rows, top), torch.int32)
        weights = rt.buffer("moe_weights", (rows, top), torch.float32)
        ops.moe_route(logits[:, :E], top, self.groups, self.keep, self.scale, ids, weights, self.correction, bias=self.router_bias, **self.route)
        most = rt.max_tokens * top
        place_of = rt.flat(f"moe_place_of_{top}", most, torch.int32)
        pair_at = rt.flat(f"moe_pair_at_{top}", most, torch.int32)
        tiles = rt.flat(f"moe_tiles_{top}_{E}", 3 * ops.moe_max_tiles(most, E), torch.int32)
        n_tiles = rt.flat("moe_n_tiles", 1, torch.int32)
        tile_rows = ops.moe_tile_rows(pairs, E, x, (s.width, s.inner))
        ops.moe_group(ids, pairs, E, place_of, pair_at, tiles, n_tiles, tile_rows)
        max_tiles = ops.moe_max_tiles(pairs, E, tile_rows)
        act = rt.flat(f"moe_act_{top}_{s.inner}", most * s.inner, x.dtype)[:pairs * s.inner].view(pairs, s.inner)
        per_pair = rt.flat(f"moe_out_{top}_{s.width}", most * s.width, torch.float32)[:pairs * s.width].view(pairs, s.width)
        if tile_rows == ops.MOE_WIDE_TILE_ROWS and ops.moe_linear_tcgen05_applies(x, self.w_up, act, self.act) \
                and ops.moe_linear_tcgen05_applies(act, self.w_down, per_pair):
            # a long step: the rows once in the order of their experts, then both products on the tcgen05 tensor cores
            sorted_rows = rt.flat(f"moe_rows_{top}_{s.width}", most * s.width, x.dtype)[:pairs * s.width].view(pairs, s.width)
            ops.moe_gather(x, pair_at, top, sorted_rows)
            ops.moe_linear_tcgen05(sorted_rows, self.w_up, act, tiles, n_tiles, max_tiles, self.act)
            ops.moe_linear_tcgen05(act, self.w_down, per_pair, tiles, n_tiles, max_tiles, "none")
        else:
            ops.moe_linear(x, pair_at, top, self.w_up, act, tiles, n_tiles, max_tiles, self.act, tile_rows)
            ops.moe_linear(act, None, 1, self.w_down, per_pair, tiles, n_tiles, max_tiles, "none", tile_rows)
        y = rt.buffer("ffn_out", (rows, s.width))
        shared = shared_z = None
        if self.shared:
            act = linear_swiglu(x, self.w_shared, rt, self.shared)
            shared, shared_z = linear_partial(act, self.w_shared_down, rt, "shared_out"), logits[:, E:E + 1]
        ops.moe_combine(per_pair, place_of, weights, top, y, shared, shared_z)
        return y
