"""Gated feed-forward: down(act(gate x) * up x), the "gated_mlp" kind
(dynalm/src/model/transformer.cpp:671-693), act silu or the tanh form of GELU (parameter `activation`). Gate and up
run as one product against [Wg; Wu]. Its third activation, "clamped_swiglu", clamps both halves: with g = min(gate x, limit)
and u = clamp(up x, -limit, limit), g sigmoid(gate_scale g) (u + 1). The projections' biases are taken when the model has
them, with that activation.
Ungated feed-forward: down(act(up x)), the "mlp" kind, act the squared ReLU, the tanh form of GELU or xIELU.
A small input that depends on the token alone: the "token_side" kind."""

from __future__ import annotations

from typing import Dict

import torch

from ..errors import Unsupported
from ..kernels import ops
from ..kernels import linear
from ..kernels.gemm import (linear_act, linear_clamped_swiglu, linear_geglu, linear_partial, linear_partial_biased, linear_swiglu,
                            linear_xielu)
from .base import TensorDecl, register_feed_forward


@register_feed_forward("gated_mlp")
class GatedMLP:
    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)
    graph_safe = True      # launches depend on row counts (and graph_key) only

    @staticmethod
    def declare(spec) -> Dict[str, TensorDecl]:
        return {
            "gate": TensorDecl((spec.inner, spec.width)),
            "up": TensorDecl((spec.inner, spec.width)),
            "down": TensorDecl((spec.width, spec.inner)),
            "gate_bias": TensorDecl((spec.inner,), role="vector", required=False, init="bias"),
            "up_bias": TensorDecl((spec.inner,), role="vector", required=False, init="bias"),
            "down_bias": TensorDecl((spec.width,), role="vector", required=False, init="bias"),
        }

    def __init__(self, spec, tensors: Dict[str, torch.Tensor], runtime):
        self.activation = spec.get("activation", "silu")
        if self.activation not in ("silu", "gelu_tanh", "clamped_swiglu"):
            raise Unsupported(f"gated_mlp: activation '{self.activation}' has no kernel (silu, gelu_tanh and clamped_swiglu do)")
        biases = [tensors.get("gate_bias"), tensors.get("up_bias")]
        self.b_down = tensors.get("down_bias")
        self.coeffs = None
        if self.activation == "clamped_swiglu":
            # limit, scale and biases lie together in memory, where the products' epilogues read them
            zeros = torch.zeros(spec.inner, dtype=torch.float32, device=runtime.device)
            self.coeffs = ops.clamped_coeffs(float(spec.limit), float(spec.gate_scale),
                                             torch.cat([b if b is not None else zeros for b in biases]), spec.inner, runtime.device)
        elif any(b is not None for b in biases + [self.b_down]):
            raise Unsupported(f"gated_mlp: biases go with clamped_swiglu, not with {self.activation}")
        self.spec = spec
        self.rt = runtime
        self.w_gate_up = torch.cat([tensors["gate"], tensors["up"]], dim=0).contiguous()
        self.w_down = tensors["down"]

    def first_weights(self) -> torch.Tensor:
        """The weights this part streams first (a block may say so to the kernel in front, kernels/ops.stream_ahead)."""
        return self.w_gate_up

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        s, rt = self.spec, self.rt
        if x.shape[0] <= ops.SKINNY_FAST_ROWS:
            ops.stream_ahead(self.w_down)              # taken by the gate | up product, read by the product after it
        if self.activation == "clamped_swiglu":
            act = linear_clamped_swiglu(x, self.w_gate_up, self.coeffs, rt, s.inner)
            return linear_partial_biased(act, self.w_down, self.b_down, rt, "ffn_out")
        if self.activation == "gelu_tanh":
            act = linear_geglu(x, self.w_gate_up, rt, s.inner)
        else:
            act = linear_swiglu(x, self.w_gate_up, rt, s.inner)
        return linear_partial(act, self.w_down, rt, "ffn_out")


@register_feed_forward("mlp")
class DenseMLP:
    """down(act(up x)) without a gate (parameters inner, activation: "relu2" = max(z, 0)^2, "gelu_tanh" =
    0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), "xielu" = softplus(p) z^2 + z / 2 above zero and (1/2 + softplus(q))
    (e^z - 1 - z) + z / 2 at and below it, p and q the two numbers of the tensor `act`)."""

    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)
    graph_safe = True      # launches depend on row counts only

    @staticmethod
    def declare(spec) -> Dict[str, TensorDecl]:
        out = {
            "up": TensorDecl((spec.inner, spec.width)),
            "down": TensorDecl((spec.width, spec.inner)),
        }
        if spec.get("activation", "relu2") == "xielu":
            out["act"] = TensorDecl((2,), role="vector", init="bias")
        return out

    def __init__(self, spec, tensors: Dict[str, torch.Tensor], runtime):
        self.activation = spec.get("activation", "relu2")
        if self.activation not in ("relu2", "gelu_tanh", "xielu"):
            raise Unsupported(f"mlp: activation '{self.activation}' has no kernel (relu2, gelu_tanh and xielu do)")
        self.spec = spec
        self.rt = runtime
        self.w_up = tensors["up"]
        self.w_down = tensors["down"]
        self.coeffs = None
        if self.activation == "xielu":
            # the kernels take the coefficients themselves, from memory (they differ from layer to layer like weights)
            soft = torch.nn.functional.softplus(tensors["act"].double())
            self.coeffs = (soft + torch.tensor([0.0, 0.5], dtype=torch.float64, device=soft.device)).float().contiguous()

    def first_weights(self) -> torch.Tensor:
        return self.w_up

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        s, rt = self.spec, self.rt
        if x.shape[0] <= ops.SKINNY_FAST_ROWS:
            ops.stream_ahead(self.w_down)              # taken by the up product, read by the product after it
        if self.coeffs is not None:
            act = linear_xielu(x, self.w_up, rt, s.inner, self.coeffs)
        else:
            act = linear_act(x, self.w_up, rt, s.inner, self.activation)
        return linear_partial(act, self.w_down, rt, "ffn_out")


@register_feed_forward("token_side")
class TokenSide:
    """y = proj(gelu_tanh(gate x) * e), e the layer's piece of a table's row for the token; x is the stream itself and y joins
    it made unit-RMS times a weight (x <- x + y / rms(y) * norm), in the kernel of the norm that follows (`post_weight`,
    `post_eps`: parts/block.py).

    Parameters: inner (n), vocab, layers, eps; the spec's `index` says which piece, [index n, (index + 1) n), of the rows of
    the tensor `table` [vocab, layers * n] is this layer's. Tensors: table, gate [n, width], proj [width, n], norm [width]."""

    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)
    graph_safe = True      # launches depend on row counts only
    gate_bias = None

    @staticmethod
    def declare(spec) -> Dict[str, TensorDecl]:
        return {
            "table": TensorDecl((spec.vocab, spec.layers * spec.inner)),
            "gate": TensorDecl((spec.inner, spec.width)),
            "proj": TensorDecl((spec.width, spec.inner)),
            "norm": TensorDecl((spec.width,), role="vector", init="around_one"),
        }

    def __init__(self, spec, tensors: Dict[str, torch.Tensor], runtime):
        if spec.get("activation", "gelu_tanh") != "gelu_tanh":
            raise Unsupported(f"token_side: activation '{spec.activation}' has no kernel (gelu_tanh has)")
        self.spec = spec
        self.rt = runtime
        n = int(spec.inner)
        self.table = tensors["table"][:, spec.index * n:(spec.index + 1) * n]
        self.w_gate, self.w_proj = tensors["gate"], tensors["proj"]
        self.post_weight, self.post_eps = tensors["norm"], float(spec.eps)

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        """x: the stream in the compute dtype."""
        z = self.rt.buffer("token_side", (x.shape[0], self.spec.inner))
        linear(x, self.w_gate, z)
        ops.token_gate(z, self.table, ctx.token_ids, z)
        return linear_partial(z, self.w_proj, self.rt, "token_side_out")
