"""The gated delta rule: the "gated_delta" mixer.

One projection of the layer's input gives, per token, q and k of G heads of d numbers, v of H heads of e numbers, the
output gate z (H x e), and per head a raw write strength b and a raw step size a. q, k and v pass a short causal
convolution over the last `taps` tokens (per channel, no bias) and silu; q and k are then made unit vectors per head
(q also times d^(-1/2)). Per head h (query/key head h / (H / G)), with a matrix state S (d x e) that starts at zero:

    g = exp(-exp(a_log_h) softplus(a + dt_bias_h)),   beta = sigmoid(b)
    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

and the mixer's output is o_proj(o / rms(o) * norm * act(z)), each head normed by itself over its e numbers with one
weight vector shared by the heads, act silu or, by the parameter `gate`, "sigmoid". Nothing is cached per token: a request
keeps one row of a float32 state array, [S of every head | the last taps - 1 inputs of the convolutions], which the cache
manager hands out zeroed.

With decay "channel" there is one g per head and key channel, acting on the rows of S: its raw numbers a (H x d, dt_bias
alike) come from a projection in two steps, decay_out(decay_in h), with an inner vector of decay_rank numbers. With
gate_rank > 0 the output gate does too: z = gate_out(gate_in h). The inner vectors are part of the first product, and one
short product against the block-diagonal matrix of the second steps gives both results in float32.

All sizes come from the spec: num_heads (H), num_kv_heads (G), head_dim (d), value_dim (e), taps, eps; decay ("head",
"channel"), decay_rank, gate ("silu", "sigmoid"), gate_rank.
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..errors import Unsupported
from ..kernels import linear, ops
from ..kernels.gemm import linear_partial, linear_short
from .base import CacheSpec, TensorDecl, register_mixer


@register_mixer("gated_delta")
class GatedDeltaMixer:
    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)
    graph_safe = True      # launches depend on row and request counts only
    out_name = "mixer_out"     # the workspace buffer of the result; a mixer that holds this one may name another

    @staticmethod
    def declare(spec) -> Dict[str, TensorDecl]:
        H, G, d, e, K = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim, spec.taps
        more = {}
        if spec.get("decay", "head") == "channel":
            more.update(decay_in=TensorDecl((spec.decay_rank, spec.width)), decay_out=TensorDecl((H * d, spec.decay_rank)))
        else:
            more["a"] = TensorDecl((H, spec.width))
        if spec.get("gate_rank", 0) > 0:
            more.update(gate_in=TensorDecl((spec.gate_rank, spec.width)), gate_out=TensorDecl((H * e, spec.gate_rank)))
        else:
            more["gate"] = TensorDecl((H * e, spec.width))
        return {
            "q": TensorDecl((G * d, spec.width)), "k": TensorDecl((G * d, spec.width)), "v": TensorDecl((H * e, spec.width)),
            "q_conv": TensorDecl((G * d, K), role="vector", init="bias"),
            "k_conv": TensorDecl((G * d, K), role="vector", init="bias"),
            "v_conv": TensorDecl((H * e, K), role="vector", init="bias"),
            "b": TensorDecl((H, spec.width)), **more,
            "a_log": TensorDecl((H,), role="vector", init="bias"),
            "dt_bias": TensorDecl((H * d if "decay_in" in more else H,), role="vector", init="bias"),
            "norm": TensorDecl((e,), role="vector", init="around_one"),
            "o": TensorDecl((spec.width, H * e)),
        }

    def __init__(self, spec, tensors: Dict[str, torch.Tensor], runtime):
        H, G, d, e = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        if H % G:
            raise Unsupported(f"gated_delta: {H} heads do not divide into {G} query/key heads")
        if d > 512:
            raise Unsupported(f"gated_delta: a state of {d} rows has no kernel (512 at most)")
        self.spec = spec
        self.rt = runtime
        if spec.get("decay", "head") not in ("head", "channel") or spec.get("gate", "silu") not in ("silu", "sigmoid"):
            raise Unsupported(f"gated_delta: no decay '{spec.decay}' (head, channel) or gate '{spec.gate}' (silu, sigmoid)")
        self.qk, self.inner = G * d, H * e
        self.channels = 2 * self.qk + self.inner
        self.by_channel = spec.get("decay", "head") == "channel"
        self.gate_act = spec.get("gate", "silu")
        two_gate = int(spec.get("gate_rank", 0)) > 0
        # one product, [inner vectors | q | k | v | gate | b | a], the pieces that are there; the convolution runs over q, k
        # and v. The inner vectors stand in front and are padded, as is the whole, so that rows and slices start on 16 bytes.
        steps = (["decay"] if self.by_channel else []) + (["gate"] if two_gate else [])
        first, second = [tensors[n + "_in"] for n in steps], [tensors[n + "_out"] for n in steps]
        mats = [self._padded(first)] if first else []
        self.inner_cols = mats[0].shape[0] if first else 0
        mats += [tensors[n] for n in ("q", "k", "v")]
        self.gate_col = self.inner_cols + self.channels
        mats += [] if two_gate else [tensors["gate"]]
        self.b_col = self.gate_col + (0 if two_gate else self.inner)
        self.a_col = self.b_col + H
        mats += [tensors["b"]] + ([] if self.by_channel else [tensors["a"]])
        self.w_in = (self._padded(mats) if first else torch.cat(mats, dim=0)).contiguous()
        self.w_two = None
        if first:
            blocks = torch.block_diag(*second)               # results side by side: [decays | gate]
            w_two = blocks.new_zeros(-(-blocks.shape[0] // 8) * 8, self.inner_cols)
            w_two[:blocks.shape[0], :blocks.shape[1]] = blocks
            self.w_two = w_two.contiguous()
        self.two_gate = two_gate
        self.taps = torch.cat([tensors[n] for n in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()   # [taps, channels]
        self.a_log, self.dt_bias, self.norm = tensors["a_log"], tensors["dt_bias"], tensors["norm"]
        self.w_o = tensors["o"]
        self.eps = float(spec.eps)
        self.keep_off = H * d * e                          # where a slot's kept convolution inputs begin

    @staticmethod
    def _padded(mats) -> torch.Tensor:
        w = torch.cat(mats, dim=0)
        pad = -w.shape[0] % 8
        return torch.cat([w, w.new_zeros(pad, w.shape[1])]) if pad else w

    def first_weights(self) -> torch.Tensor:
        return self.w_in

    def cache_spec(self) -> Optional[CacheSpec]:
        return CacheSpec(kind="state", state_shape=(self.keep_off + (self.spec.taps - 1) * self.channels,), dtype="float32")

    def forward(self, x: torch.Tensor, ctx, cache, owns_cache: bool = True) -> torch.Tensor:
        """x: [rows, width] in the compute dtype -> [rows, width] (or split-K partial sums of it)."""
        s, rt = self.spec, self.rt
        if not owns_cache or cache is None or cache.kind != "state":
            raise Unsupported("gated_delta: every run of the layer keeps a state of its own")
        (state,) = cache.arrays
        rows = x.shape[0]
        H, G, d, e = s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim
        proj = rt.buffer("delta_proj", (rows, self.w_in.shape[0]))
        linear(x, self.w_in, proj)
        two = None
        if self.w_two is not None:
            two = linear_short(proj[:, :self.inner_cols], self.w_two, rt.buffer("delta_two", (rows, self.w_two.shape[0]), torch.float32))
        u = rt.buffer("delta_conv", (rows, self.channels))
        ops.short_conv(proj, self.inner_cols, self.channels, self.taps, None, state, self.keep_off, ctx.positions, ctx.row_request,
                       ctx.row_slot, ctx.pos_start, u, act="silu")
        ops.ssm_conv_keep(proj, self.inner_cols, self.channels, s.taps, state, self.keep_off, ctx.q_start, ctx.state_slots,
                          ctx.num_requests)
        o = rt.buffer("delta_o", (rows, self.inner), torch.float32)
        ops.delta_rule(u, 0, self.qk, 2 * self.qk, proj, self.b_col, self.a_col, self.a_log, self.dt_bias, state, ctx.q_start,
                       ctx.state_slots, o, ctx.num_requests, H, G, d, e, channel_decay=two if self.by_channel else None)
        g = rt.buffer("delta_gated", (rows, self.inner))
        gate, gate_col = (two, H * d if self.by_channel else 0) if self.two_gate else (proj, self.gate_col)
        ops.head_norm_gate(o, gate, gate_col, self.norm, self.eps, g, H, e, act=self.gate_act)
        return linear_partial(g, self.w_o, rt, self.out_name)
