"""Position encodings a mixer can apply to its queries and keys.

"rotary": half-split rotary embedding with optional per-pair frequency divisors (llama3 scaling) and a
position scale (linear scaling), as CpuDevice::rope (dynacore/cpu/cpu_device.cpp:1228-1262). The
frequencies are made here in 32-bit floats exactly as the reference makes them,
`pow(base, -2 i / rot) / factor_i`; the rotation itself happens inside the fused kernel
(csrc/rope_cache.cu), which asks this part for `table()`.
"rotary_interleaved": rotary embedding in the interleaved layout: numbers 2i and 2i + 1 of the first `rotary_dim`
of a vector form a pair that turns by position * theta^(-2i / rotary_dim). The frequencies are kept in double
precision and the kernels form the angle in double precision (csrc/latent_attention.cu), so the rotation is exact to
float32 at any position; the mixer that uses it asks for `frequencies` (and `magnitude`, a factor on the turned numbers).
"rotary_halves": the same precision for the half-split layout: numbers i and i + rotary_dim / 2 form a pair. A mixer whose
kernels turn neighbours only may reorder its rows with `neighbours()` (queries and keys alike: their products stay).
"none": no position encoding.

A further kind implements `table()` returning None and `apply(q, k, positions)` rotating its views in
place; the attention mixer then calls `apply` before its cache write.
"""

from __future__ import annotations

from typing import Optional, Tuple

import numpy as np
import torch

from ..errors import Unsupported
from .base import register_position


@register_position("rotary")
class RotaryEncoding:
    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)

    def __init__(self, spec, runtime):
        if spec.rotary_dim <= 0 or spec.rotary_dim > spec.head_dim or spec.rotary_dim % 2:
            raise Unsupported(f"rotary_dim {spec.rotary_dim} invalid for head_dim {spec.head_dim}")
        half = spec.rotary_dim // 2
        base = np.float32(spec.theta)
        i = np.arange(half, dtype=np.float32)
        inv = np.power(base, (np.float32(-2.0) * i) / np.float32(spec.rotary_dim), dtype=np.float32)
        if spec.factors is not None:
            if len(spec.factors) != half:
                raise Unsupported(f"rotary encoding has {len(spec.factors)} factors for {half} pairs")
            inv = (inv / np.asarray(spec.factors, dtype=np.float32)).astype(np.float32)
        self.spec = spec
        self.inv_freq = torch.from_numpy(inv).to(runtime.device)
        self.rotary_dim = spec.rotary_dim
        self.pos_scale = float(np.float32(spec.pos_scale))

    def table(self) -> Optional[Tuple[torch.Tensor, int, float]]:
        """(inverse frequencies float32 [rotary_dim / 2], rotary_dim, position scale) for the fused kernel."""
        return self.inv_freq, self.rotary_dim, self.pos_scale

    def step_angles(self, ctx, runtime) -> torch.Tensor:
        """(cos, sin) of every pair for every row of the step, float32 [rows, rotary_dim / 2, 2]: computed once per
        step and shared by all layers with the same encoding."""
        key = ("rope_angles", self.rotary_dim, self.pos_scale, float(self.spec.theta), self.spec.factors)
        got = ctx.extras.get(key)
        if got is None:
            from ..kernels import ops
            half = self.rotary_dim // 2
            flat = runtime.flat(f"rope_angles_{abs(hash(key)) % (1 << 32):08x}", runtime.max_tokens * half * 2)
            got = flat[:ctx.num_tokens * half * 2].view(ctx.num_tokens, half, 2)
            ops.rope_angles(ctx.positions, self.inv_freq, self.pos_scale, ctx.num_tokens, got)
            ctx.extras[key] = got
        return got


@register_position("rotary_interleaved")
class InterleavedRotaryEncoding:
    replay_safe = True     # it launches nothing itself
    interleaved = True

    def __init__(self, spec, runtime):
        if spec.rotary_dim <= 0 or spec.rotary_dim > spec.head_dim or spec.rotary_dim % 2:
            raise Unsupported(f"rotary_dim {spec.rotary_dim} invalid for a rotated part of {spec.head_dim} numbers")
        i = np.arange(spec.rotary_dim // 2, dtype=np.float64)
        self.spec = spec
        self.rotary_dim = spec.rotary_dim
        freq = np.power(float(spec.theta), -2.0 * i / spec.rotary_dim)
        if spec.get("factors") is not None:
            if len(spec.factors) != spec.rotary_dim // 2:
                raise Unsupported(f"rotary encoding has {len(spec.factors)} factors for {spec.rotary_dim // 2} pairs")
            freq = freq / np.asarray(spec.factors, dtype=np.float64)
        self.magnitude = float(spec.get("magnitude", 1.0))     # what cos and sin are multiplied by
        self.frequencies = torch.from_numpy(freq).to(runtime.device)
        # the same in float32, for a kernel that forms the angle in float32 (csrc/qk_proj_norm.cu)
        self.inv_freq = torch.from_numpy(freq.astype(np.float32)).to(runtime.device)

    def table(self):
        return None


@register_position("rotary_halves")
class HalvesRotaryEncoding(InterleavedRotaryEncoding):
    interleaved = False
    halves = True

    def neighbours(self, size: int) -> torch.Tensor:
        """The order of a vector's `size` numbers in which the two of a pair stand side by side: 0, h, 1, h + 1, ... (h =
        rotary_dim / 2), then the numbers that are not turned."""
        half = self.rotary_dim // 2
        turned = torch.arange(self.rotary_dim).view(2, half).t().reshape(-1)
        return torch.cat([turned, torch.arange(self.rotary_dim, size)])


@register_position("none")
class NoPosition:
    replay_safe = True     # all device work goes through the recorded launches of kernels/ops.py (engine/launch_memo.py)

    def __init__(self, spec, runtime):
        self.spec = spec

    def table(self):
        return None

    def apply(self, q, k, positions) -> None:
        return None
