"""A selective state-space layer (Mamba-2, state-space duality) as a mixer part.

One projection gives a gate z (heads x vdim), x (heads x vdim), B and C (groups x state) and a step logit per head.  x, B and
C pass a short causal convolution per channel with a bias and SiLU; dt = softplus(logit + dt_bias).  Per head (which reads
the B and C of its group) a matrix S [state, vdim] lives in float32 in the cache's state rows (zero for a new sequence,
carried from step to step):

    S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,     y_t = S_t^T C_t + D x_t

y is multiplied by SiLU(z), brought to unit rms in `norm_groups` equal parts of the row, multiplied by a weight and projected
by W_o.  The step logits leave their product in 32-bit; step sizes, decays, state, outputs and norm are 32-bit whatever the
compute type.  A sequence's state row holds heads x state x vdim values and, behind them, the convolution's last taps - 1
input rows.  No keys in the cache.  Decode steps and the 32-bit path walk token by token (`ops.decay_scan`); bfloat16 prompts
run in chunks on the tensor cores (`ops.ssd_prompt`).
"""
from __future__ import annotations

from typing import Optional

import torch

from ..cache.book import CacheNeed
from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear

TENSOR_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "a_log": "A_log", "skip": "D", "norm": "norm",
                "o": "o"}

chunk_rows = 32      # from this many new tokens of the longest sequence on, bfloat16 steps run the chunked form


class StateSpace(Part):
    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state: int, groups: int, taps: int, norm_groups: int, eps: float,
                 prefix: str = "", names: Optional[dict] = None):
        if num_heads <= 0 or groups <= 0 or num_heads % groups or not 0 < state <= 256 or not 0 < value_dim <= 256 or not 0 < taps <= 64:
            raise ValueError("state space: heads in equal groups, state and value sizes up to 256, up to 64 taps")
        if norm_groups <= 0 or num_heads * value_dim % norm_groups:
            raise ValueError("state space: the norm's groups divide heads x value size")
        self.hidden_size, self.num_heads, self.value_dim, self.state = int(hidden_size), int(num_heads), int(value_dim), int(state)
        self.groups, self.taps, self.norm_groups, self.eps, self.prefix = int(groups), int(taps), int(norm_groups), float(eps), prefix
        self.inner = self.num_heads * self.value_dim
        self.channels = self.inner + 2 * self.groups * self.state          # what the convolution runs over
        self.names = dict(TENSOR_NAMES, **(names or {}))
        self.out_name = "mixer.out"
        self.w_in = self.w_dt = self.w_o = self.conv = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.norm_weight = None

    def weight_specs(self, prefix: str) -> dict:
        p, n, H, h = prefix + self.prefix, self.names, self.hidden_size, self.num_heads
        return {p + n["in"]: WeightSpec((self.inner + self.channels + h, H)), p + n["conv"]: WeightSpec((self.channels, self.taps), "bias"),
                p + n["conv_bias"]: WeightSpec((self.channels,), "bias"), p + n["dt_bias"]: WeightSpec((h,), "bias"),
                p + n["a_log"]: WeightSpec((h,), "bias"), p + n["skip"]: WeightSpec((h,), "bias"),
                p + n["norm"]: WeightSpec((self.inner,), "norm"), p + n["o"]: WeightSpec((H, self.inner))}

    def bind(self, weights: dict, prefix: str, dtype, device) -> None:
        p, n = prefix + self.prefix, self.names
        whole = weights.pop(p + n["in"])
        # the step logits are a product of their own: they stay in 32-bit
        self.w_in, self.w_dt = whole[:self.inner + self.channels], whole[self.inner + self.channels:]
        self.w_o = weights.pop(p + n["o"]).contiguous()
        f32 = dict(device=device, dtype=torch.float32)
        conv = weights[p + n["conv"]]
        self.conv_bias, self.dt_bias, self.a_log, self.skip, self.norm_weight = (
            weights[p + n[k]].to(**f32).contiguous() for k in ("conv_bias", "dt_bias", "a_log", "skip", "norm"))
        getattr(weights, "wait", lambda: None)()              # a streamed checkpoint: the tensors are in place now
        self.conv = conv.to(**f32).t().contiguous()           # [taps, channels], as the kernel reads it

    def cache_need(self) -> CacheNeed:
        return CacheNeed("none", state_shape=(self.cells() + (self.taps - 1) * self.channels,))

    def cells(self) -> int:
        return self.num_heads * self.state * self.value_dim

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        N, h, vd, n, G, inner = ctx.n_tokens, self.num_heads, self.value_dim, self.state, self.groups, self.inner
        s = ctx.scratch
        proj = linear(x, self.w_in, s.get("ssm.proj", (N, inner + self.channels), ctx.dtype))
        dt = linear(x, self.w_dt, s.get("ssm.dt", (N, h), torch.float32))
        rows = cache.state.view(cache.state.shape[0], -1)
        conv_state = rows[:, self.cells():] if self.taps > 1 else s.get("ssm.no_state", (1, 0), torch.float32)
        u = s.get("ssm.conv", (N, self.channels), ctx.dtype)
        ops.short_conv(proj[:, inner:], self.conv, conv_state, ctx.token_seq, ctx.seq_start, ctx.seq_slots, u, ctx.n_seqs,
                       bias=self.conv_bias, silu=True, single=ctx.is_decode)
        B, C = u[:, inner:inner + G * n], u[:, inner + G * n:]
        y = s.get("ssm.y", (N, inner), torch.float32)
        steps = dict(share=h // G, dt_logits=dt, dt_bias=self.dt_bias, a_log=self.a_log, skip=self.skip)
        args = (C, B, u[:, :inner], rows[:, :self.cells()], ctx.seq_start, ctx.seq_slots, y, ctx.n_seqs, h, n, vd)
        if not ctx.is_decode and ctx.max_new >= chunk_rows and ops.ssd_prompt_fits(u, n, vd):
            segments = ops.ssd_segments(ctx.n_seqs, ctx.max_new, h, n, vd)
            between = s.get("ssm.segments", (ctx.n_seqs * segments * h * (n * vd + 1),), torch.float32) if segments > 1 else None
            ops.ssd_prompt(*args, max_new=ctx.max_new, scratch=between, segments=segments, **steps)
        else:
            ops.decay_scan(*args, **steps, single=ctx.is_decode and ops.state_step_fits(args[3], vd))
        gated = s.get("ssm.gated", (N, inner), ctx.dtype)
        ops.gate_group_norm(y, proj[:, :inner], self.norm_weight, self.eps, gated, self.norm_groups)
        return linear(gated, self.w_o, s.get(self.out_name, (N, self.hidden_size), ctx.dtype))


register_part("mixer", "state_space", StateSpace)
