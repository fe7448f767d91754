"""Retention as a mixer part: linear attention with a fixed decay per head, no softmax and no denominator.

q = W_q x and k = W_k x (heads x dim), v = W_v x (heads x vdim); q and k may carry a rotary encoding, k is multiplied by
`k_scale`.  Per head a state S [dim, vdim] that lives in float32 in the cache's state rows (zero for a new sequence,
carried from step to step):

    S_t = decay_h S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t

Every head's o is brought to unit rms by itself (no weight), the heads side by side are multiplied by SiLU(W_g x) and
projected by W_o.  The four input projections run as one product; rotation, recurrence and norm are 32-bit whatever the
compute type, in the kernels of the lightning attention (parts/lightning.py), whose recurrence is the same.  It needs no
keys in the cache: `CacheNeed("none", state_shape=(heads, dim, vdim))`.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from ..cache.book import CacheNeed
from ..config.plan import PartSpec
from ..csrc import ops
from ..weights.loader import WeightSpec
from ..weights.upload import fuse_rows
from . import lightning
from .base import Part, build_part, register_part
from .linear import linear

TENSOR_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o"}


class Retention(Part):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, decay: Sequence[float], eps: float,
                 position: Optional[PartSpec] = None, k_scale: float = 1.0, prefix: str = "", names: Optional[dict] = None):
        if len(decay) != num_heads:
            raise ValueError("one decay per head")
        if not 0 < head_dim <= 256 or not 0 < value_dim <= 256:
            raise ValueError("head sizes up to 256")
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim = int(hidden_size), int(num_heads), int(head_dim), int(value_dim)
        self.decay_values, self.eps, self.k_scale, self.prefix = [float(v) for v in decay], float(eps), float(k_scale), prefix
        self.position = build_part("position", position) if position else None
        if self.position is not None and (not getattr(self.position, "fused_tables", False) or self.position.kernel_order() is not None):
            raise ValueError("retention takes a rotary encoding with tables, in pairs (i, i + dims/2)")
        self.names = dict(TENSOR_NAMES, **(names or {}))
        self.out_name = "mixer.out"
        self.w_in = self.w_o = self.decay = None

    def weight_specs(self, prefix: str) -> dict:
        p, n, H = prefix + self.prefix, self.names, self.hidden_size
        qk, vg = self.num_heads * self.head_dim, self.num_heads * self.value_dim
        return {p + n["q"]: WeightSpec((qk, H)), p + n["k"]: WeightSpec((qk, H)), p + n["v"]: WeightSpec((vg, H)),
                p + n["g"]: WeightSpec((vg, H)), p + n["o"]: WeightSpec((H, vg))}

    def bind(self, weights: dict, prefix: str, dtype, device) -> None:
        p, n = prefix + self.prefix, self.names
        self.w_in = fuse_rows(weights, [p + n[k] for k in ("q", "k", "v", "g")])
        self.w_o = weights.pop(p + n["o"]).contiguous()
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("none", state_shape=(self.num_heads, self.head_dim, self.value_dim))

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        N, h, d, vd = ctx.n_tokens, self.num_heads, self.head_dim, self.value_dim
        proj = ctx.scratch.get("retention.proj", (N, 2 * h * (d + vd)), ctx.dtype)
        linear(x, self.w_in, proj)
        cos = sin = None
        if self.position is not None:
            self.position.prepare(ctx.max_positions, ctx.device)
            cos, sin = self.position.cos, self.position.sin
        o = ctx.scratch.get("retention.o", (N, h * vd), torch.float32)
        chunked = not ctx.is_decode and ctx.max_new >= lightning.chunk_rows and ops.lightning_chunks_fit(d, vd)
        ops.lightning_attention(proj, cache.state, self.decay, ctx.seq_start, ctx.seq_slots, o, ctx.n_seqs, h, d, vd, chunked,
                                silu=False, k_scale=self.k_scale, cos=cos, sin=sin, token_pos=ctx.token_pos,
                                **lightning.segment_scratch(ctx, h, d, vd, chunked))
        gated = ctx.scratch.get("retention.gated", (N, h * vd), ctx.dtype)
        ops.head_gated_norm(o, None, proj[:, 2 * h * d + h * vd:], self.eps, gated, h, vd, act="silu")
        out = ctx.scratch.get(self.out_name, (N, self.hidden_size), ctx.dtype)
        return linear(gated, self.w_o, out)


register_part("mixer", "retention", Retention)
