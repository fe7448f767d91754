"""Token embedding and output head as parts.

Embedding: a row gather (src/ops/embedding.cu:38-52).  Head: logits = x . W^T with W
either `lm_head.weight` or, for tied checkpoints, the embedding table, in which case
`lm_head.weight` is not read (src/model/weights.cpp:116-118,198-204).  The reference
rounds logits to bfloat16 (src/ops/linear.cpp:118); here they leave the product as
float32.

Parameters beyond Qwen3: a sinusoidal vector of the token's position can be added (`positions`); the embedding can be multiplied by a constant (`scale`; its output is
then float32, the hidden state of a model that keeps it in 32-bit); the logits can be
multiplied by a constant (`scale`) and capped smoothly (`softcap`: z <- c tanh(z / c)); the
tensors' names are the prefix plus `tensor`.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear


class TokenEmbedding(Part):
    def __init__(self, vocab_size: int, hidden_size: int, scale: Optional[float] = None, tensor: str = "weight",
                 copies: int = 1, positions: Optional[str] = None, position_base: float = 10000.0):
        """`copies` > 1: every token's row is written that many times side by side (out [N, copies * hidden]).  `positions`
        "sinusoid": column 2i of the output gets sin(p position_base^(-2i / hidden)) added, column 2i + 1 the cosine of the
        same, p the token's position (a float32 hidden state; the vector is not multiplied by `scale`)."""
        if positions not in (None, "sinusoid") or (positions and copies > 1) or not position_base > 0:
            raise ValueError("embedding: positions is None or 'sinusoid', on one copy, with a positive base")
        self.positions, self.position_base = positions, float(position_base)
        self.freq = None
        self.vocab_size, self.hidden_size, self.copies = int(vocab_size), int(hidden_size), int(copies)
        self.scale = None if scale is None else float(scale)
        self.tensor = tensor
        self.table = None

    def weight_specs(self, prefix: str) -> dict:
        return {prefix + self.tensor: WeightSpec((self.vocab_size, self.hidden_size))}

    def bind(self, weights: dict, prefix: str, dtype, device) -> None:
        self.table = weights[prefix + self.tensor].contiguous()
        if self.positions:
            # in float64, handed over as two floats a frequency: the angle p f is then right to 32-bit rounding at any position
            exponent = torch.arange((self.hidden_size + 1) // 2, dtype=torch.float64) * (-2.0 / self.hidden_size)
            freq = torch.pow(torch.tensor(self.position_base, dtype=torch.float64), exponent)
            lead = freq.to(torch.float32)
            self.freq = torch.stack([lead, (freq - lead.to(torch.float64)).to(torch.float32)]).contiguous().to(device)

    def forward(self, token_ids: torch.Tensor, out: torch.Tensor, token_pos: Optional[torch.Tensor] = None) -> torch.Tensor:
        if self.positions:
            if out.dtype != torch.float32 or token_pos is None:
                raise ops.KernelError("an embedding with positions writes a float32 hidden state and needs the tokens' positions")
            return ops.embedding_sinusoid(token_ids, token_pos, self.table, self.freq, out, 1.0 if self.scale is None else self.scale)
        if self.copies > 1:
            return ops.embedding_streams(token_ids, self.table, out, 1.0 if self.scale is None else self.scale, self.copies)
        if out.dtype == torch.float32 and (self.scale is not None or self.table.dtype != torch.float32):
            return ops.embedding_scaled(token_ids, self.table, out, 1.0 if self.scale is None else self.scale)
        if self.scale is not None:
            raise ops.KernelError("a scaled embedding writes a float32 hidden state")
        return ops.embedding(token_ids, self.table, out)


class LMHead(Part):
    def __init__(self, vocab_size: int, hidden_size: int, tied_to: Optional[str] = None, scale: Optional[float] = None,
                 softcap: Optional[float] = None, tensor: str = "weight"):
        self.vocab_size, self.hidden_size, self.tied_to = int(vocab_size), int(hidden_size), tied_to
        self.scale = 1.0 if scale is None else float(scale)
        self.softcap = float(softcap) if softcap else 0.0
        self.tensor = tensor
        self.weight = None

    def weight_specs(self, prefix: str) -> dict:
        return {} if self.tied_to else {prefix + self.tensor: WeightSpec((self.vocab_size, self.hidden_size))}

    def ignorable(self, prefix: str):
        return [prefix + self.tensor] if self.tied_to else []

    def bind(self, weights: dict, prefix: str, dtype, device) -> None:
        self.weight = weights[self.tied_to if self.tied_to else prefix + self.tensor].contiguous()

    def forward(self, x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        linear(x, self.weight, out)
        if self.scale != 1.0 or self.softcap:
            ops.scale_softcap(out, self.scale, self.softcap)
        return out


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("head", "lm_head", LMHead)
