"""Two mixers side by side on the same input, ``left_scale * left(h) + right_scale * right(h)``: an attention (``layers/gated_attention.py``) and a
decaying linear attention (``layers/linear_attention.py``), both built with ``own_projection=False``.

One projection GEMM with rows [left q | k | v | g | right v | k | q | g] (a bias where the left side has one), and one output GEMM over the two
sides' gated heads side by side: the constants are folded into the epilogues that produce the heads, and the left output bias (if any) times
its constant is added by the GEMM.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..model_executor.forward_batch import ForwardBatch
from .gated_attention import GatedAttention
from .linear_attention import DecayLinearAttention


class ParallelMixer(nn.Module):
    def __init__(self, width: int, left: GatedAttention, right: DecayLinearAttention, left_scale: float, right_scale: float, dtype):
        super().__init__()
        self.left, self.right = left, right
        left.out_scale, right.out_scale = float(left_scale), float(right_scale)
        has_o_bias = left.o_bias is not None
        left.o_weight = left.o_bias = right.o_weight = None          # they live in ``o_weight`` / ``o_bias`` below
        nl, nr = left.rows, right.rows
        self.in_weight = nn.Parameter(torch.zeros(nl + nr, width, dtype=dtype), requires_grad=False)
        self.in_bias = nn.Parameter(torch.zeros(nl + nr, dtype=dtype), requires_grad=False) if left.has_bias else None
        self.n_ol, self.n_or = left.H * left.Dv, right.n_v
        self.o_weight = nn.Parameter(torch.zeros(width, self.n_ol + self.n_or, dtype=dtype), requires_grad=False)
        self.o_bias = nn.Parameter(torch.zeros(width, dtype=dtype), requires_grad=False) if has_o_bias else None       # left output bias times left_scale

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        side, _, rest = leaf.partition(".")
        if side == "left":
            if rest == "o":
                self.o_weight.data[:, :self.n_ol].copy_(w)
                return True
            if rest == "o.b" and self.o_bias is not None:
                self.o_bias.data.copy_((w.float() * self.left.out_scale).to(self.o_bias.dtype))
                return True
            return self.left.load_in(rest, w, self.in_weight, self.in_bias, 0) or self.left.load(rest, w)
        if side == "right":
            if rest == "o":
                self.o_weight.data[:, self.n_ol:].copy_(w)
                return True
            return self.right.load_in(rest, w, self.in_weight, None, self.left.rows) or self.right.load(rest, w)
        return False

    def forward(self, h: torch.Tensor, fb: ForwardBatch, cache_idx: int, state_idx: int) -> torch.Tensor:
        proj = ops.linear(h, self.in_weight, self.in_bias)
        cat = torch.empty(h.shape[0], self.n_ol + self.n_or, dtype=h.dtype, device=h.device)
        self.left.attend(proj[:, :self.left.rows], fb, cache_idx, None, cat[:, :self.n_ol])
        self.right.attend(proj[:, self.left.rows:], fb, state_idx, cat[:, self.n_ol:])
        return ops.linear(cat, self.o_weight, self.o_bias)
