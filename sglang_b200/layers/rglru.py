"""Gated linear recurrence block, the RG-LRU layer of Griffin-style models:

    y, x = W_y h + b_y, W_x h + b_x                      one GEMM, rows [y | x]
    u    = causal convolution of x per channel (+ bias, no activation)
    r, i = sigmoid(R_b u_b + b_r), sigmoid(I_b u_b + b_i)          block-diagonal: ``blocks`` equal parts of the width, square matrices
    log a = -8 r softplus(lam)                           per channel
    S_t  = a S_(t-1) + sqrt(1 - a^2) i u                 S: one fp32 number per channel, zero at the start
    out  = W_o (S * gelu_tanh(y))

It sits beside the other recurrent mixers (``layers/mamba1_scan.py``, ``layers/mamba2_scan.py``): the same ragged convolution kernel and the same
``LayeredStatePool`` row per request slot (``state_idx``), prompt portions, decode tokens and mixed batches in the same launches.  The gates are a
block-diagonal tcgen05 product with an fp32 result (``ops.block_linear_f32``); gate activations, decay, recurrence and output branch are one
kernel that scans the tokens in parallel segments (``ops.rglru_scan``, csrc/kernels/rglru.cu).  Gates, decays and state are fp32; the projections and the convolution's output are
in the model dtype.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..model_executor.forward_batch import ForwardBatch


class RGLRUMixer(nn.Module):
    POWER = 8.0          # the constant in log a

    def __init__(self, width: int, channels: int, blocks: int, taps: int, dtype):
        super().__init__()
        assert channels % blocks == 0, "equal blocks"
        self.C, self.blocks, self.taps = channels, blocks, taps
        self.n = channels // blocks
        mk = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype), requires_grad=False)
        f32 = lambda *s: nn.Parameter(torch.zeros(*s, dtype=torch.float32), requires_grad=False)
        self.in_weight, self.in_bias = mk(2 * channels, width), mk(2 * channels)          # rows [y | x]
        self.conv_weight, self.conv_bias = mk(channels, taps), mk(channels)
        self.gate_weight = mk(blocks, 2 * self.n, self.n)                                   # per block: recurrence-gate rows, input-gate rows
        self.gate_bias = f32(blocks, 2 * self.n)
        self.lam = f32(channels)
        self.o_weight = mk(width, channels)

    # ---- geometry for the recurrent-state pool: (conv channels, taps, heads, state rows, head_dim)
    def state_geometry(self):
        return (self.C, self.taps, 1, 1, self.C)

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        C, n = self.C, self.n
        dst = {"y": lambda: self.in_weight.data[:C], "y.b": lambda: self.in_bias.data[:C], "x": lambda: self.in_weight.data[C:], "x.b": lambda: self.in_bias.data[C:],
               "conv": lambda: self.conv_weight.data, "conv.b": lambda: self.conv_bias.data, "ra": lambda: self.gate_weight.data[:, :n],
               "ri": lambda: self.gate_weight.data[:, n:], "ra.b": lambda: self.gate_bias.data[:, :n], "ri.b": lambda: self.gate_bias.data[:, n:],
               "lam": lambda: self.lam.data, "o": lambda: self.o_weight.data}.get(leaf)
        if dst is None:
            return False
        d = dst()
        d.copy_(w.to(d.dtype).reshape(d.shape))
        return True

    def forward(self, h: torch.Tensor, fb: ForwardBatch, state_idx: int) -> torch.Tensor:
        pool, C = fb.kv_pool.mamba, self.C
        proj = ops.linear(h, self.in_weight, self.in_bias)                       # [T, y | x]
        x = proj[:, C:]
        if self.taps > 1:
            u = ops.causal_conv1d(x, self.conv_weight, self.conv_bias, pool.conv[state_idx], fb.cu_q, fb.req_slots, fb.seq_lens, fb.max_q_len, silu=False,
                                  out_dtype=h.dtype)
        else:
            u = (x.float() * self.conv_weight[:, 0].float() + self.conv_bias.float()).to(h.dtype).contiguous()
        gates = ops.block_linear_f32(u, self.gate_weight)                        # [T, blocks, r | i] fp32
        s = ops.rglru_scan(gates, self.gate_bias, u, self.lam, proj[:, :C], pool.ssm[state_idx], fb.req_slots, fb.seq_lens, fb.cu_q, fb.q_lens, self.blocks,
                           self.POWER)
        return ops.linear(s, self.o_weight)
