"""Hyper-connections: S parallel residual streams instead of one.  For a sublayer with the numbers ``in`` [S], ``out`` [S] and ``mix`` [S, S]
(indexed [from, to]):

    u   = sum_s in[s] x_s
    y   = sublayer(norm(u))
    x_t <- sum_s mix[s, t] x_s + mult * out[t] * y            simultaneously for every t

The streams start as S copies of the embedding output and end as their sum.  ``ops.stream_mix_norm`` applies one sublayer's update, forms the
next sublayer's u and norms it in one kernel over the fp32 streams; ``StreamMix.pack`` makes the numbers it takes.  With one stream and
``in = out = mix = 1`` this is the ordinary residual sum.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn


class StreamMix(nn.Module):
    """the numbers of one sublayer (fp32)"""

    def __init__(self, streams: int):
        super().__init__()
        f32 = lambda t: nn.Parameter(t.float(), requires_grad=False)
        self.cin, self.cout, self.mix = f32(torch.full((streams,), 1.0 / streams)), f32(torch.ones(streams)), f32(torch.eye(streams))

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        p = {"in": self.cin, "out": self.cout, "mix": self.mix}.get(leaf)
        if p is None:
            return False
        p.data.copy_(w.float().reshape(p.shape))
        return True

    @staticmethod
    def pack(prev: Optional["StreamMix"], nxt: Optional["StreamMix"], mult: float, streams: int, device) -> torch.Tensor:
        """``prev``: the sublayer whose output is added (None: none yet); ``nxt``: the sublayer to be fed (None: the sum of the streams) ->
        fp32 [S*S + 2*S] = mix | mult * out | in"""
        dev = dict(dtype=torch.float32, device=device)
        mix = prev.mix.detach().to(**dev).reshape(-1) if prev is not None else torch.eye(streams, **dev).reshape(-1)
        out = prev.cout.detach().to(**dev) * mult if prev is not None else torch.zeros(streams, **dev)
        cin = nxt.cin.detach().to(**dev) if nxt is not None else torch.ones(streams, **dev)
        return torch.cat([mix, out, cin]).contiguous()
