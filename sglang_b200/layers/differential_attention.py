"""Differential grouped-query attention with a short convolution over its projections:

    q, k, v   = W h                               one GEMM, rows [q | k | v]; q and k carry two maps per head, [map 1 | map 2]
    u_t       <- sum_j w[c, j] u_(t - taps + 1 + j)   per channel of q, k and v; zeros before the sequence
    q, k      <- rms(q) * w_q, rms(k) * w_k       per head and map, plain weights shared by all of them
    q, k      <- rotation by position             ``rotary = (dims, inv_freq, mult)``: the first ``dims`` coordinates of every map, coordinate i paired
                                                  with i + dims/2; ``mult`` on sine and cosine
    visible   j <= i and i // chunk == j // chunk     ``chunk > 0``; otherwise every j <= i
    a_m       = softmax(q_m . k_m * scale) v       per map m of a head, over the same values
    o         = a_1 - lam a_2;   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)
    lam       = exp(lq1 . lk1) - exp(lq2 . lk2) + diff          one number per layer
    y         = W_o o

How it maps to the kernels: ``ops.conv_attention_prepare`` (csrc/kernels/conv_attention.cu) does lines two to four, the cache write and the
convolution state.  A key head is cached as its two maps side by side, and a query map is laid out over that width with zeros in the other
map's place, so that two maps over shared values are ordinary grouped-query attention with twice the query heads: values are read once for
both, and the framework's attention kernels serve it with two additions, the chunk in their masks (keys before the chunk are never loaded)
and an epilogue that combines neighbouring query heads in fp32 before anything is rounded.  bf16 models whose maps are at most 64 and values
at most 128 wide run the tcgen05 kernels (``pad = 128``: two 64-column segments, which is exactly the key tile's two swizzled halves); other
sizes and fp32 serving run ``ops.window_attention``.

The paged pool holds one flat row per token and plane (``FlatCacheSpec`` of ``layers/window_attention.py``); the chunk only masks, pages behind it
stay with the request until it ends.  The last ``taps - 1`` projection rows of every request live in the ``LayeredStatePool``.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..model_executor.forward_batch import ForwardBatch


class DifferentialAttention(nn.Module):
    tc_route = True            # class-wide switch of the tcgen05 route (tests compare it with the general kernel)
    MAPS = 2

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: Optional[float], diff: float, eps: float, dtype, *,
                 taps: int = 1, rotary: Optional[Tuple[int, torch.Tensor, float]] = None, chunk: int = 0, qk_norm: bool = True):
        super().__init__()
        assert heads % kv_heads == 0 and taps >= 1
        self.H, self.G, self.D, self.Dv, self.eps, self.taps = heads, kv_heads, dim, vdim, eps, taps
        self.scale = float(scale) if scale is not None else dim ** -0.5
        self.diff, self.chunk = float(diff), int(chunk or 0)
        M = self.MAPS
        self.n_q, self.n_k, self.n_v = heads * M * dim, kv_heads * M * dim, kv_heads * vdim
        self.rows = self.n_q + self.n_k + self.n_v
        mk = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype), requires_grad=False)
        self.in_weight = mk(self.rows, width)
        self.conv_weight = mk(self.rows, taps)
        self.o_weight = mk(width, heads * vdim)
        self.q_norm = mk(dim) if qk_norm else None
        self.k_norm = mk(dim) if qk_norm else None
        self.lam_vecs = nn.Parameter(torch.zeros(4, dim, dtype=torch.float32), requires_grad=False)          # rows lq1, lk1, lq2, lk2
        self._lam: Optional[float] = None
        if rotary is not None:
            assert rotary[0] % 2 == 0 and rotary[0] <= dim and rotary[1].numel() == rotary[0] // 2
        self.inv_freq = nn.Parameter(rotary[1].float().clone(), requires_grad=False) if rotary is not None else None
        self.rot_mult = float(rotary[2]) if rotary is not None else 1.0
        self.pad = 128 if self._fits_tc(dtype) else 0

    def _fits_tc(self, dtype) -> bool:
        return bool(self.tc_route and dtype == torch.bfloat16 and self.D <= 64 and self.Dv <= 128 and 128 % (self.MAPS * (self.H // self.G)) == 0)

    @property
    def cache_width(self) -> int:
        return self.G * (self.pad if self.pad else max(self.MAPS * self.D, self.Dv))

    @property
    def query_heads(self) -> int:
        """query heads as the attention kernel sees them"""
        return self.MAPS * self.H

    def state_geometry(self) -> Tuple[int, int, int, int, int]:
        return self.rows, self.taps, 0, 0, 0

    # ---- weights
    def load(self, leaf: str, w: torch.Tensor) -> bool:
        a, b = self.n_q, self.n_q + self.n_k
        rows = {"q": (0, a), "k": (a, b), "v": (b, self.rows)}
        head, _, tail = leaf.partition(".")
        if leaf in rows:
            self.in_weight.data[rows[leaf][0]:rows[leaf][1]].copy_(w)
        elif head in rows and tail == "conv":
            self.conv_weight.data[rows[head][0]:rows[head][1]].copy_(w)
        elif leaf in ("q.norm", "k.norm") and self.q_norm is not None:
            (self.q_norm if head == "q" else self.k_norm).data.copy_(w)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            self.lam_vecs.data[("lq1", "lk1", "lq2", "lk2").index(leaf)].copy_(w.float())
            self._lam = None
        elif leaf == "o":
            self.o_weight.data.copy_(w)
        else:
            return False
        return True

    def lam(self) -> float:
        if self._lam is None:
            v = self.lam_vecs.detach().double().cpu()
            self._lam = math.exp(float((v[0] * v[1]).sum())) - math.exp(float((v[2] * v[3]).sum())) + self.diff
        return self._lam

    # ---- forward
    def forward(self, h: torch.Tensor, fb: ForwardBatch, cache_idx: int, state_idx: int) -> torch.Tensor:
        T = h.shape[0]
        H, G, D, Dv, M, pad = self.H, self.G, self.D, self.Dv, self.MAPS, self.pad
        kc, vc = fb.kv_pool.k(cache_idx), fb.kv_pool.v(cache_idx)                  # [slots, 1, cache_width] each
        q = ops.conv_attention_prepare(ops.linear(h, self.in_weight), H, G, M, D, Dv, self.conv_weight, fb.kv_pool.mamba.conv[state_idx], fb.positions, fb.cu_q,
                                       fb.req_slots, fb.seq_lens, self.q_norm, self.k_norm, self.eps, self.inv_freq, self.rot_mult, kc, vc, fb.out_cache_loc, pad)
        diff = (self.lam(), 1.0 - self.diff, self.eps)
        if self.tc_route and pad == 128:
            k4, v4 = kc[:, 0, :G * 128].unflatten(-1, (G, 128)), vc[:, 0, :G * 128].unflatten(-1, (G, 128))      # the leading columns of the pool's rows
            if ops.tc_attention_ok(q, k4, v4, fb.page_size):
                dec = fb.cu_q is None
                splits = fb.num_splits if dec else 1
                if self.chunk > 0:             # a chunk bounds the keys of a query: no more parts than give every one a few key tiles
                    splits = min(splits, max(1, self.chunk // 256))
                o = ops.paged_attention(q, k4, v4, fb.page_table, fb.req_slots, fb.seq_lens, fb.cu_q, fb.q_lens, fb.max_q_len, fb.page_size, self.scale,
                                        causal=True, num_splits=splits, workspace=fb.attn_workspace if splits > 1 else None, chunk=self.chunk, diff=diff,
                                        diff_dv=Dv)
                return ops.linear(o.view(T, H * Dv), self.o_weight)
        o = ops.window_attention(q, kc, vc, G, Dv, fb.page_table, fb.req_slots, fb.seq_lens, fb.cu_q, fb.q_lens, fb.max_q_len, fb.page_size, self.scale,
                                 dim=pad if pad else M * D, pad=pad, chunk=self.chunk, diff=diff)
        return ops.linear(o.reshape(T, H * Dv), self.o_weight)
