"""Surasun beside the closest existing family at equal size (``python bench.py --hybrid-compare --hybrid-family surasun``).

Two parts, random weights, one GPU:

1. **engine**: prefill and decode throughput of a four-layer Surasun slice (gated recurrence, Mamba-2, attention beside retention, gated recurrence, a
   feed-forward behind each; four streams) and of a Resatar slice of the same width (selective scan, selective scan, window attention beside
   decaying linear attention, selective scan): equal head counts and sizes, inner widths, taps, feed-forward parameters; through
   ``Scheduler.replay_step`` (the serving step), and for Surasun also with captured decode steps through ``Engine.generate`` (Resatar has none).
2. **kernels**: each new kernel beside the like op of the closest model on the same shapes: ``stream_mix_norm`` vs the fp32-residual norm kernel;
   ``rglru_scan`` vs ``mamba1_scan`` at equal channels; the block-diagonal product vs the batched cuBLAS product; the convolution in the model
   dtype vs its fp32 form; attention with score cap and head gate on the tcgen05 kernels vs the same kernels alone, and the general kernel
   likewise; ``attention_prepare`` with neighbouring pairs vs the other layout and vs ``rope_kv_write``; ``linear_attention_prepare`` vs the
   activation pass; the scan at retention's and Mamba-2's shapes; the head norm with the SiLU gate vs the joint norm with the sigmoid gate.
   Roofline: algorithmic bytes over the measured copy bandwidth, or FLOPs over the measured bf16 GEMM rate where they take longer.

Timing: CUDA events on the launching stream, >= 3 warm-ups, an L2 flush (a 256 MB write) between timed iterations.  Kernels are enqueued while the
flush still runs, so that an op of a few microseconds is not timed by its host-side launch; engine steps are timed from an idle stream.
Prints one JSON line per measurement and a closing summary line.
"""
from __future__ import annotations

import json
from typing import List

import torch

from .hybrid_compare import _engine_numbers, _peaks, _Timer
from .mumasun_compare import _captured_decode


class _KernelTimer(_Timer):
    """events around work that is already enqueued behind the flush"""

    def __call__(self, fn, iters: int = 7, warmup: int = 3) -> float:
        for _ in range(warmup):
            fn()
        ts = []
        for _ in range(iters):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            self.flush.fill_(1)
            self.flush.fill_(2)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return sorted(ts)[len(ts) // 2]


def _decays(n: int) -> list:
    return [1.0 - 2.0 ** (-5 - 3 * i / max(1, n - 1)) for i in range(n)]


def _surasun_cfg(width: int, heads: int, ff: int, streams: int = 4) -> dict:
    rot = {"dims": 128, "base": 10000.0}
    par = {"type": "parallel", "mixer": {"left": {"heads": heads // 2, "kv_heads": max(1, heads // 16), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                                                  "rot": rot},
                                         "right": {"heads": heads // 2, "dim": 128, "vdim": 128, "decay": _decays(heads // 2), "rot": rot},
                                         "left_scale": 1.0, "right_scale": 1.0}}
    lru = {"type": "rglru", "mixer": {"width": 2 * width, "blocks": 2 * width // 256, "conv": 4}}
    m2 = {"type": "mamba2", "mixer": {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4}}
    mlp = {"kind": "dense", "ff": ff}
    return {"architecture": "Surasun", "width": width, "vocab": 32000, "norm": {"eps": 1e-6}, "streams": streams, "residual_mult": 1.0,
            "layers": [dict(l, mlp=mlp) for l in (lru, m2, par, lru)]}


def _resatar_cfg(width: int, heads: int, ff: int) -> dict:
    par = {"type": "parallel", "mixer": {"left": {"heads": heads // 2, "kv_heads": max(1, heads // 16), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                                  "mask": {"size": 8192, "keep_first": 4}},
                                         "right": {"heads": heads // 2, "dim": 128, "vdim": 128, "decay": _decays(heads // 2)},
                                         "left_scale": 1.0, "right_scale": 1.0}}
    m1 = {"type": "mamba1", "mixer": {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}}
    mlp = {"kind": "dense", "ff": 3 * ff // 2}          # two matrices against three
    return {"architecture": "Resatar", "width": width, "vocab": 32000, "norm": {"eps": 1e-6}, "layers": [dict(l, mlp=mlp) for l in (m1, m1, par, m1)]}


def _kernel_numbers(timer: _Timer, hbm_gbs: float, tflops: float) -> List[dict]:
    from .. import ops
    from ..layers.gated_attention import scaled_inv_freq

    dev, out, bf = "cuda", [], torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(bf)

    def rec(kernel, phase, shape, ms, nbytes, like, like_ms, like_bytes=None, flops=None, like_flops=None):
        """the fraction of the roofline that bounds the kernel: bytes, or FLOPs when given and slower"""
        def frac(b, f, t):
            tb, tf = b / (hbm_gbs * 1e9), (f or 0.0) / (tflops * 1e12)
            return max(tb, tf) / (t * 1e-3), "tensor" if tf > tb else "bytes"

        lb = nbytes if like_bytes is None else like_bytes
        lf = flops if like_flops is None else like_flops
        (a, bound), (b, _) = frac(nbytes, flops, ms), frac(lb, lf, like_ms)
        out.append({"part": "kernel", "kernel": kernel, "phase": phase, "shape": shape, "ms": round(ms, 4), "algorithmic_mb": round(nbytes / 1e6, 2), "bound": bound,
                    "roofline_frac": round(a, 4), "like": like, "like_ms": round(like_ms, 4), "like_roofline_frac": round(b, 4),
                    "distance_ratio": round(b / max(a, 1e-9), 3)})

    def ragged(B, S, past=2000):
        T = B * S
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        sl = torch.full((B,), S if S > 1 else past, dtype=torch.int32, device=dev)
        cu = torch.arange(0, T + 1, S, dtype=torch.int32, device=dev) if S > 1 else None
        return T, slots, sl, cu, (sl if S > 1 else None), ("prefill" if S > 1 else "decode")

    # ---- streams
    for T in (8192, 32):
        W = 4096
        res, d, w = torch.randn(T, W, device=dev, generator=g), rnd(T, W), torch.ones(W, device=dev, dtype=bf)
        like = timer(lambda: ops.add_rmsnorm_f32(res, d, w, 1e-6, False, bf, w))
        for S in (1, 2, 3, 4, 6):
            x, coef = torch.randn(T, S, W, device=dev, generator=g), torch.randn(S * S + 2 * S, device=dev, generator=g) * 0.3
            ms = timer(lambda: ops.stream_mix_norm(x, d, coef, S, w, 1e-5, bf))
            rec("stream_mix_norm", "any", f"T{T} W{W} streams{S}", ms, T * W * (8 * S + 4), "add_rmsnorm_f32(post_weight), one stream", like, T * W * 12)
    # ---- gated recurrence: convolution, gates, scan
    for C, nb in ((2560, 10), (4096, 16)):
        n = C // nb
        gw, gb, lam = rnd(nb, 2 * n, n, sc=n ** -0.5), torch.zeros(nb, 2 * n, device=dev), torch.full((C,), -4.0, device=dev)
        cw, cb = rnd(C, 4), rnd(C)
        dtb, A_log, D = torch.zeros(C, device=dev), torch.zeros(C, 16, device=dev), torch.ones(C, device=dev)
        for B, S in ((4, 2048), (1, 4096), (32, 1), (256, 1)):
            T, slots, sl, cu, ql, ph = ragged(B, S)
            shape = f"B{B} S{S} C{C}"
            yx, cs = rnd(T, 2 * C), torch.zeros(B + 1, C, 3, device=dev, dtype=bf)
            ms = timer(lambda: ops.causal_conv1d(yx[:, C:], cw, cb, cs, cu, slots, sl, S, False, bf))
            like = timer(lambda: ops.causal_conv1d(yx[:, C:], cw, cb, cs, cu, slots, sl, S))
            rec("causal_conv1d, model dtype out", ph, shape, ms, T * C * 4, "causal_conv1d, SiLU, fp32 out (same kernel)", like, T * C * 6)
            u = rnd(T, C)
            ms = timer(lambda: ops.block_linear_f32(u, gw))
            ub, wt = u.view(T, nb, n).transpose(0, 1), gw.transpose(1, 2)
            like = timer(lambda: torch.bmm(ub, wt, out_dtype=torch.float32))
            rec("block_linear_f32 (tcgen05, block-diagonal, fp32 out)", ph, f"{shape} blocks of {n}", ms, T * C * 10 + gw.numel() * 2, "batched cuBLAS product, fp32 out", like,
                None, 4.0 * T * C * n)
            gates, st = ops.block_linear_f32(u, gw), torch.zeros(B + 1, 1, 1, C, device=dev)
            ms = timer(lambda: ops.rglru_scan(gates, gb, u, lam, yx[:, :C], st, slots, sl, cu, ql, nb))
            u32, dtr, low = torch.randn(T, C, device=dev, generator=g), torch.randn(T, C, device=dev, generator=g), rnd(T, 32)
            st1 = torch.zeros(B + 1, 1, C, 16, device=dev)
            like = timer(lambda: ops.mamba1_scan(u32, dtr, dtb, A_log, low[:, :16], low[:, 16:], D, yx[:, C:], st1, slots, sl, cu, ql, bf))
            rec("rglru_scan", ph, shape, ms, T * C * 14 + B * C * 8, "mamba1_scan, 16 states", like, T * C * 12 + T * 64 + 2 * B * C * 64)
    # ---- the scan at Mamba-2's and retention's shapes
    for H, P, N, G in ((64, 64, 128, 1), (16, 128, 128, 16), (8, 512, 256, 8)):
        for B, S in ((4, 2048), (32, 1)):
            T, slots, sl, cu, ql, ph = ragged(B, S)
            st = torch.zeros(B + 1, H, N, P, device=dev)
            u = torch.randn(T, H * P + 2 * G * N, device=dev, generator=g) * 0.1
            dtr, dtb, A, decay = rnd(T, H), torch.zeros(H, device=dev), torch.zeros(H, device=dev), torch.full((H,), 0.99, device=dev)
            like = timer(lambda: ops.mamba2_scan(u, None, dtr, dtb, A, None, st, slots, sl, cu, ql, H, P, N, G))
            ms = timer(lambda: ops.mamba2_scan(u, None, None, None, None, None, st, slots, sl, cu, ql, H, P, N, G, decay))
            rec("mamba2_scan(decay): retention", ph, f"B{B} S{S} H{H} D{N} Dv{P} groups{G}", ms, u.numel() * 4 + T * H * P * 4 + 2 * B * H * N * P * 4,
                "mamba2_scan (input-dependent step, same kernel)", like)
    # ---- attention: score cap and head gate
    for H, Gk, Dh, B, S, Q in ((32, 8, 128, 4, 2048, 2048), (32, 8, 128, 64, 2048, 1), (24, 8, 64, 4, 2048, 2048), (24, 8, 64, 64, 2048, 1)):
        ps, pages = 64, B * S // 64
        kc, vc = rnd((pages + 1) * ps, 1, Gk * Dh), rnd((pages + 1) * ps, 1, Gk * Dh)
        pt = (torch.arange(pages, dtype=torch.int32, device=dev) + 1).view(B, S // ps).contiguous()
        slots, sl = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), S, dtype=torch.int32, device=dev)
        ql = torch.full((B,), Q, dtype=torch.int32, device=dev) if Q > 1 else None
        cu = None if Q == 1 else torch.arange(0, B * Q + 1, Q, dtype=torch.int32, device=dev)
        q, gh = rnd(B * Q, H, Dh), rnd(B * Q, H)
        ph, shape, keys = "prefill" if Q > 1 else "decode", f"B{B} S{S} q{Q} H{H} G{Gk} D{Dh}", sum(i + 1 for i in range(S - Q, S))
        nb, fl = q.numel() * 4 + B * S * Gk * Dh * 4, 4.0 * B * keys * H * Dh
        if Dh == 128:
            k4, v4 = kc.view(-1, Gk, Dh), vc.view(-1, Gk, Dh)
            run = lambda cap: ops.paged_attention(q, k4, v4, pt, slots, sl, cu, ql, Q, ps, Dh ** -0.5, True, -1, logit_cap=cap, num_splits=1 if Q > 1 else 4)
            ms, like = timer(lambda: ops.sigmoid_gate(run(30.0), gh, Dh)), timer(lambda: run(0.0))
            rec("capped attention on the tcgen05 kernels + sigmoid_gate", ph, shape, ms, nb + q.numel() * 4, "paged_attention (same kernels, no cap, no gate)", like, nb, fl)
            like = timer(lambda: run(30.0))
            rec("capped attention on the tcgen05 kernels + sigmoid_gate", ph, shape, ms, nb + q.numel() * 4, "paged_attention with the cap (Gemma's form)", like, nb, fl)
        else:          # three query heads per key head: the general kernel
            run = lambda cap, gate: ops.window_attention(q, kc, vc, Gk, Dh, pt, slots, sl, cu, ql, Q, ps, Dh ** -0.5, cap, -1, None, None, Dh, gate=gate)
            ms, like = timer(lambda: run(30.0, gh), iters=3), timer(lambda: run(0.0, None), iters=3)
            rec("window_attention (general kernel), cap and head gate", ph, shape, ms, nb, "window_attention, plain", like, nb, fl)
    # ---- preparations
    T, H, Gk, Dh = 8192, 32, 8, 128
    qkv = rnd(T, (H + 2 * Gk) * Dh + H)
    kc, vc = torch.zeros(T + 64, 1, Gk * Dh, device=dev, dtype=bf), torch.zeros(T + 64, 1, Gk * Dh, device=dev, dtype=bf)
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    loc, fr = pos + 64, scaled_inv_freq(Dh, 10000.0).to(dev)
    qw, kw = torch.ones(H * Dh, device=dev, dtype=bf), torch.ones(Gk * Dh, device=dev, dtype=bf)
    prep = lambda inter: ops.attention_prepare(qkv, H, Gk, Dh, Dh, pos, kc, vc, loc, qw, kw, 1e-6, fr, interleaved=inter)
    ms, like = timer(lambda: prep(True)), timer(lambda: prep(False))
    nb = T * (H + 2 * Gk) * Dh * 4
    rec("attention_prepare (projection norm, neighbouring pairs)", "any", f"T{T} H{H} G{Gk} D{Dh}", ms, nb, "attention_prepare (projection norm, half-apart pairs)", like)
    q3, k3, v3 = qkv[:, :H * Dh].clone().view(T, H, Dh), qkv[:, H * Dh:(H + Gk) * Dh].clone().view(T, Gk, Dh), qkv[:, :Gk * Dh].clone().view(T, Gk, Dh)
    cs = torch.randn(T, Dh, device=dev)
    like = timer(lambda: ops.rope_kv_write(q3, k3, v3, pos, cs, kc.view(-1, Gk, Dh), vc.view(-1, Gk, Dh), loc))
    rec("attention_prepare (projection norm, neighbouring pairs)", "any", f"T{T} H{H} G{Gk} D{Dh}", ms, nb, "rope_kv_write (table of cos / sin, no norm)", like)
    for H, D, Dv in ((16, 128, 128), (8, 256, 512)):
        m = H * (Dv + 2 * D)
        pr, fr = rnd(T, m + H * Dv), scaled_inv_freq(D, 10000.0).to(dev)
        ms = timer(lambda: ops.linear_attention_prepare(pr, H, D, Dv, pos, fr, False, D ** -0.5))
        like = timer(lambda: ops.activation(pr[:, :m], "silu", torch.float32))
        rec("linear_attention_prepare (rotation, constant on k, fp32 out)", "any", f"T{T} H{H} D{D} Dv{Dv}", ms, T * m * 6, "activation(silu) -> fp32", like)
        o, gate, w = torch.randn(T, H * Dv, device=dev), pr[:, m:], torch.ones(H * Dv, device=dev, dtype=bf)
        ms = timer(lambda: ops.grouped_rmsnorm(o, None, H, 1e-5, bf, gate, 1.0, None, "silu"))
        like = timer(lambda: ops.grouped_rmsnorm(o, w, 1, 1e-5, bf, gate))
        rec("grouped_rmsnorm (heads alone, SiLU gate)", "any", f"T{T} H{H} Dv{Dv}", ms, T * H * Dv * 8, "grouped_rmsnorm (joint, sigmoid gate)", like)
    return out


def main(sizes: str = "2048,4096") -> None:
    pk = _peaks()
    timer = _Timer()
    rows: List[dict] = []

    def put(r):
        rows.append(r)
        print(json.dumps(r), flush=True)

    for w in [int(x) for x in sizes.split(",") if x]:
        heads, ff = w // 64, 2 * w
        for name, cfg in (("surasun", _surasun_cfg(w, heads, ff)), ("resatar", _resatar_cfg(w, heads, ff))):
            extra = [_captured_decode(name, cfg, 32, 2048, 64)] if name == "surasun" else []
            for r in _engine_numbers(name, cfg, 4, 2048, 32, 8, timer) + extra:
                r["width"] = w
                put(r)
    for r in _kernel_numbers(_KernelTimer(), pk["hbm_gbs"], pk["bf16_tflops"]):
        put(r)
    worst = max((r.get("distance_ratio", 0.0) for r in rows if r["part"] == "kernel"), default=0.0)
    print(json.dumps({"metric": "hybrid_compare", "family": "surasun", "roofline": f"{pk['hbm_gbs']} GB/s, {pk['bf16_tflops']} TFLOP/s ({pk['src']})",
                      "worst_kernel_distance_ratio": worst, "rows": len(rows), "data": "synthetic", "dtype": "bf16"}), flush=True)
