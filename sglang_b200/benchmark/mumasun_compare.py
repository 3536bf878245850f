"""Mumasun beside the closest existing family at equal size (``python bench.py --hybrid-compare --hybrid-family mumasun``).

Two parts, random weights, one GPU:

1. **engine**: prefill and decode throughput of a four-layer Mumasun slice (differential attention with two 64-wide maps per head over 128-wide
   values, chunks of 8192 positions, three taps; 32 experts, two per token) and of a Qwen3-MoE slice of the same width with as many query
   and key heads of 128 (so that the projections and the cache rows have the same sizes), 32 gated experts of two thirds of the width
   (as many expert weights per token), both through ``Scheduler.replay_step`` (the serving step, eager), and decode once more through
   ``Engine.generate`` with captured steps.
2. **kernels**: each new or extended kernel beside the like op of the closest model on the same shapes: differential attention on the tcgen05
   kernels (and with chunks of 1024) vs plain attention on them; the general kernel (fp32 serving, other group sizes) in its differential
   and its plain form; ``conv_attention_prepare`` vs the q / k norms + ``rope_kv_write`` it stands in for; the expert block (relu2, weighted
   inputs) vs the SwiGLU expert block; ``moe_sigmoid_route`` vs ``moe_topk_softmax``; the fp32-output router product vs the bf16 one;
   ``norm_add_f32`` vs ``postnorm_add_rmsnorm_f32`` and vs the bf16 ``fused_add_rmsnorm``.
   Roofline: algorithmic bytes over the measured copy bandwidth; FLOPs over the measured bf16 GEMM rate where ``bound`` says tensor.

Timing: CUDA events on the launching stream, >= 3 warm-ups, an L2 flush (a 256 MB write) between timed iterations.
Prints one JSON line per measurement and a closing summary line.
"""
from __future__ import annotations

import json
import time
from typing import List

import torch

from .hybrid_compare import _engine_numbers, _peaks, _Timer


def _mumasun_cfg(width: int, heads: int, ff: int, experts: int = 32, top: int = 2) -> dict:
    attn = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 64, "vdim": 128, "scale": 0.125, "conv": 3, "diff": 0.4, "mask": {"size": 8192},
            "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {"architecture": "Mumasun", "width": width, "vocab": 32000, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [{"type": "attention", "mixer": attn, "mlp": mlp}] * 4}


def _qwen3_moe_cfg(width: int, heads: int, ff: int, experts: int = 32, top: int = 2) -> dict:
    return {"architectures": ["Qwen3MoeForCausalLM"], "hidden_size": width, "num_hidden_layers": 4, "num_attention_heads": heads,
            "num_key_value_heads": max(1, heads // 8), "head_dim": 128, "vocab_size": 32000, "rms_norm_eps": 1e-6, "intermediate_size": ff,
            "num_experts": experts, "num_experts_per_tok": top, "moe_intermediate_size": 2 * ff // 3, "decoder_sparse_step": 1, "mlp_only_layers": [],
            "norm_topk_prob": True, "max_position_embeddings": 32768, "rope_theta": 10000.0, "tie_word_embeddings": True}


def _captured_decode(name: str, cfg: dict, B: int, S: int, steps: int) -> dict:
    """decode rate of ``Engine.generate`` with captured steps: the time of ``steps`` more tokens per request, wall clock"""
    import os
    import tempfile

    import numpy as np

    import sglang_b200 as sgl

    d = tempfile.mkdtemp(prefix="hybrid_cmp_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    eng = sgl.Engine(model_path=d, load_format="dummy", skip_tokenizer_init=True, page_size=64, max_total_tokens=B * (S + 2 * steps + 64) + 4096,
                     max_running_requests=B, context_length=8192, disable_radix_cache=True, cuda_graph_bs=[B], log_level="warning")
    rng = np.random.default_rng(0)
    prompts = [rng.integers(0, 32000, S).tolist() for _ in range(B)]

    def run(n):
        torch.cuda.synchronize()
        t = time.perf_counter()
        eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": n, "temperature": 0, "ignore_eos": True})
        return time.perf_counter() - t

    run(steps)
    t1, t2 = min(run(8) for _ in range(3)), min(run(8 + steps) for _ in range(3))
    eng.shutdown()
    del eng
    torch.cuda.empty_cache()
    ms = (t2 - t1) / steps * 1e3
    return {"part": "engine", "model": name, "phase": "decode (captured steps, Engine.generate)", "batch": B, "context": S, "ms_per_step": round(ms, 3),
            "tokens_per_s": round(B / ms * 1e3)}


def _kernel_numbers(timer: _Timer, hbm_gbs: float, tflops: float) -> List[dict]:
    from .. import ops
    from ..layers.latent_attention import yarn_inv_freq
    from ..ops import moe_ops, torch_ref

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

    # ---- attention: H heads of two 64-wide maps over 128-wide values, beside H plain 128-wide heads over the same cache rows
    H, G, ps, scale = 32, 4, 64, 0.125
    diff = (0.7, 0.6, 1e-6)
    for B, S, Q in ((4, 2048, 2048), (64, 2048, 1), (64, 8192, 1)):
        pages = B * S // ps
        kc, vc = rnd((pages + 1) * ps, 1, G * 128), rnd((pages + 1) * ps, 1, G * 128)
        pt = (torch.arange(pages, dtype=torch.int32, device=dev) + 1).view(B, S // ps).contiguous()
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        sl = torch.full((B,), S, dtype=torch.int32, device=dev)
        ql = torch.full((B,), Q, dtype=torch.int32, device=dev) if Q > 1 else None
        cu = None if Q == 1 else torch.arange(0, B * Q + 1, Q, dtype=torch.int32, device=dev)
        q1, q2 = rnd(B * Q, H, 128), torch.zeros(B * Q, H, 2, 2, 64, device=dev, dtype=bf)
        q2[:, :, 0, 0], q2[:, :, 1, 1] = q1[:, :, :64], q1[:, :, 64:]
        q2 = q2.view(B * Q, 2 * H, 128)
        k4, v4 = kc.view(-1, G, 128), vc.view(-1, G, 128)
        ns = 1
        ph = "prefill" if Q > 1 else "decode"
        shape = f"B{B} S{S} q{Q} H{H} G{G} dim2x64 vdim128"
        kv = B * S * G * 256 * 2
        for chunk in (0, 1024):
            lo = lambda i: i // chunk * chunk if chunk else 0
            keys = sum(i + 1 - lo(i) for i in range(S - Q, S))
            kvb = kv if Q > 1 else B * (S - lo(S - 1)) * G * 512
            ms = timer(lambda: ops.paged_attention(q2, k4, v4, pt, slots, sl, cu, ql, Q, ps, scale, num_splits=ns, chunk=chunk, diff=diff, diff_dv=128))
            kw = dict(window=chunk) if chunk else {}
            like = timer(lambda: ops.paged_attention(q1, k4, v4, pt, slots, sl, cu, ql, Q, ps, 128 ** -0.5, num_splits=ns, **kw))
            wkeys = sum(min(i + 1, chunk) for i in range(S - Q, S)) if chunk else keys
            rec("differential attention on the tcgen05 kernels" + (f", chunks of {chunk}" if chunk else ""), ph, shape, ms, kvb + q1.numel() * 4,
                "paged_attention (plain, same heads and cache)" + (f", window {chunk}" if chunk else ""), like, kvb + q1.numel() * 4,
                2.0 * B * keys * H * 2 * (64 + 128), 2.0 * B * wkeys * H * 256)
        if Q > 1 or S == 2048:
            nb = kv + q1.numel() * 4
            keys = sum(i + 1 for i in range(S - Q, S))
            ms = timer(lambda: ops.window_attention(q2, kc, vc, G, 128, pt, slots, sl, cu, ql, Q, ps, scale, dim=128, diff=diff), iters=3)
            like = timer(lambda: ops.window_attention(q1, kc, vc, G, 128, pt, slots, sl, cu, ql, Q, ps, scale, dim=128), iters=3)
            rec("window_attention (general kernel), differential", ph, shape, ms, nb, "window_attention, plain", like, nb, 2.0 * B * keys * H * 2 * 192,
                2.0 * B * keys * H * 256)
    # ---- preparation: convolution, norms, rotation, cache write and state, beside norms + rope_kv_write
    f, mult = yarn_inv_freq(64, 10000.0, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    f = f.to(dev)
    C = (H + G) * 128 + G * 128
    cos_sin = torch_ref.build_cos_sin_cache(128, 8192, 10000.0, None, 128).to(dev)
    nw, n64 = torch.ones(128, device=dev, dtype=bf), torch.ones(64, device=dev, dtype=bf)
    w = rnd(C, 3, sc=0.5)
    for B, S in ((4, 2048), (64, 1)):
        T = B * S
        x = rnd(T, C)
        kc, vc = torch.zeros(T + 64, 1, G * 128, device=dev, dtype=bf), torch.zeros(T + 64, 1, G * 128, device=dev, dtype=bf)
        state = torch.zeros(B + 1, C, 2, device=dev, dtype=bf)
        pos = torch.arange(T, dtype=torch.int32, device=dev) % S + (0 if S > 1 else 2000)
        loc = torch.arange(T, dtype=torch.int32, device=dev) + 64
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        sl = torch.full((B,), S if S > 1 else 2001, dtype=torch.int32, device=dev)
        cu = torch.arange(0, T + 1, S, dtype=torch.int32, device=dev) if S > 1 else None
        ms = timer(lambda: ops.conv_attention_prepare(x, H, G, 2, 64, 128, w, state, pos, cu, slots, sl, n64, n64, 1e-6, f, mult, kc, vc, loc, 128))
        qs, ks = H * 128, G * 128
        k3c, v3c = kc.view(-1, G, 128), vc.view(-1, G, 128)

        def norms_rope():
            q = ops.rmsnorm(x[:, :qs].reshape(T * H, 128), nw, 1e-6).view(T, H, 128)
            k = ops.rmsnorm(x[:, qs:qs + ks].reshape(T * G, 128), nw, 1e-6).view(T, G, 128)
            ops.rope_kv_write(q, k, x[:, qs + ks:].view(T, G, 128), pos, cos_sin, k3c, v3c, loc)

        like = timer(norms_rope)
        rec("conv_attention_prepare (convolution, map norms, rotation, cache and state)", "prefill" if S > 1 else "decode", f"T{T} H{H} G{G} taps3", ms,
            T * (C + 2 * qs + 2 * ks) * 2 + B * C * 2 * 2 * (1 if S > 1 else 2), "q norm + k norm + rope_kv_write", like, T * C * 2 * 2)
    # ---- experts and router
    for W, ff in ((2048, 1152), (4096, 2304)):
        E, K, I = 32, 2, 2 * ff // 3
        w1, w2 = rnd(E, ff, W, sc=W ** -0.5), rnd(E, W, ff, sc=ff ** -0.5)
        a13, a2 = rnd(E, 2 * I, W, sc=W ** -0.5), rnd(E, W, I, sc=I ** -0.5)
        for T in (8192, 64):
            h = rnd(T, W)
            wr = rnd(E, W, sc=W ** -0.5)
            z = ops.linear_f32(h, wr)
            rw, ids = moe_ops.sigmoid_route(z, K)
            hit = int(torch.unique(ids).numel())
            ms = timer(lambda: moe_ops.fused_moe(h, w1, w2, rw, ids, 0, ("relu2",), True))
            like = timer(lambda: moe_ops.fused_moe(h, a13, a2, rw, ids, 0))
            nb = hit * 2 * W * ff * 2 + T * W * 4
            rec("expert block (relu2, weighted inputs)", "prefill" if T > 64 else "decode", f"T{T} W{W} ff{ff} E{E} top{K}", ms, nb, f"expert block (SwiGLU, ff {I})", like, nb,
                2.0 * T * K * 2 * W * ff)
            ms = timer(lambda: moe_ops.sigmoid_route(z, K))
            zb = z.to(bf)
            like = timer(lambda: moe_ops.topk_softmax(zb, K))
            rec("moe_sigmoid_route", "any", f"T{T} E{E} top{K}", ms, T * (E * 4 + K * 8), "moe_topk_softmax (bf16 logits)", like, T * (E * 2 + K * 8))
            ms = timer(lambda: ops.linear_f32(h, wr))
            like = timer(lambda: ops.linear(h, wr))
            rec("router product with fp32 output (cuBLAS)", "any", f"T{T} W{W} E{E}", ms, T * W * 2 + E * W * 2 + T * E * 4, "ops.linear (bf16 output)", like,
                T * W * 2 + E * W * 2 + T * E * 2)
    # ---- residual
    for T in (8192, 64):
        W = 4096
        res, d = torch.randn(T, W, device=dev), rnd(T, W)
        rb, wt = rnd(T, W), torch.zeros(W, device=dev, dtype=bf)
        ms = timer(lambda: ops.norm_add_f32(res, d, wt, 1e-6, True, bf))
        like = timer(lambda: ops.add_rmsnorm_f32(res, d, wt, 1e-6, True, bf, wt))
        rec("norm_add_f32", "any", f"T{T} W{W}", ms, T * W * 12, "postnorm_add_rmsnorm_f32 (one more norm)", like, T * W * 12)
        like = timer(lambda: ops.fused_add_rmsnorm(d, rb, wt, 1e-6))
        rec("norm_add_f32", "any", f"T{T} W{W}", ms, T * W * 12, "fused_add_rmsnorm (bf16 stream)", like, T * W * 8)
    return out


def main(sizes: str = "2048,4096") -> None:
    pk = _peaks()
    timer = _Timer()
    rows: List[dict] = []

    def put(r):
        rows.append(r)
        print(json.dumps(r), flush=True)

    for w in [int(x) for x in sizes.split(",") if x]:
        heads, ff = w // 128, 9 * w // 16
        for name, cfg in (("mumasun", _mumasun_cfg(w, heads, ff)), ("qwen3_moe", _qwen3_moe_cfg(w, heads, ff))):
            for r in _engine_numbers(name, cfg, 4, 2048, 32, 8, timer) + [_captured_decode(name, cfg, 32, 2048, 64)]:
                r["width"] = w
                put(r)
    for r in _kernel_numbers(timer, pk["hbm_gbs"], pk["bf16_tflops"]):
        put(r)
    worst = max((r.get("distance_ratio", 0.0) for r in rows if r["part"] == "kernel"), default=0.0)
    print(json.dumps({"metric": "hybrid_compare", "family": "mumasun", "roofline": f"{pk['hbm_gbs']} GB/s, {pk['bf16_tflops']} TFLOP/s ({pk['src']})",
                      "worst_kernel_distance_ratio": worst, "rows": len(rows), "data": "synthetic", "dtype": "bf16"}), flush=True)
