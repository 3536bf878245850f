"""Mumasun: a decoder whose configuration lists its layers one by one.  A layer norms the output of its sublayers only, and the sublayers read
the stream itself:

    x <- x + norm1(mixer(x));   x <- x + norm2(ff(x))        (no second half when the layer has no feed-forward)

with the mixer ``attention``: differential grouped-query attention over short-convolved projections, unit-RMS maps, rotary positions
(YaRN-blended), chunked visibility (``layers/differential_attention.py``); and the feed-forward a mixture of ungated squared-relu experts
behind a sigmoid router whose weights, not renormalised, multiply an expert's input (``layers/moe.py`` with ``weight_input``).  Norms are RMS
norms with weights stored around zero (``1 + w``).  The embedding is normed; the head is the embedding table, its logits times a constant.

How it sits in the engine: the residual stream is fp32 on every path; ``ops.norm_add_f32`` norms a sublayer's output, adds it and emits the
stream in the GEMM dtype for the next sublayer in one kernel (and the normed embedding at the start).  Every attention layer owns a layer of
the paged pool, laid out as flat rows as wide as the widest layer needs, and an entry of the ``LayeredStatePool`` with the last projection
rows of every request.  Prompt portions, decode steps and mixed batches are the same forward: every kernel is ragged over ``cu_q`` /
``seq_lens``.  bf16 decode steps are captured into CUDA graphs when the expert sizes take the grouped tcgen05 path (no host
synchronisation).  Prefix caching is off (the convolution state has no page-aligned snapshot); tensor parallelism is not split for this family.

Checkpoint names: ``embed``, ``embed.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``q|k|v`` + ``.conv``, ``q.norm|k.norm``, ``lq1|lk1|lq2|lk2``, ``o``),
``l<i>.mlp.e<j>.{up,down}``, ``l<i>.mlp.router``, ``final.norm``; linear weights are [out, in].
"""
from __future__ import annotations

import zlib
from typing import Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..configs.model_config import ModelConfig
from ..layers.differential_attention import DifferentialAttention
from ..layers.latent_attention import yarn_inv_freq
from ..layers.moe import FusedMoE
from ..layers.window_attention import FlatCacheSpec
from ..mem_cache.memory_pool import LayeredStatePool
from ..model_executor.forward_batch import ForwardBatch
from ..ops import moe_ops
from ..parallel.parallel_state import get_pp_group, get_tp_group
from .llama import _DT
from .rirotar import ZeroCentredNorm
from .zaparax import _CacheLayer


class SigmoidInputMoE(nn.Module):
    """ungated squared-relu experts behind a sigmoid router; the chosen scores multiply the experts' inputs.  Expert widths are padded to a
    multiple of 32 with zero rows (a zero row of the up-projection contributes max(0, 0)^2 = 0) so that any size takes the grouped kernels."""

    def __init__(self, width: int, mlp: dict, dtype, layer_id: int):
        super().__init__()
        r = mlp["router"]
        self.E, self.top, self.ff = int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"])
        self.router = nn.Parameter(torch.zeros(self.E, width, dtype=dtype), requires_grad=False)
        self.experts = FusedMoE(self.E, self.top, width, -(-self.ff // 32) * 32, dtype, False, 1, None, layer_id, gated=False)
        self.experts.act, self.experts.weight_input = ("relu2",), True

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        if leaf == "router":
            self.router.data.copy_(w)
            return True
        head, _, proj = leaf.partition(".")
        if not (head[:1] == "e" and head[1:].isdigit() and int(head[1:]) < self.E and proj in ("up", "down")):
            return False
        ex, gap = self.experts, self.experts.inter_local - self.ff
        if gap:
            w = torch.nn.functional.pad(w, (0, 0, 0, gap) if proj == "up" else (0, gap))
        ex.weight_loader(ex.w2 if proj == "down" else ex.w13, w, int(head[1:]), "w2" if proj == "down" else "w3")
        return True

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        w, ids = moe_ops.sigmoid_route(ops.linear_f32(h, self.router), self.top)          # fp32 logits of the (possibly bf16-rounded) input
        y = self.experts.forward_routed(h, w, ids)
        return y.resolve() if hasattr(y, "resolve") else y


class MumasunBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: dict, idx: int, dtype):
        super().__init__()
        W, m, eps = cfg.hidden_size, spec["mixer"], cfg.rms_norm_eps
        if spec["type"] != "attention":
            raise ValueError(f"Mumasun: unknown mixer type {spec['type']!r} in layer {idx}")
        rot = m.get("rot") or {}
        rotary = (int(rot["dims"]), *yarn_inv_freq(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))) if rot.get("dims") else None
        self.mix = DifferentialAttention(W, int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m.get("vdim", m["dim"])), m.get("scale"),
                                         float(m["diff"]), eps, dtype, taps=int(m.get("conv") or 1), rotary=rotary,
                                         chunk=int((m.get("mask") or {}).get("size") or 0))
        self.norm1 = ZeroCentredNorm(W, dtype)
        mlp = spec.get("mlp")
        self.norm2 = self.mlp = None
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"Mumasun: unknown feed-forward kind {mlp.get('kind')!r} in layer {idx}")
            self.norm2 = ZeroCentredNorm(W, dtype)
            self.mlp = SigmoidInputMoE(W, mlp, dtype, idx)


class MumasunForCausalLM(nn.Module):
    disable_radix_cache = True           # convolution state per request: no page-aligned prefix to share

    def __init__(self, cfg: ModelConfig, quant_name: Optional[str] = None, device="cpu"):
        super().__init__()
        assert get_tp_group().world_size == 1 and get_pp_group().world_size == 1, "Mumasun runs on one rank"
        assert cfg.hybrid and cfg.hybrid.get("layers") is not None, "Mumasun needs the per-layer list of its configuration"
        self.cfg = cfg
        dtype = _DT[cfg.dtype]
        self.dtype = dtype
        specs = cfg.hybrid["layers"]
        self.logit_scale = float(cfg.hybrid.get("logit_scale", 1.0))
        bb = nn.Module()
        bb.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype)          # also the output head
        bb.embed_tokens.weight.requires_grad_(False)
        bb.embed_norm = ZeroCentredNorm(cfg.hidden_size, dtype)
        bb.all_layers = nn.ModuleList([MumasunBlock(cfg, s, i, dtype) for i, s in enumerate(specs)])
        mixers = [b.mix for b in bb.all_layers]
        cache_width = -(-max([m.cache_width for m in mixers] or [0]) // 8) * 8          # rows in multiples of 16 bytes (tensor maps over the pool)
        heads = max([m.query_heads for m in mixers] or [1])                              # sizes the split-KV workspace of captured decode steps
        # ``layers``: what the runner sizes the paged pool from (one entry per attention layer)
        bb.layers = [_CacheLayer(FlatCacheSpec(heads, cache_width, i, m.scale, -1)) for i, m in enumerate(mixers)]
        bb.norm = ZeroCentredNorm(cfg.hidden_size, dtype)
        self.model = bb
        # decode steps are captured when nothing in them needs the host: bf16, attention on the native kernels, experts on the grouped tcgen05 path
        self.supports_cuda_graph = dtype == torch.bfloat16 and cfg.hidden_size % 32 == 0 and all(
            max(m.MAPS * m.D, m.Dv) <= 256 and m.taps <= 16 for m in mixers) and all(b.mlp is None or (b.mlp.E <= 512 and b.mlp.top <= 32) for b in bb.all_layers)
        self.layer_tap = None            # callable(layer index, fp32 residual [T, width]) after every layer (debugging / tests)
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False          # fp32 serving means fp32 products

    # ---- forward: fp32 residual stream; a sublayer's output norm, the residual add and the cast for the next sublayer are one kernel
    def forward(self, fb: ForwardBatch, inputs_embeds=None):
        m, eps, dt = self.model, self.cfg.rms_norm_eps, self.dtype
        if inputs_embeds is None:
            # decode reads every request's input token from the device-side token buffer (where sampling leaves it)
            ids = fb.input_ids if fb.input_ids is not None else fb.next_token_buf[fb.req_slots.long()]
            x, h = ops.norm_add_f32(None, m.embed_tokens.weight, m.embed_norm.weight, eps, True, dt, ids)
        else:
            x, h = ops.norm_add_f32(torch.zeros(inputs_embeds.shape, dtype=torch.float32, device=inputs_embeds.device), inputs_embeds.contiguous(),
                                    m.embed_norm.weight, eps, True, dt)
        subs = []                        # (sublayer, its output norm, layer index when it ends a layer)
        for i, blk in enumerate(m.all_layers):
            subs.append((lambda h, blk=blk, i=i: blk.mix(h, fb, i, i), blk.norm1, i if blk.mlp is None else -1))
            if blk.mlp is not None:
                subs.append((blk.mlp, blk.norm2, i))
        for n, (sub, norm, ends) in enumerate(subs):
            y = sub(h)
            if n + 1 < len(subs) or self.layer_tap is not None:
                x, h = ops.norm_add_f32(x, y, norm.weight, eps, True, dt)
                if ends >= 0 and self.layer_tap is not None:
                    self.layer_tap(ends, x)
            else:                        # the last sublayer: its update and the model's final norm in one kernel
                return ops.add_rmsnorm_f32(x, y, m.norm.weight, eps, True, dt, norm.weight)
        return ops.add_rmsnorm_f32(x, None, m.norm.weight, eps, True, dt)

    def compute_logits(self, hidden: torch.Tensor, key: str = "logits") -> torch.Tensor:
        z = ops.linear_f32(hidden, self.model.embed_tokens.weight)
        return z.mul_(self.logit_scale) if self.logit_scale != 1.0 else z

    # ---- convolution state
    def make_mamba_pool(self, slots: int, device) -> Optional[LayeredStatePool]:
        geo = [b.mix.state_geometry() for b in self.model.all_layers]
        return LayeredStatePool(slots, geo, self.dtype, device) if geo else None

    # ---- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> List[str]:
        loaded = []
        m = self.model
        plain = {"embed": m.embed_tokens, "embed.norm": m.embed_norm, "final.norm": m.norm}
        for name, w in weights:
            ok = False
            if name in plain:
                plain[name].weight.data.copy_(w)
                ok = True
            elif name[:1] == "l" and "." in name and name[1:name.index(".")].isdigit():
                i, rest = int(name[1:name.index(".")]), name[name.index(".") + 1:]
                if i < len(m.all_layers):
                    blk = m.all_layers[i]
                    if rest in ("norm1", "norm2") and getattr(blk, rest) is not None:
                        getattr(blk, rest).weight.data.copy_(w)
                        ok = True
                    elif rest.startswith("mix."):
                        ok = blk.mix.load(rest[4:], w)
                    elif rest.startswith("mlp.") and blk.mlp is not None:
                        ok = blk.mlp.load(rest[4:], w)
            if ok:
                loaded.append(name)
        return loaded

    @staticmethod
    def dummy_checkpoint(cfg: ModelConfig, device, dtype, seed: int = 0, scale: float = 0.02):
        """random tensors under the checkpoint names (name-seeded), scaled so that activations stay O(1) through many layers"""
        def rnd(name: str, *shape: int, s: float = 1.0, off: float = 0.0) -> torch.Tensor:
            g = torch.Generator(device="cpu").manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
            return (torch.randn(*shape, generator=g) * s + off).to(dtype)

        lin = lambda name, o, i, s=1.0: rnd(name, o, i, s=s * i ** -0.5)
        W = cfg.hidden_size
        yield "embed", rnd("embed", cfg.vocab_size, W, s=W ** -0.5)
        yield "embed.norm", rnd("embed.norm", W, s=0.1)
        for i, sp in enumerate(cfg.hybrid["layers"]):
            p, m = f"l{i}.", sp["mixer"]
            H, D = int(m["heads"]), int(m["dim"])
            G, Dv, taps = int(m.get("kv_heads", H)), int(m.get("vdim", D)), int(m.get("conv") or 1)
            q = p + "mix."
            for nm, n in (("q", 2 * H * D), ("k", 2 * G * D), ("v", G * Dv)):
                yield q + nm, lin(q + nm, n, W)
                yield q + nm + ".conv", rnd(q + nm + ".conv", n, taps, s=taps ** -0.5)
            for nm in ("q.norm", "k.norm"):
                yield q + nm, rnd(q + nm, D, s=0.1, off=1.0)
            for nm in ("lq1", "lk1", "lq2", "lk2"):
                yield q + nm, rnd(q + nm, D, s=0.5 * D ** -0.25)
            yield q + "o", lin(q + "o", W, H * Dv)
            yield p + "norm1", rnd(p + "norm1", W, s=0.1, off=-0.5)
            mlp = sp.get("mlp")
            if not mlp:
                continue
            E, ff = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            for e in range(E):
                yield p + f"mlp.e{e}.up", lin(p + f"u{e}", ff, W)
                yield p + f"mlp.e{e}.down", lin(p + f"d{e}", W, ff)
            yield p + "mlp.router", lin(p + "r", E, W)
            yield p + "norm2", rnd(p + "norm2", W, s=0.1, off=-0.5)
        yield "final.norm", rnd("fn", W, s=0.1)
