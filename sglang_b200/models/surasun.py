"""Surasun: a decoder whose configuration lists its layers one by one and whose residual is ``streams`` parallel streams (hyper-connections,
``layers/hyper_connections.py``).  A sublayer reads the layer norm (weight, no bias) of a weighted sum of the streams; its output, times a
constant, is added to every stream while the streams are mixed.  The sublayers of a layer are its mixer, one of

* ``mamba2``:   Mamba-2 state-space mixer with a gated, group-wise RMS-normed read-out (``layers/mamba2_scan.py``);
* ``parallel``: causal grouped-query attention (projection biases, q / k normed over their whole projection, partial rotation of neighbouring
  coordinates, capped scores, one sigmoid output gate per head; ``layers/gated_attention.py``) beside retention (rotated q / k, a constant
  decay per head, heads normed alone, SiLU gate; ``layers/linear_attention.py``), summed with two constants (``layers/parallel_mixer.py``);
* ``rglru``:    gated linear recurrence behind a short convolution (``layers/rglru.py``);

and, where it has one, a SiLU-GLU feed-forward.  The streams' sum passes a last layer norm; the head is the embedding table.

How it sits in the engine: the streams are fp32 on every path; ``ops.stream_mix_norm`` applies a sublayer's update to all streams and emits the
next sublayer's normed input in the GEMM dtype in one kernel (the first update reads the embedding row itself, the last one stores no
streams).  A parallel layer owns a layer of the paged pool (flat rows as wide as the widest layer needs) and an entry of the
``LayeredStatePool``; a recurrent layer owns an entry of the latter (state, convolution history), indexed by request slot.  Prompt portions,
decode steps and mixed batches are the same forward: every kernel is ragged over ``cu_q`` / ``seq_lens``.  bf16 decode steps are captured into
CUDA graphs.  Prefix caching is off (recurrent state has no page-aligned snapshot); tensor parallelism is not split for this family.

Checkpoint names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.hc1.*|hc2.*`` (``in``, ``out``, ``mix``), ``l<i>.mix.*`` (``left.*`` / ``right.*`` under a parallel
mixer), ``l<i>.mlp.{gate,up,down}``, ``final.norm``; linear weights are [out, in].
"""
from __future__ import annotations

import zlib
from typing import Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..configs.model_config import ModelConfig
from ..layers.gated_attention import GatedAttention, scaled_inv_freq
from ..layers.hyper_connections import StreamMix
from ..layers.linear_attention import DecayLinearAttention
from ..layers.mamba2_scan import Mamba2ScanMixer
from ..layers.parallel_mixer import ParallelMixer
from ..layers.rglru import RGLRUMixer
from ..layers.window_attention import FlatCacheSpec
from ..mem_cache.memory_pool import LayeredStatePool
from ..model_executor.forward_batch import ForwardBatch
from ..parallel.parallel_state import get_pp_group, get_tp_group
from .llama import _DT
from .zaparax import SiluGLU, _CacheLayer


class LayerNormWeight(nn.Module):
    """the weight of a layer norm without bias; the norm itself runs fused with the stream update (``ops.stream_mix_norm``)"""

    def __init__(self, width: int, dtype):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(width, dtype=dtype), requires_grad=False)


def _rotary(rot: Optional[dict]):
    return (int(rot["dims"]), scaled_inv_freq(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))) if rot and rot.get("dims") else None


def parallel_mixer(width: int, m: dict, eps: float, dtype) -> ParallelMixer:
    """``left_scale * attention + right_scale * retention`` on the same input"""
    a, b = m["left"], m["right"]
    left = GatedAttention(width, int(a["heads"]), int(a.get("kv_heads", a["heads"])), int(a["dim"]), int(a.get("vdim", a["dim"])), a.get("scale"), eps, dtype,
                          bias=True, out_bias=False, qk_norm=True, rotary=_rotary(a.get("rot")), interleaved=True, softcap=float(a.get("softcap") or 0.0),
                          gate="head", own_projection=False)
    dim = int(b["dim"])
    right = DecayLinearAttention(width, int(b["heads"]), dim, int(b.get("vdim", dim)), b["decay"], eps, dtype, own_projection=False, act=None,
                                 rotary=_rotary(b.get("rot")), k_scale=dim ** -0.5, norm="head", gate_act="silu")
    return ParallelMixer(width, left, right, float(m.get("left_scale", 1.0)), float(m.get("right_scale", 1.0)), dtype)


class SurasunBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: dict, idx: int, dtype, streams: int):
        super().__init__()
        W, m, eps = cfg.hidden_size, spec["mixer"], cfg.rms_norm_eps
        kind = spec["type"]
        self.kind = kind
        if kind == "mamba2":
            self.mix = Mamba2ScanMixer(W, int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m.get("groups", 1)), int(m.get("conv") or 1),
                                       int(m.get("norm_groups", 1)), eps, dtype)
        elif kind == "parallel":
            self.mix = parallel_mixer(W, m, eps, dtype)
        elif kind == "rglru":
            self.mix = RGLRUMixer(W, int(m["width"]), int(m["blocks"]), int(m.get("conv") or 1), dtype)
        else:
            raise ValueError(f"Surasun: unknown mixer type {kind!r} in layer {idx}")
        self.norm1, self.hc1 = LayerNormWeight(W, dtype), StreamMix(streams)
        mlp = spec.get("mlp")
        self.norm2 = self.hc2 = self.mlp = None
        if mlp:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"Surasun: unknown feed-forward kind {mlp.get('kind')!r} in layer {idx}")
            self.norm2, self.hc2, self.mlp = LayerNormWeight(W, dtype), StreamMix(streams), SiluGLU(W, int(mlp["ff"]), dtype)

    def attention(self) -> Optional[GatedAttention]:
        return self.mix.left if self.kind == "parallel" else None

    def state_geometry(self):
        return (self.mix.right if self.kind == "parallel" else self.mix).state_geometry()

    def capturable(self) -> bool:
        """whether a decode step of this layer stays on the native kernels (no host synchronisation)"""
        if self.kind == "parallel":
            a, r = self.mix.left, self.mix.right
            return max(a.D, a.Dv) <= 256 and r.D <= 1024
        return self.mix.taps <= 8 and (self.kind == "rglru" or self.mix.N <= 1024)


class SurasunForCausalLM(nn.Module):
    disable_radix_cache = True           # recurrent state per request: no page-aligned prefix to share

    def __init__(self, cfg: ModelConfig, quant_name: Optional[str] = None, device="cpu"):
        super().__init__()
        assert get_tp_group().world_size == 1 and get_pp_group().world_size == 1, "Surasun runs on one rank"
        assert cfg.hybrid and cfg.hybrid.get("layers") is not None, "Surasun needs the per-layer list of its configuration"
        self.cfg = cfg
        dtype = _DT[cfg.dtype]
        self.dtype = dtype
        self.streams, self.mult = int(cfg.hybrid["streams"]), float(cfg.hybrid["residual_mult"])
        bb = nn.Module()
        bb.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype)          # also the output head
        bb.embed_tokens.weight.requires_grad_(False)
        bb.all_layers = nn.ModuleList([SurasunBlock(cfg, s, i, dtype, self.streams) for i, s in enumerate(cfg.hybrid["layers"])])
        # bf16 layers whose heads fit the tcgen05 kernels lay them out 128 columns wide in the leading columns of the pool's rows (the widest layer's width)
        attn = [b.attention() for b in bb.all_layers if b.attention() is not None]
        for m in attn:
            if m.wants_padding(dtype):
                m.pad = 128
        cache_width = -(-max([m.cache_width for m in attn] or [0]) // 8) * 8          # rows in multiples of 16 bytes (tensor maps over the pool)
        heads = max([m.H for m in attn] or [1])                                        # sizes the split-KV workspace of captured decode steps
        self.cache_of: List[int] = []      # per block: index of its layer in the paged pool, -1 where it has none
        bb.layers = []                     # what the runner sizes the paged pool from (one entry per attention layer)
        for blk in bb.all_layers:
            a = blk.attention()
            self.cache_of.append(-1 if a is None else len(bb.layers))
            if a is not None:
                bb.layers.append(_CacheLayer(FlatCacheSpec(heads, cache_width, len(bb.layers), a.scale, -1)))
        bb.norm = LayerNormWeight(cfg.hidden_size, dtype)
        self.model = bb
        self.supports_cuda_graph = dtype == torch.bfloat16 and bool(attn) and self.streams <= 16 and all(b.capturable() for b in bb.all_layers)
        self.layer_tap = None            # callable(layer index, fp32 sum of the streams [T, width]) after every layer (debugging / tests)
        self._coef = None
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False          # fp32 serving means fp32 products

    def _coefs(self, device) -> List[torch.Tensor]:
        """the stream numbers of every update: the sublayer before it and the one behind it"""
        if self._coef is None or self._coef[0].device != torch.device(device):
            hcs = [hc for blk in self.model.all_layers for hc in (blk.hc1, blk.hc2) if hc is not None]
            self._coef = [StreamMix.pack(p, n, self.mult, self.streams, device) for p, n in zip([None] + hcs, hcs + [None])]
        return self._coef

    # ---- forward: fp32 streams; a sublayer's update of all streams, the next sublayer's weighted sum and its norm are one kernel
    def forward(self, fb: ForwardBatch, inputs_embeds=None):
        m, eps, dt, S = self.model, self.cfg.rms_norm_eps, self.dtype, self.streams
        table, ids, x = m.embed_tokens.weight, None, None
        if inputs_embeds is not None:
            x = inputs_embeds.float()[:, None, :].expand(-1, S, -1).contiguous()
        else:                              # decode reads every request's input token from the device-side token buffer (where sampling leaves it)
            ids = fb.input_ids if fb.input_ids is not None else fb.next_token_buf[fb.req_slots.long()]
        coef = self._coefs(table.device)
        y, n = None, 0
        for i, blk in enumerate(m.all_layers):
            x, h = ops.stream_mix_norm(x, y, coef[n], S, blk.norm1.weight, eps, dt, True, table, ids, keep=n > 0 or x is not None)
            if self.layer_tap is not None and i > 0:
                self.layer_tap(i - 1, x.sum(1))
            n += 1
            if blk.kind == "parallel":
                y = blk.mix(h, fb, self.cache_of[i], i)
            else:
                y = blk.mix(h, fb, i)
            if blk.mlp is not None:
                x, h = ops.stream_mix_norm(x, y, coef[n], S, blk.norm2.weight, eps, dt, True, table, ids)
                y, n = blk.mlp(h), n + 1
        x, h = ops.stream_mix_norm(x, y, coef[n], S, m.norm.weight, eps, dt, True, table, ids, keep=self.layer_tap is not None)
        if self.layer_tap is not None and len(m.all_layers):
            self.layer_tap(len(m.all_layers) - 1, x.sum(1))
        return h

    def compute_logits(self, hidden: torch.Tensor, key: str = "logits") -> torch.Tensor:
        return ops.linear_f32(hidden, self.model.embed_tokens.weight)

    # ---- recurrent state: every layer has some
    def make_mamba_pool(self, slots: int, device) -> Optional[LayeredStatePool]:
        geo = [b.state_geometry() for b in self.model.all_layers]
        return LayeredStatePool(slots, geo, self.dtype, device) if geo else None

    # ---- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> List[str]:
        loaded = []
        m = self.model
        plain = {"embed": m.embed_tokens, "final.norm": m.norm}
        for name, w in weights:
            ok = False
            if name in plain:
                plain[name].weight.data.copy_(w)
                ok = True
            elif name[:1] == "l" and "." in name and name[1:name.index(".")].isdigit():
                i, rest = int(name[1:name.index(".")]), name[name.index(".") + 1:]
                if i < len(m.all_layers):
                    blk = m.all_layers[i]
                    head, _, leaf = rest.partition(".")
                    part = getattr(blk, head) if head in ("norm1", "norm2", "hc1", "hc2", "mix", "mlp") else None
                    if part is not None and isinstance(part, LayerNormWeight):
                        part.weight.data.copy_(w)
                        ok = True
                    elif part is not None:
                        ok = part.load(leaf, w)
            if ok:
                loaded.append(name)
        self._coef = None
        return loaded

    @staticmethod
    def dummy_checkpoint(cfg: ModelConfig, device, dtype, seed: int = 0, scale: float = 0.02):
        """random tensors under the checkpoint names (name-seeded), scaled so that activations stay O(1) through many layers"""
        def rnd(name: str, *shape: int, s: float = 1.0, off: float = 0.0) -> torch.Tensor:
            g = torch.Generator(device="cpu").manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
            return (torch.randn(*shape, generator=g) * s + off).to(dtype)

        lin = lambda name, o, i, s=1.0: rnd(name, o, i, s=s * i ** -0.5)
        W, S = cfg.hidden_size, int(cfg.hybrid["streams"])
        yield "embed", rnd("embed", cfg.vocab_size, W, s=W ** -0.5)
        for i, sp in enumerate(cfg.hybrid["layers"]):
            p, m, kind = f"l{i}.", sp["mixer"], sp["type"]
            q = p + "mix."
            if kind == "mamba2":
                H, P, N, G, taps = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m.get("groups", 1)), int(m.get("conv") or 1)
                cd = H * P + 2 * G * N
                yield q + "in", lin(q + "in", H * P + cd + H, W)
                yield q + "conv", rnd(q + "conv", cd, taps, s=taps ** -0.5)
                yield q + "conv.b", rnd(q + "conv.b", cd, s=0.1)
                yield q + "dt_bias", rnd(q + "dt_bias", H, s=0.5, off=-2.0)
                yield q + "A_log", rnd(q + "A_log", H, s=0.5)
                yield q + "D", rnd(q + "D", H, s=0.1, off=1.0)
                yield q + "norm", rnd(q + "norm", H * P, s=0.1, off=1.0)
                yield q + "o", lin(q + "o", W, H * P)
            elif kind == "parallel":
                a, b = m["left"], m["right"]
                H, D = int(a["heads"]), int(a["dim"])
                G, Dv = int(a.get("kv_heads", H)), int(a.get("vdim", D))
                l = q + "left."
                for nm, n in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                    yield l + nm, lin(l + nm, n, W)
                    yield l + nm + ".b", rnd(l + nm + ".b", n, s=0.1)
                yield l + "q.norm", rnd(l + "q.norm", H * D, s=0.1, off=1.0)
                yield l + "k.norm", rnd(l + "k.norm", G * D, s=0.1, off=1.0)
                yield l + "g", lin(l + "g", H, W)
                yield l + "o", lin(l + "o", W, H * Dv)
                H, D = int(b["heads"]), int(b["dim"])
                Dv = int(b.get("vdim", D))
                r = q + "right."
                for nm, n in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                    yield r + nm, lin(r + nm, n, W)
                yield r + "o", lin(r + "o", W, H * Dv)
            else:
                C, nb, taps = int(m["width"]), int(m["blocks"]), int(m.get("conv") or 1)
                n = C // nb
                for nm in ("y", "x"):
                    yield q + nm, lin(q + nm, C, W)
                    yield q + nm + ".b", rnd(q + nm + ".b", C, s=0.1)
                yield q + "conv", rnd(q + "conv", C, taps, s=taps ** -0.5)
                yield q + "conv.b", rnd(q + "conv.b", C, s=0.1)
                for nm in ("ra", "ri"):
                    yield q + nm, rnd(q + nm, nb, n, n, s=n ** -0.5)
                    yield q + nm + ".b", rnd(q + nm + ".b", nb, n, s=0.1)
                yield q + "lam", rnd(q + "lam", C, s=0.5, off=-4.0)
                yield q + "o", lin(q + "o", W, C)
            yield p + "norm1", rnd(p + "norm1", W, s=0.1, off=1.0)
            mlp = sp.get("mlp")
            for hc in ("hc1",) + (("hc2",) if mlp else ()):
                yield p + hc + ".in", rnd(p + hc + "i", S, s=0.1, off=1.0 / S)
                yield p + hc + ".out", rnd(p + hc + "o", S, s=0.2, off=1.0)
                yield p + hc + ".mix", torch.eye(S, dtype=dtype) + rnd(p + hc + "m", S, S, s=0.05)
            if mlp:
                ff = int(mlp["ff"])
                yield p + "norm2", rnd(p + "norm2", W, s=0.1, off=1.0)
                for nm, o, n in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                    yield p + "mlp." + nm, lin(p + nm, o, n)
        yield "final.norm", rnd("fn", W, s=0.1, off=1.0)
