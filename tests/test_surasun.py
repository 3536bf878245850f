"""Surasun through the serving engine (CPU tier, fp32) against the plain oracle in ``surasun_oracle.py``: every mechanism alone, prefill against
token-by-token decoding, prompt portions down to two tokens, unequal batches, page and slot reuse, page borders, far keys and far memory,
the first tokens, long decoding, sizes that differ from layer to layer, and greedy generation through ``Engine.generate``."""
import json
import math
import os

import numpy as np
import pytest
import torch

import sglang_b200 as sgl
import surasun_oracle as O
from sglang_b200.layers.gated_attention import scaled_inv_freq
from sglang_b200.layers.hyper_connections import StreamMix
from sglang_b200.ops import torch_ref

PAGE = 8


def _m2(heads=4, vdim=6, state=5, groups=2, norm_groups=2, conv=3):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv)}


def _par(heads=4, kv_heads=2, dim=8, vdim=6, rot=4, base=100.0, scale=0.5, cap=6.0, rh=3, rd=6, rv=4, rrot=4, rbase=50.0, decay=(0.5, 0.9, 0.999), ls=0.7,
         rs=1.3):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=cap, rot={"dims": rot, "base": base})
    right = dict(heads=rh, dim=rd, vdim=rv, decay=list(decay), rot={"dims": rrot, "base": rbase})
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs}}


def _lru(width=12, blocks=3, conv=4):
    return {"type": "rglru", "mixer": dict(width=width, blocks=blocks, conv=conv)}


def L(mix, ff=0):
    return dict(mix, mlp={"kind": "dense", "ff": ff} if ff else None)


def _cfg(layers, width=24, vocab=50, eps=1e-5, streams=2, mult=0.7):
    return {"architecture": "Surasun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult}


# sizes differ from layer to layer; feed-forwards behind every kind of mixer; one group and one block, and one per head
MIXED = _cfg([L(_m2(), 20), L(_par()), L(_lru(), 9), L(_m2(heads=3, vdim=4, state=9, groups=3, norm_groups=1, conv=4)),
              L(_par(heads=6, kv_heads=1, dim=6, vdim=9, rot=6, scale=0.3, cap=3.0, rh=1, rd=8, rv=7, rrot=8, decay=(0.8,), ls=1.0, rs=1.0), 14),
              L(_lru(width=20, blocks=1, conv=2)), L(_par(heads=2, kv_heads=2, dim=10, vdim=3, rot=2, rh=2, rd=5, rv=5, rrot=2, decay=(1.0, 0.97)), 11)],
             streams=3, mult=0.4)


def drawn_config(seed, friendly=False):
    """a randomly drawn stack: order of layers, head counts and sizes, state sizes, groups, taps, rotary widths, decays, caps, side weights, blocks,
    streams, feed-forwards.  ``friendly``: sizes in multiples of 16 (vector lanes, GEMM tiles)"""
    rng = np.random.default_rng(seed)
    pick = lambda *a: a[int(rng.integers(len(a)))]
    layers = []
    for _ in range(int(rng.integers(2, 7))):
        r = rng.random()
        if r < 0.33:
            g = pick(1, 2, 3)
            h, vd = g * pick(1, 2, 4), pick(16, 32) if friendly else pick(2, 5, 8, 12)
            ng = pick(*[k for k in (1, 2, g, h) if (h * vd) % k == 0])
            mix = _m2(heads=h, vdim=vd, state=pick(16, 32, 48) if friendly else pick(1, 3, 9, 17, 40), groups=g, norm_groups=ng, conv=pick(1, 2, 3, 4, 5))
        elif r < 0.66:
            g, rh = pick(1, 2, 3), pick(1, 2, 4)
            dim, rd = pick(16, 32, 64) if friendly else pick(2, 6, 8, 12), pick(16, 32) if friendly else pick(2, 6, 9, 17)
            mix = _par(heads=g * pick(1, 2, 3, 4), kv_heads=g, dim=dim, vdim=pick(16, 48) if friendly else pick(3, 5, 8), rot=pick(2, dim, max(2, dim // 4 * 2)),
                       base=pick(10.0, 1e4, 5e5), scale=pick(0.2, 0.6), cap=pick(2.0, 15.0), rh=rh, rd=rd, rv=pick(16, 32) if friendly else pick(2, 5, 11),
                       rrot=pick(2, rd // 2 * 2), rbase=pick(10.0, 1e4), decay=[pick(0.3, 0.9, 0.995, 1.0) for _ in range(rh)], ls=pick(1.0, 0.6), rs=pick(1.0, 1.4))
        else:
            nb = pick(1, 2, 5)
            mix = _lru(width=nb * (pick(16, 32, 64) if friendly else pick(1, 3, 7, 10)), blocks=nb, conv=pick(1, 2, 3, 4, 6))
        layers.append(L(mix, pick(0, 16, 64) if friendly else pick(0, 5, 12)))
    return _cfg(layers, width=pick(32, 64) if friendly else pick(10, 24, 36), vocab=pick(64, 128) if friendly else pick(19, 50, 131), eps=pick(1e-5, 1e-6),
                streams=pick(1, 2, 3, 4, 5), mult=pick(1.0, 0.5))


class Harness:
    """a model folder with random weights, an engine on it, and the oracle's logits for any token sequence"""

    def __init__(self, tmp, cfg, seed=0, slots=4, max_tokens=512, device="cpu", dtype="float32", page=PAGE, weights=None, **kw):
        from safetensors.torch import save_file

        self.cfg = cfg
        self.W = weights if weights is not None else O.random_weights(cfg, seed)
        d = os.path.join(str(tmp), f"m{seed}")
        os.makedirs(d, exist_ok=True)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump({**cfg, "dtype": dtype}, f)
        if dtype == "bfloat16":          # the oracle sees the rounded weights the engine serves
            self.W = {k: v.to(torch.bfloat16).float() for k, v in self.W.items()}
        save_file({k: v.contiguous() for k, v in self.W.items()}, os.path.join(d, "model.safetensors"))
        self.dir = d
        self.eng = sgl.Engine(model_path=d, device=device, skip_tokenizer_init=True, page_size=page, max_total_tokens=max_tokens,
                              max_running_requests=slots, context_length=max_tokens, disable_radix_cache=True, chunked_prefill_size=-1,
                              max_prefill_tokens=max_tokens, log_level="warning", **kw)
        self.sched = self.eng.scheduler
        self._oracle = {}

    @property
    def model(self):
        w = self.sched.worker
        return w.runner.model if hasattr(w, "runner") else w.model

    def oracle(self, tokens):
        k = tuple(tokens)
        if k not in self._oracle:
            self._oracle[k] = O.forward(self.cfg, self.W, list(tokens)).float().numpy()
        return self._oracle[k]

    def step(self, entries, end=()):
        return self.sched.replay_step([(i, list(t), list(w)) for i, t, w in entries], list(end))

    def run_cut(self, rid, tokens, cuts):
        """feed one request in portions of the given sizes (the rest token by token); returns logits of every position"""
        out, at = [], 0
        sizes = list(cuts) + [1] * (len(tokens) - sum(cuts))
        for n in sizes:
            last = at + n == len(tokens)
            out.append(self.step([(rid, tokens[at:at + n], range(n))], [rid] if last else []))
            at += n
        return np.concatenate(out, 0)

    def close(self):
        self.eng.shutdown()


def _tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def _close(a, b, tol=2e-4):
    err = np.abs(a - b).max() / max(1.0, float(np.sqrt((b ** 2).mean())))
    assert err < tol, err


# ------------------------------------------------------------------ mechanisms alone (functions of the serving path against the oracle's)
def test_stream_mix_and_layer_norm_reference_op():
    g = torch.Generator().manual_seed(0)
    S, T, W, mult = 3, 5, 12, 0.3
    X, y, w = torch.randn(T, S, W, generator=g), torch.randn(T, W, generator=g), torch.randn(W, generator=g)
    a, b = StreamMix(S), StreamMix(S)
    for hc in (a, b):
        hc.load("in", torch.randn(S, generator=g)), hc.load("out", torch.randn(S, generator=g)), hc.load("mix", torch.randn(S, S, generator=g))
    assert not a.load("other", torch.zeros(1))
    Wd = {"a.mix": a.mix.double(), "a.out": a.cout.double(), "a.in": a.cin.double(), "b.in": b.cin.double()}
    xs = [X[:, s].double() for s in range(S)]
    new = O.stream_update(xs, y.double(), Wd, "a.", mult)
    x2, h = torch_ref.stream_mix_norm(X.clone(), y, StreamMix.pack(a, b, mult, S, "cpu"), S, w, 1e-5, torch.float32, True, None, None, True)
    torch.testing.assert_close(x2.double(), torch.stack(new, 1), rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h.double(), O.layer_norm(O.stream_input(new, Wd, "b."), w.double(), 1e-5), rtol=1e-5, atol=1e-5)
    # before the first sublayer: copies of an embedding row, nothing added; behind the last one: the sum of the streams
    table, ids = torch.randn(7, W, generator=g), torch.tensor([3, 0, 6])
    x3, h = torch_ref.stream_mix_norm(None, None, StreamMix.pack(None, a, mult, S, "cpu"), S, w, 1e-5, torch.float32, True, table, ids, False)
    assert x3 is None
    e = table[ids].double()
    torch.testing.assert_close(h.double(), O.layer_norm(O.stream_input([e] * S, Wd, "a."), w.double(), 1e-5), rtol=1e-5, atol=1e-5)
    _, h = torch_ref.stream_mix_norm(X.clone(), y, StreamMix.pack(a, None, mult, S, "cpu"), S, w, 1e-5, torch.float32, True, None, None, False)
    torch.testing.assert_close(h.double(), O.layer_norm(sum(new), w.double(), 1e-5), rtol=1e-5, atol=1e-5)
    # one stream with unit numbers is the ordinary residual sum; without centring the norm is an RMS norm
    one = StreamMix.pack(StreamMix(1), StreamMix(1), 1.0, 1, "cpu")
    x4, h = torch_ref.stream_mix_norm(X[:, :1].clone(), y, one, 1, w, 1e-5, torch.float32, False, None, None, True)
    torch.testing.assert_close(x4[:, 0], X[:, 0] + y)
    torch.testing.assert_close(h.double(), O.rms((X[:, 0] + y).double(), 1e-5) * w.double(), rtol=1e-5, atol=1e-5)


def test_attention_prepare_with_neighbouring_pairs():
    g = torch.Generator().manual_seed(1)
    H, G, D, Dv, T = 4, 2, 6, 5, 9
    qkv = torch.randn(T, (H + G) * D + G * Dv + 3, generator=g)
    pos = torch.arange(500, 500 + T, dtype=torch.int32)
    loc = torch.randperm(40, generator=g)[:T].int()
    kc, vc = torch.full((40, 1, 14), 9.0), torch.full((40, 1, 14), 9.0)
    qw, kw = torch.randn(H * D, generator=g), torch.randn(G * D, generator=g)
    rot = {"dims": 4, "base": 300.0}
    fr = scaled_inv_freq(4, 300.0)
    q = torch_ref.attention_prepare(qkv, H, G, D, Dv, pos, kc, vc, loc, qw, kw, 1e-5, fr, interleaved=True)
    nq = (O.rms(qkv[:, :H * D].double(), 1e-5) * qw.double()).view(T, H, D)                        # all heads normed at once, before the rotation
    nk = (O.rms(qkv[:, H * D:(H + G) * D].double(), 1e-5) * kw.double()).view(T, G, D)
    for t in range(T):
        torch.testing.assert_close(q[t].double(), O.rotate(nq[t], int(pos[t]), rot, True), rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(kc[int(loc[t]), 0, :G * D].double().view(G, D), O.rotate(nk[t], int(pos[t]), rot, True), rtol=1e-5, atol=1e-5)
    v = qkv[:, (H + G) * D:(H + G) * D + G * Dv]
    assert torch.equal(vc[loc.long(), 0, :G * Dv], v) and float(kc[loc.long(), 0, G * D:].min()) == 9.0
    half = torch_ref.attention_prepare(qkv, H, G, D, Dv, pos, kc, vc, loc, qw, kw, 1e-5, fr)       # the other layout pairs other coordinates
    assert (half - q).abs().max() > 0.1


def _paged(g, n_pos, ps, width, n_pages=64):
    kc, vc = torch.randn(n_pages * ps, 1, width, generator=g) * 0.1, torch.randn(n_pages * ps, 1, width, generator=g) * 0.1
    need = (n_pos + ps - 1) // ps
    pages = torch.randperm(n_pages - 1, generator=g)[:need] + 1
    pt = torch.zeros(3, need + 2, dtype=torch.int32)
    pt[1, :need] = pages.int()
    return kc, vc, pt, (lambda pos: int(pages[pos // ps]) * ps + pos % ps)


def test_far_key_under_the_score_cap():
    """no window: a key 300 positions back wins when its score stands out, and the cap bounds by how much; the gate is one number per head"""
    H, G, D, Dv, ps, n, cap = 2, 1, 4, 2, 8, 330, 7.0
    g = torch.Generator().manual_seed(3)
    kc, vc, pt, at = _paged(g, n, ps, 4)
    kc[at(9), 0, :D] = torch.tensor([9.0, 0, 0, 0])
    vc[at(9), 0, :Dv] = 10.0
    q = torch.zeros(1, H, D)
    q[0, 0, 0], q[0, 1, 0] = 3.0, -3.0
    args = (kc, vc, G, Dv, pt, torch.tensor([1]), torch.tensor([n]), None, ps, 1.0, cap, -1, None, None)
    out = torch_ref.window_attention(q, *args)
    K, V = (torch.stack([c[at(p), 0, :d] for p in range(n)]).double() for c, d in ((kc, D), (vc, Dv)))
    for h in range(H):
        s = cap * torch.tanh(K @ q[0, h].double() / cap)
        torch.testing.assert_close(out[0, h].double(), O.softmax_rows(s, V), rtol=1e-5, atol=1e-6)
    assert out[0, 0, 0].item() > 5.0 and abs(out[0, 1, 0].item()) < 0.5
    gate = torch.randn(1, H, generator=g)
    torch.testing.assert_close(torch_ref.window_attention(q, *args, gate=gate, out_scale=0.8), out * torch.sigmoid(gate)[:, :, None] * 0.8)


def test_retention_inputs_scan_and_head_norm():
    """rotated q and k, the constant on k, the decaying memory in two portions on a used slot, heads normed alone, the SiLU gate"""
    g = torch.Generator().manual_seed(4)
    H, D, Dv, T, eps = 3, 6, 4, 30, 1e-5
    proj = torch.randn(T, H * (2 * Dv + 2 * D), generator=g)                                       # [v | k | q | g]
    nv, nk = H * Dv, H * D
    rot, decay = {"dims": 4, "base": 77.0}, [0.5, 0.97, 1.0]
    u = torch_ref.linear_attention_prepare(proj, H, D, Dv, torch.arange(T), scaled_inv_freq(4, 77.0), False, D ** -0.5, False)
    state = torch.randn(3, H, D, Dv, generator=g)
    outs = [torch_ref.mamba2_scan(u[a:b], None, None, None, None, None, state, torch.tensor([2]), torch.tensor([b]), torch.tensor([b - a]), H, Dv, D, H,
                                  torch.tensor(decay)) for a, b in ((0, 11), (11, 13), (13, T))]
    got = torch_ref.grouped_rmsnorm(torch.cat(outs), None, H, eps, torch.float32, proj[:, nv + 2 * nk:], 1.3, "silu")
    W = {"q": torch.zeros(nk, proj.shape[1]), "k": torch.zeros(nk, proj.shape[1]), "v": torch.zeros(nv, proj.shape[1]), "g": torch.zeros(nv, proj.shape[1])}
    for nm, at, n in (("v", 0, nv), ("k", nv, nk), ("q", nv + nk, nk), ("g", nv + 2 * nk, nv)):
        W[nm][torch.arange(n), at + torch.arange(n)] = 1.0                                         # the projections pick their columns
    W = {k: v.double() for k, v in W.items()} | {"o": torch.eye(nv, dtype=torch.float64)}
    want = O.retention(proj.double(), dict(heads=H, dim=D, vdim=Dv, decay=decay, rot=rot), W, "", eps)
    torch.testing.assert_close(got.double(), 1.3 * want, rtol=1e-4, atol=1e-5)
    silu = torch_ref.linear_attention_prepare(proj, H, D, Dv, torch.arange(T), None, False, 1.0, True)
    torch.testing.assert_close(silu, torch.nn.functional.silu(proj[:, :nv + 2 * nk]))
    inter = torch_ref.linear_attention_prepare(proj, H, D, Dv, torch.arange(T), scaled_inv_freq(4, 77.0), True, 2.0, False)
    k = torch.stack([O.rotate(proj[t, nv:nv + nk].double().view(H, D), t, rot, True) for t in range(T)]).reshape(T, nk) * 2.0
    torch.testing.assert_close(inter[:, nv:nv + nk].double(), k, rtol=1e-5, atol=1e-5)


def test_retention_far_memory():
    """a write at t = 3 read back 400 tokens later through a slow decay, and forgotten by a fast one"""
    H, D, Dv, T = 2, 4, 3, 404
    g = torch.Generator().manual_seed(5)
    u = torch.randn(T, H * (Dv + 2 * D), generator=g) * 0.01
    for h in range(H):
        u[3, h * Dv:(h + 1) * Dv] = torch.tensor([5.0, -4.0, 3.0])
        u[3, H * Dv + h * D] = 6.0
        u[-1, H * Dv + H * D + h * D] = 7.0
    y = torch_ref.mamba2_scan(u, None, None, None, None, None, torch.zeros(1, H, D, Dv), torch.tensor([0]), torch.tensor([T]), torch.tensor([T]), H, Dv, D, H,
                              torch.tensor([0.9995, 0.9]))
    want = 42.0 * torch.tensor([5.0, -4.0, 3.0])
    assert (y[-1, :Dv] - want * 0.9995 ** (T - 4)).abs().max() < 0.02 * want.abs().max() and y[-1, Dv:].abs().max() < 0.05


def test_gated_recurrence_and_far_memory():
    """gates, decay and state in three portions on a used slot; then a write at t = 3 that stands out, read back 400 tokens later"""
    g = torch.Generator().manual_seed(6)
    nb, n, T = 3, 4, 30
    C = nb * n
    u, y, lam = torch.randn(T, C, generator=g), torch.randn(T, C, generator=g), torch.randn(C, generator=g)
    ra, ri, ba, bi = (torch.randn(nb, n, *s, generator=g) for s in ((n,), (n,), (), ()))
    gw, gb = torch.cat([ra, ri], 1), torch.cat([ba, bi], 1)
    state = torch.randn(3, 1, 1, C, generator=g)
    outs = [torch_ref.rglru_scan(torch_ref.block_linear_f32(u[a:b], gw), gb, u[a:b], lam, y[a:b], state, torch.tensor([1]), torch.tensor([b]),
                                 torch.tensor([b - a]), torch.float32, nb) for a, b in ((0, 2), (2, 19), (19, T))]
    W = {"ra": ra.double(), "ri": ri.double(), "ra.b": ba.double(), "ri.b": bi.double(), "lam": lam.double()}
    a, i = O.rglru_gates(u.double(), W, "", nb)
    S, want = torch.zeros(C, dtype=torch.float64), []
    for t in range(T):
        S = a[t] * S + torch.sqrt(1 - a[t] ** 2) * i[t] * u[t].double()
        want.append(S * O.gelu_tanh(y[t].double()))
    torch.testing.assert_close(torch.cat(outs).double(), torch.stack(want), rtol=1e-4, atol=1e-5)
    torch.testing.assert_close(state[1, 0, 0].double(), S, rtol=1e-4, atol=1e-5)
    T = 404
    u = torch.zeros(T, 2)
    u[3] = 40.0
    gates = torch.zeros(T, 1, 4)
    gates[:, 0, :2] = -2.0                                              # recurrence gate nearly closed; input gate half open
    out = torch_ref.rglru_scan(gates, None, u, torch.tensor([-9.0, 2.0]), torch.full((T, 2), 3.0), torch.ones(1, 1, 1, 2), torch.tensor([0]), torch.tensor([T]),
                               torch.tensor([T]), torch.float32, 1)
    la = [-8.0 / (1 + math.exp(2.0)) * math.log1p(math.exp(v)) for v in (-9.0, 2.0)]
    want = math.sqrt(-math.expm1(2 * la[0])) * 20.0 * math.exp(la[0] * (T - 4)) * 3.0 / (1 + math.exp(-2 * math.sqrt(2 / math.pi) * (3 + 0.044715 * 27)))
    assert abs(float(out[-1, 0]) - want) < 1e-4 * want and want > 0.3 and abs(float(out[-1, 1])) < 1e-6


def test_config_reader(tmp_path):
    from sglang_b200.configs.model_config import load_model_config

    d = tmp_path / "cfg"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(MIXED))
    c = load_model_config(str(d))
    assert c.architecture == "Surasun" and c.hidden_size == 24 and c.vocab_size == 50 and c.num_hidden_layers == 7 and c.rms_norm_eps == 1e-5
    assert c.hybrid["streams"] == 3 and c.hybrid["residual_mult"] == 0.4 and c.hybrid["layers"][1]["mixer"]["right"]["decay"][2] == 0.999


# ------------------------------------------------------------------ single mechanisms through the engine
@pytest.mark.parametrize("cfg", [
    _cfg([L(_m2())]), _cfg([L(_m2(heads=1, vdim=5, state=1, groups=1, norm_groups=1, conv=1), 7)], streams=1, mult=1.0),
    _cfg([L(_m2(heads=6, groups=6, norm_groups=6, state=17, conv=5))], streams=5), _cfg([L(_par())]),
    _cfg([L(_par(heads=5, kv_heads=1, rot=8, cap=1.5, rh=1, decay=(1.0,)), 10)], streams=1), _cfg([L(_par(heads=3, kv_heads=3, vdim=11, rrot=6, ls=0.2, rs=3.0))]),
    _cfg([L(_lru())]), _cfg([L(_lru(width=7, blocks=7, conv=1), 6)], streams=4), _cfg([L(_lru(width=10, blocks=1, conv=6))], mult=1.0)])
def test_one_layer_models(tmp_path, cfg):
    h = Harness(tmp_path, cfg)
    toks = _tokens(37, 50, 5)
    ref = h.oracle(toks)
    _close(h.step([("a", toks, range(len(toks)))], ["a"]), ref)                    # whole prompt
    _close(h.run_cut("b", toks, []), ref)                                          # token by token from the first token
    h.close()


def test_a_far_token_decides(tmp_path):
    """weights under which one early token stands out for attention: its key answers every later query, so the logits 100 tokens on, across many
    pages, in a portion and in decoding, follow the far value; a model that lost the key would differ everywhere"""
    cfg = _cfg([L(_par(heads=2, kv_heads=1, dim=4, rot=2, scale=1.0, cap=30.0, rs=0.0))], streams=1, mult=1.0)
    W = O.random_weights(cfg, 5)
    W["embed"][7] *= 3.0
    W["l0.mix.left.q"] = W["l0.mix.left.q"] * 4
    W["l0.mix.left.k"] = W["l0.mix.left.k"] * 4
    W["l0.mix.left.v"] = W["l0.mix.left.v"] * 6
    h = Harness(tmp_path, cfg, weights=W)
    a = [int(t) for t in np.random.default_rng(0).integers(8, 50, size=120)]
    b = list(a)
    a[3], b[3] = 7, 20
    ra, rb = h.oracle(a), h.oracle(b)
    assert np.abs(ra[100:] - rb[100:]).max() > 0.02                                # the far token shows in the oracle
    for toks, ref in ((a, ra), (b, rb)):
        _close(h.run_cut("x", toks, [2, 60, 2, 31]), ref)
    h.close()


# ------------------------------------------------------------------ the mixed model: cuts, batches, reuse
@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    h = Harness(tmp_path_factory.mktemp("surasun"), MIXED, seed=3, slots=4, max_tokens=40 * PAGE)
    yield h
    h.close()


def test_streams_after_every_layer(mixed):
    toks = _tokens(17, 50, 6)
    want, got = [], []
    O.forward(mixed.cfg, mixed.W, toks, tap=lambda i, x: want.append(x.float()))
    mixed.model.layer_tap = lambda i, x: got.append(x.clone())
    try:
        mixed.step([("t", toks, [])], ["t"])
    finally:
        mixed.model.layer_tap = None
    assert len(got) == len(want) == 7
    for a, b in zip(got, want):
        torch.testing.assert_close(a.cpu(), b, rtol=1e-4, atol=1e-4)


def test_first_tokens_and_prefill_against_decode(mixed):
    toks = _tokens(61, 50, 7)
    ref = mixed.oracle(toks)
    whole = mixed.step([("w", toks, range(len(toks)))], ["w"])
    _close(whole, ref)
    _close(whole[:3], ref[:3], 1e-4)                                               # positions 0, 1, 2: zero history, zero state
    _close(mixed.run_cut("d", toks, [30]), ref)
    one = mixed.step([("s", toks[:1], [0])], ["s"])                                # a sequence of one token
    _close(one, ref[:1])


@pytest.mark.parametrize("cuts", [[2, 2, 2, 3, 2], [7, 8, 9, 2, 16], [1, 2, 17, 2, 2, 23], [PAGE, PAGE, 2 * PAGE], [PAGE - 1, 2, PAGE + 1, 19]])
def test_portions_of_many_sizes(mixed, cuts):
    toks = _tokens(70, 50, 11)
    _close(mixed.run_cut("c", toks, cuts), mixed.oracle(toks))


def test_unequal_batches_and_reuse_of_pages_and_slots(mixed):
    rng = np.random.default_rng(5)
    lens = [53, 9, 31, 2, 44, 18, 27]
    seqs = [_tokens(n, 50, 100 + i) for i, n in enumerate(lens)]
    at = [0] * len(seqs)
    got = [[] for _ in seqs]
    waiting, live = list(range(len(seqs))), []
    rounds = 0
    while waiting or live:
        while waiting and len(live) < 4:                                           # four slots: later requests take over freed slots and pages
            live.append(waiting.pop(0))
        entries, end = [], []
        for i in live:
            left = len(seqs[i]) - at[i]
            n = int(min(left, rng.choice([1, 1, 2, 3, 5, 11, 16])))
            if at[i] and rng.random() < 0.2:
                continue                                                           # a request may sit a step out
            entries.append((f"r{i}", seqs[i][at[i]:at[i] + n], range(n)))
        if not entries:
            continue
        for rid, t, _ in entries:
            i = int(rid[1:])
            if at[i] + len(t) == len(seqs[i]):
                end.append(rid)
        out = mixed.step(entries, end)
        o = 0
        for rid, t, _ in entries:
            i = int(rid[1:])
            got[i].append(out[o:o + len(t)])
            o += len(t)
            at[i] += len(t)
            if at[i] == len(seqs[i]):
                live.remove(i)
        rounds += 1
    assert rounds > 10
    for i, s in enumerate(seqs):
        _close(np.concatenate(got[i], 0), mixed.oracle(s))
    assert mixed.sched.kv.allocator.available_pages() == mixed.sched.kv.allocator.total_pages        # everything was given back
    assert mixed.sched.kv.slots.available() == 4


def test_long_decoding(mixed):
    toks = _tokens(5 + 90, 50, 13)
    _close(mixed.run_cut("l", toks, [5]), mixed.oracle(toks), 3e-4)


def test_greedy_generation_through_the_engine(mixed):
    prompts = [_tokens(n, 50, 40 + n) for n in (12, 3, 25)]
    outs = mixed.eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 10, "temperature": 0, "ignore_eos": True})
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(10):
            seq.append(int(mixed.oracle(seq)[-1].argmax()))
        assert o["output_ids"] == seq[len(p):]
    mixed.sched.check_invariants()


def test_text_prompts_on_a_weights_only_folder(tmp_path):
    """a folder with only config.json and model.safetensors serves text through the byte tokenizer (what `cli generate` and the HTTP server do)"""
    h = Harness(tmp_path, _cfg([L(_lru(), 8), L(_par()), L(_m2())], vocab=300), seed=8)
    h.close()
    eng = sgl.Engine(model_path=h.dir, device="cpu", page_size=PAGE, max_total_tokens=256, max_running_requests=2, log_level="warning")
    out = eng.generate("hello there", {"max_new_tokens": 4, "temperature": 0.7, "top_k": 5, "ignore_eos": True})
    assert len(out["output_ids"]) == 4 and isinstance(out["text"], str)
    eng.shutdown()


def test_random_init_weights_cover_the_model(tmp_path):
    """the random-weight path (benchmarks without a checkpoint) names every tensor of the model and runs"""
    d = tmp_path / "dummy"
    d.mkdir()
    (d / "config.json").write_text(json.dumps({**MIXED, "dtype": "float32"}))
    eng = sgl.Engine(model_path=str(d), load_format="dummy", device="cpu", skip_tokenizer_init=True, page_size=PAGE, max_total_tokens=256,
                     max_running_requests=2, log_level="warning")
    w = eng.scheduler.worker
    model = w.runner.model if hasattr(w, "runner") else w.model
    named = dict(model.dummy_checkpoint(model.cfg, "cpu", torch.float32))
    assert set(named) == set(O.random_weights(MIXED)) and len(model.load_weights(named.items())) == len(named)
    out = eng.generate(input_ids=[_tokens(9, 50, 1)], sampling_params={"max_new_tokens": 4, "temperature": 0, "ignore_eos": True})
    assert len(out[0]["output_ids"]) == 4
    eng.shutdown()


@pytest.mark.parametrize("seed", [1, 2, 3, 4])
def test_randomly_drawn_stacks(tmp_path, seed):
    cfg = drawn_config(seed)
    h = Harness(tmp_path, cfg, seed=50 + seed, max_tokens=30 * PAGE)
    V = cfg["vocab"]
    a, b = _tokens(45, V, 1), _tokens(14, V, 2)
    ra, rb = h.oracle(a), h.oracle(b)
    _close(h.step([("w", a, range(len(a)))], ["w"]), ra, 3e-4)
    _close(h.run_cut("c", a, [19, 2, 9, 2]), ra, 3e-4)
    out = h.step([("a", a[:30], range(30)), ("b", b, range(len(b)))], ["b"])
    _close(out[:30], ra[:30], 3e-4); _close(out[30:], rb, 3e-4)
    _close(h.step([("a", a[30:], range(15))], ["a"]), ra[30:], 3e-4)
    h.close()
