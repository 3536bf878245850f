"""Mumasun through the serving engine (CPU tier, fp32) against the plain oracle in ``mumasun_oracle.py``: every mechanism alone, prefill against
token-by-token decoding, prompt portions down to two tokens, unequal batches, page and slot reuse, far keys, keys just inside and just outside
a chunk, page borders, the first tokens, long decoding, sizes that differ from layer to layer, and greedy generation through
``Engine.generate``."""
import json
import math
import os
import types

import numpy as np
import pytest
import torch

import mumasun_oracle as O
import sglang_b200 as sgl
from sglang_b200.layers.differential_attention import DifferentialAttention
from sglang_b200.layers.latent_attention import yarn_inv_freq
from sglang_b200.ops import moe_ops, torch_ref

PAGE = 8
YARN = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}


def _mix(heads=4, kv_heads=2, dim=6, vdim=10, rot_dims=4, base=100.0, scaling=YARN, scale=0.5, chunk=12, conv=3, diff=0.4):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, conv=conv, diff=diff)
    if chunk:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims, **({"scaling": scaling} if scaling else {})}
    return {"type": "attention", "mixer": m}


def _moe(ff=9, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def L(mix, mlp):
    return dict(mix, mlp=mlp)


def _cfg(layers, width=24, vocab=50, eps=1e-5, logit_scale=1.5):
    return {"architecture": "Mumasun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}


# sizes, chunks, taps and constants differ from layer to layer
MIXED = _cfg([L(_mix(), _moe()), L(_mix(heads=3, kv_heads=3, dim=8, vdim=5, rot_dims=8, base=1000.0, scaling=None, chunk=7, conv=2, diff=0.2), None),
              L(_mix(heads=4, kv_heads=1, dim=4, vdim=8, rot_dims=2, chunk=16, conv=5, diff=0.8, scale=0.3), _moe(12, 3, 1)),
              L(_mix(heads=2, kv_heads=2, dim=5, vdim=3, rot_dims=0, chunk=0, conv=1, diff=0.1), _moe(4, 4, 4))])


def drawn_config(seed, friendly=False):
    """a randomly drawn stack: head counts and sizes, chunks, taps, rotary widths, experts.  ``friendly``: sizes in multiples of 16 (vector lanes,
    GEMM tiles)"""
    rng = np.random.default_rng(seed)
    pick = lambda *a: a[int(rng.integers(len(a)))]
    layers = []
    for _ in range(int(rng.integers(2, 5))):
        g = pick(1, 2, 3)
        dim = pick(16, 32, 64) if friendly else pick(2, 5, 8, 11)
        mix = _mix(heads=g * pick(1, 2, 3, 4), kv_heads=g, dim=dim, vdim=pick(16, 64, 128) if friendly else pick(2, 6, 9),
                   rot_dims=pick(0, 2, dim // 2 * 2), base=pick(50.0, 30000.0), scaling=pick(None, YARN, {"factor": 2.0, "original": 16, "fast": 4.0, "slow": 0.5}),
                   scale=pick(0.2, 0.5), chunk=pick(0, 5, 16, 23, 40), conv=pick(1, 2, 3, 4, 6), diff=pick(0.1, 0.3, 0.7))
        layers.append(L(mix, None if rng.random() < 0.25 else _moe(pick(16, 64) if friendly else pick(3, 12, 33), pick(1, 2, 6), pick(1, 1, 2))))
        if layers[-1]["mlp"]:
            r = layers[-1]["mlp"]["router"]
            r["top"] = min(r["top"], r["experts"])
    return _cfg(layers, width=pick(32, 64) if friendly else pick(10, 24, 36), vocab=pick(64, 128) if friendly else pick(19, 50, 131), eps=pick(1e-5, 1e-6),
                logit_scale=pick(1.0, 0.5, 3.0))


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
        self.eng = sgl.Engine(**{**dict(model_path=d, device=device, skip_tokenizer_init=True, page_size=page, max_total_tokens=max_tokens,
                                        max_running_requests=slots, context_length=max_tokens, disable_radix_cache=True, chunked_prefill_size=-1,
                                        max_prefill_tokens=max_tokens, log_level="warning"), **kw})
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


class LayerBench:
    """one attention layer whose projections are identities (its input rows ARE the projection rows [q | k | v]) over a scattered paged cache,
    fed portion by portion: what the serving path computes for chosen queries, keys and values"""

    def __init__(self, H, G, D, Dv, scale, diff, lam_extra=0.0, taps=1, chunk=0, ps=8, pages=64, device="cpu", dtype=torch.float32, conv=None, rotary=None):
        self.m = m = DifferentialAttention(2 * H * D + 2 * G * D + G * Dv, H, G, D, Dv, scale, diff, 1e-5, dtype, taps=taps, rotary=rotary, chunk=chunk, qk_norm=False)
        n = m.rows
        m.load("q", torch.eye(n)[:m.n_q]); m.load("k", torch.eye(n)[m.n_q:m.n_q + m.n_k]); m.load("v", torch.eye(n)[m.n_q + m.n_k:])
        m.load("o", torch.eye(n)[:, :H * Dv])
        if conv is None:
            conv = torch.zeros(n, taps)
            conv[:, -1] = 1.0
        m.load("q.conv", conv[:m.n_q]); m.load("k.conv", conv[m.n_q:m.n_q + m.n_k]); m.load("v.conv", conv[m.n_q + m.n_k:])
        m.load("lq1", torch.full((D,), 0.0)); m.load("lk1", torch.full((D,), 0.0))
        m.load("lq2", torch.tensor([math.log(1.0 - lam_extra)] + [0.0] * (D - 1))); m.load("lk2", torch.ones(D))          # lam = 1 - (1 - x) + diff
        self.lam = lam_extra + diff
        m.to(device)
        self.dev, self.ps, self.n_out = device, ps, H * Dv
        wid = -(-m.cache_width // 8) * 8
        self.kc, self.vc = torch.zeros((pages + 1) * ps, 1, wid, dtype=dtype, device=device), torch.zeros((pages + 1) * ps, 1, wid, dtype=dtype, device=device)
        self.pt = torch.zeros(2, pages + 1, dtype=torch.int32)
        self.pt[1, :pages] = torch.randperm(pages, generator=torch.Generator().manual_seed(1)).int() + 1
        conv_state = torch.full((2, n, max(1, taps - 1)), 7.0, dtype=dtype, device=device)               # a used slot: a new request must not see it
        self.pool = types.SimpleNamespace(k=lambda i: self.kc, v=lambda i: self.vc, mamba=types.SimpleNamespace(conv=[conv_state]))
        self.done, self.dtype = 0, dtype

    def run(self, x, decode=False):
        """rows [n, rows] -> heads [n, H * Dv]; ``decode``: in the layout of decode steps (one token per request)"""
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=self.dev)
        n, pos = x.shape[0], list(range(self.done, self.done + x.shape[0]))
        self.done += n
        fb = types.SimpleNamespace(kv_pool=self.pool, positions=i32(pos), cu_q=None if decode else i32([0, n]), req_slots=i32([1]), seq_lens=i32([self.done]),
                                   q_lens=None if decode else i32([n]), max_q_len=n, page_size=self.ps, page_table=self.pt.to(self.dev), num_splits=2 if decode else 1,
                                   attn_workspace=None, out_cache_loc=i32([int(self.pt[1, p // self.ps]) * self.ps + p % self.ps for p in pos]))
        return self.m(x.to(self.dtype).to(self.dev), fb, 0, 0)[:, :self.n_out].float().cpu()


def check_chunk_edges(device, dtype, ps, D, Dv, tol, tc_route=True):
    """one key stands out for one query; just inside the query's chunk its value takes over, just outside it is not seen.  Keys at the chunk's first
    position, at page borders and far back among hundreds; the query in a prompt, at the start of a portion, and decoded alone"""
    H, G = 2, 1
    for chunk, i, j in ((16, 31, 16), (16, 32, 31), (16, 31, 15), (110, 109, 0), (110, 110, 109), (110, 219, 110), (110, 219, 109), (0, 299, 3), (300, 299, 0), (300, 300, 299),
                        (13, 25, 13), (13, 26, 25), (64, 127, 64), (64, 128, 127), (1, 5, 4), (1, 5, 5), (7, 48, 42), (7, 49, 48)):
        if j > i:
            continue
        T = i + 3
        g = torch.Generator().manual_seed(i * 1000 + j)
        rows = 2 * H * D + 2 * G * D + G * Dv
        x = torch.zeros(T, rows)
        k0, v0 = 2 * H * D, 2 * H * D + 2 * G * D
        x[:, k0 + 1] = 3.0; x[:, k0 + D + 1] = 3.0                            # every key along axis 1 in both maps ...
        x[j, k0:k0 + 2 * D] = 0.0
        x[j, k0] = 6.0                                                        # ... but the marked one: map 1 along axis 0
        x[i, 0] = 6.0                                                         # head 0, map 1 of the query looks for it (map 2 sees no difference)
        base, mark = torch.randn(Dv, generator=g), torch.randn(Dv, generator=g)
        x[:, v0:] = base
        x[j, v0:] = mark
        vis = j >= (i // chunk * chunk if chunk else 0)
        lo = i // chunk * chunk if chunk else 0
        n = i - lo + 1
        b, mk = base.to(dtype).double(), mark.to(dtype).double()
        mean = (b * (n - 1) + mk) / n if vis else b                           # map 2 (and the other head): equal weights over the chunk
        lam, diff = 0.5, 0.3
        want = O.combine(mk if vis else b, mean, lam, diff, 1e-5)
        for mode in ("prompt", "portion", "decode", "tokens"):
            lb = LayerBench(H, G, D, Dv, 1.0, diff, lam_extra=0.2, chunk=chunk, ps=ps, pages=400 // ps, device=device, dtype=dtype)
            if mode == "prompt":
                o = lb.run(x)[i]
            elif mode == "portion":                                           # the query opens a portion of two
                parts = [lb.run(x[:i])] if i else []
                o = lb.run(x[i:i + 2])[0]
            elif mode == "decode":
                if i:
                    lb.run(x[:i])
                o = lb.run(x[i:i + 1], decode=True)[0]
            else:
                if i > 64:
                    continue
                o = [lb.run(x[t:t + 1], decode=True)[0] for t in range(i + 1)][-1]
            torch.testing.assert_close(o[:Dv].double(), want, rtol=tol, atol=tol)
            hidden = O.combine(b, b, lam, diff, 1e-5)                         # what a query that does not see the key gives
            assert not vis or float((o[:Dv].double() - hidden).abs().max()) > 0.1
            other = O.combine(mean, mean, lam, diff, 1e-5)                    # head 1 did not look for it
            torch.testing.assert_close(o[Dv:2 * Dv].double(), other, rtol=tol, atol=tol)


# ------------------------------------------------------------------ mechanisms alone (functions of the serving path against the oracle's or hand-written sums)
def test_chunk_edges_and_far_keys():
    check_chunk_edges("cpu", torch.float32, 8, 4, 6, 1e-3)


def test_rotary_frequencies_and_yarn_blend():
    for dims, base, sc in ((24, 2e5, {"factor": 3.0, "original": 1024, "fast": 24.0, "slow": 2.0}), (8, 100.0, YARN), (6, 50.0, None), (2, 10.0, YARN)):
        want, wm = O.frequencies(base, dims, sc)
        got, gm = yarn_inv_freq(dims, base, sc)
        torch.testing.assert_close(got.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0)
        assert abs(gm - wm) < 1e-12


@pytest.mark.parametrize("taps", [1, 2, 3, 5])
def test_short_convolution_crosses_portions_and_starts_from_zero(taps):
    """portions shorter than the taps, single tokens, and a used slot: the values that reach the cache are the oracle's convolution"""
    H, G, D, Dv, T = 2, 1, 3, 4, 23
    g = torch.Generator().manual_seed(taps)
    n = 2 * H * D + 2 * G * D + G * Dv
    conv, x = torch.randn(n, taps, generator=g), torch.randn(T, n, generator=g)
    want = O.short_conv(x.double(), conv.double())
    for cuts in ([T], [1] * T, [2, 1, 2, 3, 2, 5, 8], [9, 2, 12]):
        for decode in (False, True):
            lb = LayerBench(H, G, D, Dv, 0.3, 0.2, taps=taps, conv=conv)
            at = 0
            for c in cuts:
                lb.run(x[at:at + c], decode=decode and c == 1)
                at += c
            rows = [int(lb.pt[1, t // 8]) * 8 + t % 8 for t in range(T)]
            torch.testing.assert_close(lb.kc[rows, 0, :2 * G * D].double(), want[:, 2 * H * D:2 * H * D + 2 * G * D], rtol=1e-5, atol=1e-5)
            torch.testing.assert_close(lb.vc[rows, 0, :G * Dv].double(), want[:, -G * Dv:], rtol=1e-5, atol=1e-5)
            if taps > 1:
                torch.testing.assert_close(lb.pool.mamba.conv[0][1], x[-(taps - 1):].T)


def test_map_norm_rotation_and_layout_of_queries_and_keys():
    g = torch.Generator().manual_seed(3)
    T, H, G, D, Dv, rot = 9, 4, 2, 6, 5, 4
    C = 2 * H * D + 2 * G * D + G * Dv
    x, nq, nk = torch.randn(T, C, generator=g), torch.randn(D, generator=g), torch.randn(D, generator=g)
    f, mult = yarn_inv_freq(rot, 100.0, YARN)
    for pad in (0, 16):
        seg = pad // 2 or D
        kc, vc = torch.full((T + 8, 1, 60), 9.0), torch.full((T + 8, 1, 60), 9.0)
        loc, pos = torch.arange(T, dtype=torch.int32) + 3, torch.arange(T, dtype=torch.int32)
        q = torch_ref.conv_attention_prepare(x, H, G, 2, D, Dv, torch.ones(C, 1), torch.zeros(2, C, 1), pos, None, torch.zeros(T, dtype=torch.int32), pos + 1, nq, nk, 1e-5,
                                             f, mult, kc, vc, loc, pad)
        fo, mo = O.frequencies(100.0, rot, YARN)
        qw = O.turn(O.unit_rms(x[:, :2 * H * D].double().view(T, H, 2, D), 1e-5) * nq.double(), fo, mo)
        kw = O.turn(O.unit_rms(x[:, 2 * H * D:2 * (H + G) * D].double().view(T, G, 2, D), 1e-5) * nk.double(), fo, mo)
        assert q.shape == (T, 2 * H, 2 * seg)
        for h in range(H):
            for m in (0, 1):
                row = q[:, 2 * h + m].double()
                torch.testing.assert_close(row[:, m * seg:m * seg + D], qw[:, h, m], rtol=1e-4, atol=1e-5)
                row[:, m * seg:m * seg + D] = 0
                assert float(row.abs().max()) == 0.0                                   # nothing in the other map's place, nor in the padding
        for gk in range(G):
            for m in (0, 1):
                torch.testing.assert_close(kc[3:3 + T, 0, (2 * gk + m) * seg:(2 * gk + m) * seg + D].double(), kw[:, gk, m], rtol=1e-4, atol=1e-5)
        torch.testing.assert_close(vc[3:3 + T, 0, :(pad or Dv)][:, :Dv], x[:, -G * Dv:][:, :Dv])


def test_lambda_and_the_combination_of_two_maps():
    m = DifferentialAttention(8, 2, 1, 3, 4, None, 0.35, 1e-5, torch.float32)
    vec = {n: torch.randn(3, generator=torch.Generator().manual_seed(i)) for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))}
    assert abs(m.lam() - 0.35) < 1e-12                                                 # exp(0) - exp(0) + diff
    for n, v in vec.items():
        assert m.load(n, v)
    assert abs(m.lam() - O.lam({n: v.double() for n, v in vec.items()}, "", {"diff": 0.35})) < 1e-6
    o = torch.randn(5, 4, 7, generator=torch.Generator().manual_seed(9))
    got = torch_ref.differential_combine(o, 0.8, 0.6, 1e-5)
    for h in (0, 1):
        torch.testing.assert_close(got[:, h].double(), O.combine(o[:, 2 * h].double(), o[:, 2 * h + 1].double(), 0.8, 0.4, 1e-5), rtol=1e-5, atol=1e-6)


def test_router_and_experts_whose_inputs_are_weighted():
    g = torch.Generator().manual_seed(4)
    W, ff, E, T = 6, 5, 4, 11
    P = {"router": torch.randn(E, W, generator=g) * 2}
    for e in range(E):
        P[f"e{e}.up"], P[f"e{e}.down"] = torch.randn(ff, W, generator=g), torch.randn(W, ff, generator=g)
    h = torch.randn(T, W, generator=g)
    from sglang_b200.models.mumasun import SigmoidInputMoE

    for top in (1, 2, 4):
        mlp = _moe(ff, E, top)
        moe = SigmoidInputMoE(W, mlp, torch.float32, 0)
        assert all(moe.load(n, w) for n, w in P.items()) and not moe.load("e9.up", P["e0.up"]) and not moe.load("e0.gate", P["e0.up"])
        want = O.experts(h.double(), {k: v.double() for k, v in P.items()}, "", mlp)
        torch.testing.assert_close(moe(h).double(), want, rtol=1e-4, atol=1e-5)
        w, ids = moe_ops.sigmoid_route(h @ P["router"].T, top)
        srt = moe_ops._fused_moe_sorted(h, moe.experts.w13, moe.experts.w2, w, ids, 0, lambda u: torch.relu(u) ** 2, True)
        torch.testing.assert_close(srt.double(), want, rtol=1e-4, atol=1e-5)
        out_w = moe_ops.fused_moe(h, moe.experts.w13, moe.experts.w2, w, ids, 0, ("relu2",), False)
        assert float((out_w.double() - want).abs().max()) > 1e-2                       # weighting the output is something else
    z = torch.tensor([[50.0, 60.0, 55.0, -1.0]])                                       # saturated scores: the order of the logits decides
    assert moe_ops.sigmoid_route(z, 2)[1].tolist() == [[1, 2]]


def test_output_norm_residual_reference_op():
    g = torch.Generator().manual_seed(0)
    x, y, w = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g), torch.randn(12, generator=g) * 0.2
    r = x.clone()
    torch_ref.norm_add_f32(r, y, w, 1e-5, True, torch.float32)
    torch.testing.assert_close(r.double(), x.double() + O.centred_norm(y.double(), w.double(), 1e-5), rtol=1e-5, atol=1e-6)


def test_config_reader(tmp_path):
    from sglang_b200.configs.model_config import load_model_config

    d = tmp_path / "cfg"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(MIXED))
    c = load_model_config(str(d))
    assert c.architecture == "Mumasun" and c.hidden_size == 24 and c.vocab_size == 50 and c.num_hidden_layers == 4 and c.rms_norm_eps == 1e-5
    assert c.hybrid["logit_scale"] == 1.5 and c.hybrid["layers"][0]["mixer"]["rot"]["scaling"] == YARN and c.num_local_experts == 5


# ------------------------------------------------------------------ single mechanisms through the engine
@pytest.mark.parametrize("cfg", [
    _cfg([L(_mix(), None)]), _cfg([L(_mix(heads=6, kv_heads=1, rot_dims=6, scaling=None, chunk=0, conv=1), _moe())]),
    _cfg([L(_mix(heads=1, kv_heads=1, dim=1, vdim=2, rot_dims=0, chunk=1, conv=4), None)]), _cfg([L(_mix(chunk=5, conv=2), _moe(7, 1, 1))], logit_scale=0.25),
    _cfg([L(_mix(heads=3, kv_heads=3, dim=2, vdim=2, rot_dims=2, chunk=9), _moe(6, 3, 3))], logit_scale=1.0),
    _cfg([L(_mix(conv=6, chunk=20), _moe()), L(_mix(heads=2, kv_heads=1, dim=12, vdim=4, rot_dims=12, chunk=3, diff=0.9), _moe(40, 2, 1))])])
def test_one_and_two_layer_models(tmp_path, cfg):
    h = Harness(tmp_path, cfg)
    toks = _tokens(37, 50, 5)
    ref = h.oracle(toks)
    _close(h.step([("a", toks, range(len(toks)))], ["a"]), ref)                    # whole prompt
    _close(h.run_cut("b", toks, []), ref)                                          # token by token from the first token
    h.close()


# ------------------------------------------------------------------ the mixed model: cuts, batches, reuse
@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    h = Harness(tmp_path_factory.mktemp("mumasun"), MIXED, seed=3, slots=4, max_tokens=40 * PAGE)
    yield h
    h.close()


def test_residual_after_every_layer(mixed):
    toks = _tokens(17, 50, 6)
    want, got = [], []
    O.forward(mixed.cfg, mixed.W, toks, tap=lambda i, x: want.append(x.float()))
    mixed.model.layer_tap = lambda i, x: got.append(x.clone())
    try:
        mixed.step([("t", toks, [])], ["t"])
    finally:
        mixed.model.layer_tap = None
    assert len(got) == len(want) == 4
    for a, b in zip(got, want):
        torch.testing.assert_close(a.cpu(), b, rtol=1e-4, atol=1e-4)


def test_first_tokens_and_prefill_against_decode(mixed):
    toks = _tokens(61, 50, 7)
    ref = mixed.oracle(toks)
    whole = mixed.step([("w", toks, range(len(toks)))], ["w"])
    _close(whole, ref)
    _close(whole[:3], ref[:3], 1e-4)                                               # positions 0, 1, 2: one key, zeros before the convolution
    _close(mixed.run_cut("d", toks, [30]), ref)                                    # 30 at once, then 31 decode steps


@pytest.mark.parametrize("cuts", [[2, 2, 2, 3, 2], [7, 8, 9, 2, 16], [1, 2, 17, 2, 2, 23], [PAGE, PAGE, 2 * PAGE], [PAGE - 1, 2, PAGE + 1, 19], [12, 12, 7, 5], [11, 2, 11, 14]])
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


def test_generation_with_prompts_in_chunks_beside_decoding(tmp_path):
    """the scheduler cuts long prompts into chunks and runs them beside decode steps of other requests"""
    h = Harness(tmp_path, MIXED, seed=4, max_tokens=60 * PAGE, chunked_prefill_size=2 * PAGE, enable_mixed_chunk=True)
    prompts = [_tokens(n, 50, 70 + n) for n in (50, 4, 39)]
    outs = h.eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 8, "temperature": 0, "ignore_eos": True})
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(8):
            seq.append(int(h.oracle(seq)[-1].argmax()))
        assert o["output_ids"] == seq[len(p):]
    h.close()


def test_text_prompts_on_a_weights_only_folder(tmp_path):
    """a folder with only config.json and model.safetensors serves text through the byte tokenizer (what `cli generate` and the HTTP server do)"""
    h = Harness(tmp_path, _cfg([L(_mix(), _moe()), L(_mix(chunk=0), None)], vocab=300), seed=8)
    h.close()
    eng = sgl.Engine(model_path=h.dir, device="cpu", page_size=PAGE, max_total_tokens=256, max_running_requests=2, log_level="warning")
    out = eng.generate("hello there", {"max_new_tokens": 4, "temperature": 0.7, "top_k": 5, "ignore_eos": True})
    assert len(out["output_ids"]) == 4 and isinstance(out["text"], str)
    eng.shutdown()


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5])
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
