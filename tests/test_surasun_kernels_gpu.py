"""Surasun CUDA kernels against their fp32 PyTorch references (``ops/torch_ref.py``) and the engine on CUDA against the plain oracle."""
import numpy as np
import pytest
import torch

from sglang_b200 import ops
from sglang_b200.layers.gated_attention import scaled_inv_freq
from sglang_b200.ops import torch_ref

pytestmark = pytest.mark.gpu

DEV = "cuda"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def _need():
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    assert ops.load_native(), "the CUDA extension must be built on a GPU box"


def _i32(x, dev=DEV):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def _tol(dtype, f32=(1e-5, 1e-5), bf=(8e-3, 8e-3)):
    r, a = bf if dtype == torch.bfloat16 else f32
    return dict(rtol=r, atol=a)


def _dv(t):
    return None if t is None else t.to(DEV)


@BOTH
@pytest.mark.parametrize("S", [1, 2, 3, 4, 7, 16])
@pytest.mark.parametrize("W", [10, 250, 1024, 4100, 9000])
def test_stream_mix_norm(W, S, dtype):
    _need()
    g = torch.Generator().manual_seed(W + S)
    T = 6
    x, y = torch.randn(T, S, W, generator=g), torch.randn(T, W, generator=g).to(dtype)
    w, coef = (1 + 0.2 * torch.randn(W, generator=g)).to(dtype), torch.randn(S * S + 2 * S, generator=g) * 0.5
    t32, t = dict(rtol=1e-4, atol=1e-4), _tol(dtype, f32=(1e-4, 1e-4), bf=(1e-2, 1e-2))
    for centre in (True, False):
        x0, h0 = torch_ref.stream_mix_norm(x.clone(), y, coef, S, w, 1e-5, dtype, centre, None, None, True)
        xd = x.to(DEV)
        x1, h1 = ops.stream_mix_norm(xd, y.to(DEV), coef.to(DEV), S, w.to(DEV), 1e-5, dtype, centre)
        assert x1 is xd and h1.dtype == dtype
        torch.testing.assert_close(x1.cpu(), x0, **t32)
        torch.testing.assert_close(h1.cpu().float(), h0.float(), **t)
    keep = x.to(DEV)
    x1, h1 = ops.stream_mix_norm(keep, y.to(DEV), coef.to(DEV), S, w.to(DEV), 1e-5, dtype, False, keep=False)          # nothing is stored
    assert x1 is None and torch.equal(keep.cpu(), x)
    torch.testing.assert_close(h1.cpu().float(), h0.float(), **t)
    # streams that start as an embedding row: nothing added yet, then the first update
    table, ids = torch.randn(11, W, generator=g).to(dtype), [3, 10, 0, 3, 7, 1]
    for yy, kp in ((None, False), (y, True), (None, True)):
        x0, h0 = torch_ref.stream_mix_norm(None, yy, coef, S, w, 1e-5, dtype, True, table, _i32(ids, "cpu"), kp)
        x1, h1 = ops.stream_mix_norm(None, _dv(yy), coef.to(DEV), S, w.to(DEV), 1e-5, dtype, True, table.to(DEV), _i32(ids), kp)
        torch.testing.assert_close(h1.cpu().float(), h0.float(), **t)
        assert (x1 is None) == (not kp)
        if kp:
            torch.testing.assert_close(x1.cpu(), x0, **t32)


@BOTH
@pytest.mark.parametrize("parts,per", [(1, 96), (3, 7), (4, 32), (8, 130), (12, 256), (5, 1200), (40, 64)])
def test_grouped_norm_without_weight_and_with_silu_gate(parts, per, dtype):
    _need()
    g = torch.Generator().manual_seed(parts)
    C, T = parts * per, 9
    x, gate = torch.randn(T, C, generator=g) * 3, torch.randn(T, C + 11, generator=g).to(dtype)
    w = (1 + 0.3 * torch.randn(C, generator=g)).to(dtype)
    for at in (0, 3, 4):
        for ww, gg, act, sc in ((None, gate[:, at:at + C], "silu", 1.3), (w, gate[:, at:at + C], "sigmoid", 0.5), (None, None, "silu", 1.0), (w, None, "silu", 1.0)):
            ref = torch_ref.grouped_rmsnorm(x, ww, parts, 1e-5, dtype, gg, sc, act)
            buf = torch.full((T, C + 13), 5.0, dtype=dtype, device=DEV)
            gd = None if gg is None else gate.to(DEV)[:, at:at + C]
            ops.grouped_rmsnorm(x.to(DEV), _dv(ww), parts, 1e-5, dtype, gd, sc, buf[:, at:at + C], act)
            torch.testing.assert_close(buf[:, at:at + C].cpu().float(), ref.float(), **_tol(dtype))
            assert float(buf[:, at + C:].min()) == 5.0 and (at == 0 or float(buf[:, :at].min()) == 5.0)
            torch.testing.assert_close(ops.grouped_rmsnorm(x.to(DEV), _dv(ww), parts, 1e-5, dtype, gd, sc, None, act).cpu().float(), ref.float(), **_tol(dtype))


@BOTH
@pytest.mark.parametrize("H,G,D,Dv,rot", [(4, 2, 6, 5, 4), (3, 1, 7, 9, 6), (8, 2, 64, 48, 32), (6, 3, 30, 128, 30), (2, 2, 128, 128, 2)])
@pytest.mark.parametrize("inter", [True, False])
def test_attention_prepare(H, G, D, Dv, rot, inter, dtype):
    _need()
    g = torch.Generator().manual_seed(D)
    T = 23
    fr = scaled_inv_freq(rot, 5000.0)
    pos, loc = torch.randint(0, 3000, (T,), generator=g).int(), torch.randperm(60, generator=g)[:T].int()
    for extra, pad, norm in ((H, 0, True), (0, 128, True), (5, 0, False)):
        qkv = torch.randn(T, (H + G) * D + G * Dv + extra, generator=g).to(dtype)
        qw, kw = ((1 + 0.3 * torch.randn(n * D, generator=g)).to(dtype) if norm else None for n in (H, G))
        width = G * max(D, Dv, pad) + 4
        k0, v0 = (torch.full((60, 1, width), 9.0, dtype=dtype) for _ in range(2))
        k1, v1 = k0.to(DEV), v0.to(DEV)
        q0 = torch_ref.attention_prepare(qkv, H, G, D, Dv, pos, k0, v0, loc, qw, kw, 1e-5, fr, pad=pad, interleaved=inter)
        q1 = ops.attention_prepare(qkv.to(DEV), H, G, D, Dv, pos.to(DEV), k1, v1, loc.to(DEV), _dv(qw), _dv(kw), 1e-5, fr.to(DEV), pad=pad, interleaved=inter)
        for a, b in ((q1, q0), (k1, k0), (v1, v0)):
            torch.testing.assert_close(a.cpu().float(), b.float(), **_tol(dtype, f32=(2e-4, 2e-4), bf=(1e-2, 2e-2)))


@BOTH
@pytest.mark.parametrize("H,D,Dv,rot,inter,silu", [(3, 6, 4, 4, False, False), (2, 7, 9, 6, True, True), (4, 64, 32, 32, False, False), (4, 64, 32, 64, True, False),
                                                  (2, 256, 128, 256, False, True), (1, 5, 3, 0, False, False), (8, 16, 16, 4, True, False), (2, 12, 8, 6, False, False)])
def test_linear_attention_prepare(H, D, Dv, rot, inter, silu, dtype):
    _need()
    g = torch.Generator().manual_seed(D + rot)
    T, n = 19, H * (Dv + 2 * D)
    fr = scaled_inv_freq(rot, 1e5) if rot else None
    pos = torch.randint(0, 3000, (T,), generator=g).int()
    for at, tail in ((0, 0), (4, 8), (3, 6)):                              # a column view of a wider projection, aligned and not
        wide = torch.randn(T, at + n + tail, generator=g).to(dtype)
        ref = torch_ref.linear_attention_prepare(wide[:, at:], H, D, Dv, pos, fr, inter, D ** -0.5, silu)
        got = ops.linear_attention_prepare(wide.to(DEV)[:, at:], H, D, Dv, pos.to(DEV), _dv(fr), inter, D ** -0.5, silu)
        assert got.dtype == torch.float32
        torch.testing.assert_close(got.cpu(), ref, rtol=3e-4, atol=3e-4)   # sines of angles up to 3000 in fp32


@BOTH
def test_convolution_in_the_model_dtype(dtype):
    """the convolution without activation, its result rounded to the model dtype: ragged portions and decode steps on used slots"""
    _need()
    g = torch.Generator().manual_seed(2)
    C, K = 37, 4
    w, b = torch.randn(C, K, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype)
    st = torch.randn(5, C, K - 1, generator=g).to(dtype)
    sd, done = st.to(DEV), [0, 0, 0]
    for ql in ([5, 1, 200], [1, 2, 3], None):
        n = ql or [1] * 3
        done = [a + c for a, c in zip(done, n)]
        x = torch.randn(sum(n), C + 3, generator=g).to(dtype)
        cu = _i32([0, *np.cumsum(n).tolist()], "cpu") if ql else None
        slots, sl = _i32([4, 1, 2], "cpu"), _i32(done, "cpu")
        ref = torch_ref.causal_conv1d(x[:, 3:], w, b, st, cu, slots, sl, False)
        for od in {torch.float32, dtype}:
            s2 = sd.clone()
            got = ops.causal_conv1d(x.to(DEV)[:, 3:], w.to(DEV), b.to(DEV), s2, _dv(cu), slots.to(DEV), sl.to(DEV), max(n), False, od)
            assert got.dtype == od and torch.equal(s2.cpu(), st)
            torch.testing.assert_close(got.cpu().float(), ref, **(_tol(dtype) if od == dtype else dict(rtol=1e-5, atol=1e-5)))
        sd = s2


@pytest.mark.parametrize("T", [1, 33, 128, 300])
@pytest.mark.parametrize("nb,n", [(1, 32), (4, 80), (3, 64), (5, 256), (7, 48), (2, 16), (3, 24), (2, 7)])
def test_block_diagonal_product(T, nb, n):
    """the tcgen05 product against fp32 sums: blocks of whole and partial K steps, tiles at block borders, sizes that leave the route"""
    _need()
    g = torch.Generator().manual_seed(T + n)
    u, w = torch.randn(T, nb * n, generator=g).bfloat16(), (torch.randn(nb, 2 * n, n, generator=g) * n ** -0.5).bfloat16()
    ref = torch_ref.block_linear_f32(u, w)
    got = ops.block_linear_f32(u.to(DEV), w.to(DEV))
    assert got.dtype == torch.float32 and got.shape == ref.shape
    torch.testing.assert_close(got.cpu(), ref, rtol=1e-4, atol=1e-4)
    wide = torch.randn(T, nb * n + 16, generator=g).bfloat16().to(DEV)
    torch.testing.assert_close(ops.block_linear_f32(wide[:, 8:8 + nb * n], w.to(DEV)).cpu(), torch_ref.block_linear_f32(wide.cpu()[:, 8:8 + nb * n], w), rtol=1e-4, atol=1e-4)


@BOTH
@pytest.mark.parametrize("nb,n", [(1, 1), (3, 7), (4, 80), (2, 64), (10, 256)])
def test_gated_recurrence(nb, n, dtype):
    """ragged portions around the tile sizes, empty requests, decode steps, slots used before"""
    _need()
    g = torch.Generator().manual_seed(nb * n)
    C, B = nb * n, 5
    lam, gb = torch.randn(C, generator=g) * 2 - 2, torch.randn(nb, 2 * n, generator=g)
    st = torch.randn(8, 1, 1, C, generator=g)
    sd, done = st.to(DEV), [0] * B
    steps = [[1, 64, 200, 0, 7], [65, 2, 1, 129, 8], None, [8, 1, 63, 16, 300], None]
    for ql in steps:
        lens = ql or [1] * B
        done = [a + c for a, c in zip(done, lens)]
        T = sum(lens)
        gates = torch.randn(T, nb, 2 * n, generator=g) * 3
        u, y = torch.randn(T, C, generator=g).to(dtype), (torch.randn(T, C + 2, generator=g) * 2).to(dtype)
        slots, sl = _i32([4, 1, 7, 2, 3], "cpu"), _i32(done, "cpu")
        ref = torch_ref.rglru_scan(gates, gb, u, lam, y[:, :C], st, slots, sl, _i32(lens, "cpu"), torch.float32, nb)
        cu = _i32([0, *np.cumsum(lens).tolist()]) if ql else None
        got = ops.rglru_scan(gates.to(DEV), gb.to(DEV), u.to(DEV), lam.to(DEV), y.to(DEV)[:, :C], sd, slots.to(DEV), sl.to(DEV), cu, _i32(lens), nb)
        assert got.dtype == dtype
        torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype, f32=(1e-4, 2e-5)))
        torch.testing.assert_close(sd.cpu(), st, rtol=1e-4, atol=2e-5)                       # the state is fp32 in both


@BOTH
def test_gated_recurrence_at_the_ends_of_its_range(dtype):
    """decays next to 1 (the input's factor is a small root) and next to 0, saturated gates, large branch values; a long prompt through tiles"""
    _need()
    C, T = 64, 2000
    g = torch.Generator().manual_seed(1)
    lam = torch.linspace(-14, 6, C)
    gates = torch.randn(T, 1, 2 * C, generator=g) * 2
    gates[5:9] = 200.0
    gates[20:24] = -200.0
    u, y = torch.randn(T, C, generator=g).to(dtype), (torch.randn(T, C, generator=g) * 5).to(dtype)
    y[30], y[31] = 60.0, -60.0
    st = torch.zeros(1, 1, 1, C)
    sd = st.to(DEV)
    ref = torch_ref.rglru_scan(gates, None, u, lam, y, st, _i32([0], "cpu"), _i32([T], "cpu"), _i32([T], "cpu"), torch.float32, 1)
    got = ops.rglru_scan(gates.to(DEV), None, u.to(DEV), lam.to(DEV), y.to(DEV), sd, _i32([0]), _i32([T]), _i32([0, T]), _i32([T]), 1)
    assert torch.isfinite(got).all()
    # a decay of 1 - 1e-3 is itself rounded by 6e-8: over its memory of a thousand tokens that is 6e-5
    torch.testing.assert_close(sd.cpu(), st, rtol=3e-4, atol=2e-4)
    torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype, f32=(3e-4, 5e-4), bf=(8e-3, 1e-2)))


@pytest.mark.parametrize("outliers", [False, True])
@pytest.mark.parametrize("decode", [False, True])
def test_score_cap_on_the_tensor_core_kernels(decode, outliers):
    """scores that stay within the cap, and a few far beyond it in some rows only: both forms of the cap, in prompt tiles and in decode"""
    _need()
    g = torch.Generator().manual_seed(7)
    H, G, D, ps, cap = 8, 2, 128, 64, 9.0
    lens, cached = ([1] * 5, [130, 0, 400, 63, 64]) if decode else ([70, 1, 300, 64], [0, 99, 31, 200])
    tot = [a + b for a, b in zip(lens, cached)]
    per = (max(tot) + ps - 1) // ps
    pt = (torch.randperm(len(lens) * per, generator=g).int() + 1).view(len(lens), per)
    kc, vc = (torch.randn((len(lens) * per + 2) * ps, G, D, generator=g).bfloat16() for _ in range(2))
    q = torch.randn(sum(lens), H, D, generator=g)
    if outliers:
        q[::37] *= 12.0
    q = q.bfloat16()
    rows, sl, ql = _i32(list(range(len(lens))), "cpu"), _i32(tot, "cpu"), _i32(lens, "cpu")
    ref = torch_ref.window_attention(q.float(), kc.float().view(-1, 1, G * D), vc.float().view(-1, 1, G * D), G, D, pt, rows, sl, ql, ps, D ** -0.5, cap, -1, None, None, D)
    cu = None if decode else _i32([0, *np.cumsum(lens).tolist()])
    a = [t.to(DEV) for t in (q, kc, vc, pt, rows, sl, ql)]
    assert ops.tc_attention_ok(a[0], a[1], a[2], ps)
    for splits in ((1, 3) if decode else (1,)):
        got = ops.paged_attention(a[0], a[1], a[2], a[3], a[4], a[5], cu, a[6], max(lens), ps, D ** -0.5, logit_cap=cap, num_splits=splits)
        torch.testing.assert_close(got.cpu().float(), ref, rtol=3e-2, atol=2e-2)


@BOTH
@pytest.mark.parametrize("H,hs,Dv", [(3, 128, 48), (8, 64, 64), (5, 7, 7), (2, 128, 100)])
def test_sigmoid_gate(H, hs, Dv, dtype):
    _need()
    g = torch.Generator().manual_seed(H)
    T = 33
    o, wide = torch.randn(T, H, hs, generator=g).to(dtype), torch.randn(T, H * Dv + 8, generator=g).to(dtype)
    for gate in (wide[:, :H], wide[:, 8:], wide[:, 3:3 + H * Dv]):
        ref = ops.sigmoid_gate(o, gate, Dv, 0.7)
        buf = torch.full((T, H * Dv + 24), 5.0, dtype=dtype, device=DEV)
        for at in (0, 8, 3):
            at_gate = wide.to(DEV)[:, gate.storage_offset():gate.storage_offset() + gate.shape[1]]
            ops.sigmoid_gate(o.to(DEV), at_gate, Dv, 0.7, buf[:, at:at + H * Dv])
            torch.testing.assert_close(buf[:, at:at + H * Dv].cpu().float(), ref.float(), **_tol(dtype))
        assert float(buf[:, 8 + H * Dv:].min()) == 5.0


# ------------------------------------------------------------------ the engine
def _spread_error(x, ref):
    """per position: root mean square of the difference over the vocabulary (mean taken off) against that of the logits"""
    d, r = x - ref, ref - ref.mean(-1, keepdims=True)
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((r ** 2).mean(-1) + 1e-12)


def _rounding_limit(h, tokens):
    """what bf16 rounding may cost at every position: the oracle's own change when every weight moves by a random 2^-9 of itself (three draws).
    Positions differ widely: retention divides a head by its own root mean square, so where a query is nearly orthogonal to all it remembers
    (at position 0 that is one product) rounding may turn the head's sign"""
    import surasun_oracle as O

    ref, worst = h.oracle(tokens), 0.0
    for k in range(3):
        g = torch.Generator().manual_seed(k)
        W = {n: v * (1 + torch.randn(v.shape, generator=g) * 2.0 ** -9) for n, v in h.W.items()}
        worst = np.maximum(worst, _spread_error(O.forward(h.cfg, W, list(tokens)).float().numpy(), ref))
    return 0.03 + 3.0 * worst


def _steady(cfg, seed):
    """random weights whose retention keys lie near its queries, so that no head's read-out is nearly zero"""
    import surasun_oracle as O

    W, g = O.random_weights(cfg, seed), torch.Generator().manual_seed(seed + 1)
    for k in W:
        if k.endswith("right.k"):
            q = W[k[:-1] + "q"]
            W[k] = q + 0.3 * q.std() * torch.randn(q.shape, generator=g)
    return W


def _engine_case(tmp_path, dtype, cfg, seed, tol, gen=True, **kw):
    """whole prompts, portions, decoding, unequal batches and reuse on CUDA against the oracle.  fp32 bounds every logit by ``tol``; bf16 bounds the
    spread error of at least 97 % of the positions by ``_rounding_limit``, that of all by three times as much, and the mean by ``tol``"""
    from test_surasun import Harness, _tokens

    h = Harness(tmp_path, cfg, seed=seed, slots=4, max_tokens=1024, device="cuda", dtype=dtype, page=16, **kw)
    V = cfg["vocab"]
    a, b, c = _tokens(150, V, 1), _tokens(41, V, 2), _tokens(3, V, 3)
    ra, rb, rc = h.oracle(a), h.oracle(b), h.oracle(c)
    la, lb, lc = (_rounding_limit(h, t) if dtype == "bfloat16" else np.zeros(len(t)) for t in (a, b, c))
    errs, lims = [], []

    def close(x, y, lim):
        if dtype == "float32":
            err = np.abs(x - y).max() / max(1.0, float(np.sqrt((y ** 2).mean())))
            assert float(err) < tol, float(err)
            return
        errs.append(_spread_error(x, y))
        lims.append(lim)

    close(h.step([("a", a, range(len(a)))], ["a"]), ra, la)                                        # whole
    close(h.run_cut("a2", a, [100, 2, 17]), ra, la)                                                # portions, then token by token
    out = h.step([("a", a[:90], range(90)), ("b", b[:7], range(7)), ("c", c, range(3))], ["c"])    # unequal batch
    close(out[:90], ra[:90], la[:90]); close(out[90:97], rb[:7], lb[:7]); close(out[97:], rc, lc)
    out = h.step([("a", a[90:], range(60)), ("b", b[7:8], range(1))], ["a"])
    close(out[:60], ra[90:], la[90:]); close(out[60:], rb[7:8], lb[7:8])
    out = h.step([("b", b[8:], range(len(b) - 8)), ("d", c, range(3))], ["b", "d"])                # "d" reuses a freed slot and pages
    close(out[:len(b) - 8], rb[8:], lb[8:]); close(out[len(b) - 8:], rc, lc)
    if errs:
        err, lim = np.concatenate(errs), np.concatenate(lims)
        over = err / lim
        assert float((over > 1).mean()) <= 0.03 and float(over.max()) < 3 and float(err.mean()) < tol, (float((over > 1).mean()), float(over.max()), float(err.mean()))
    if dtype == "float32" and gen:  # greedy generation through the engine's own entry point, scheduler and sampler
        prompts = [b[:9], c]
        outs = h.eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 6, "temperature": 0, "ignore_eos": True})
        for pr, o in zip(prompts, outs):
            seq = list(pr)
            for _ in range(6):
                seq.append(int(h.oracle(seq)[-1].argmax()))
            assert o["output_ids"] == seq[len(pr):]
    h.close()


def _wide():
    """lane-friendly sizes: bf16 attention with groups of 4 and 1 takes the tcgen05 kernels, the one with three query heads per key head the
    general kernel; gate blocks of 64 and 48 take the tcgen05 product"""
    from test_surasun import L, _cfg, _lru, _m2, _par

    return _cfg([L(_lru(width=192, blocks=3), 128), L(_par(heads=8, kv_heads=2, dim=64, vdim=96, rot=32, base=1e4, scale=0.2, cap=12.0, rh=4, rd=32, rv=48, rrot=32,
                                                           decay=(0.9, 0.99, 0.999, 1.0)), 96),
                 L(_m2(heads=8, vdim=32, state=48, groups=2, norm_groups=4, conv=4)), L(_par(heads=6, kv_heads=2, dim=32, vdim=32, rot=8, rh=2, rd=64, rv=32, rrot=16,
                                                                                            decay=(0.95, 0.995))),
                 L(_lru(width=96, blocks=2, conv=3)), L(_par(heads=2, kv_heads=2, dim=128, vdim=128, rot=128, scale=0.1, cap=20.0, rh=1, rd=16, rv=16, rrot=16, decay=(0.97,)), 64)],
                width=128, vocab=256, streams=3, mult=0.5)


def test_engine_on_cuda_fp32(tmp_path):
    from test_surasun import MIXED

    _need()
    _engine_case(tmp_path, "float32", MIXED, 1, 3e-4)


def test_engine_on_cuda_bf16(tmp_path):
    from test_surasun import MIXED

    _need()
    _engine_case(tmp_path, "bfloat16", MIXED, 2, 0.06, weights=_steady(MIXED, 2))


def test_engine_on_cuda_lane_friendly_sizes_fp32(tmp_path):
    _need()
    _engine_case(tmp_path, "float32", _wide(), 3, 3e-4)


def test_engine_on_cuda_lane_friendly_sizes_bf16(tmp_path):
    _need()
    _engine_case(tmp_path, "bfloat16", _wide(), 4, 0.04, weights=_steady(_wide(), 4))


def test_tensor_core_routes_agree_with_the_general_kernels(tmp_path, monkeypatch):
    from sglang_b200.layers.gated_attention import GatedAttention
    from test_surasun import Harness

    _need()
    h = Harness(tmp_path, _wide(), seed=5, slots=2, max_tokens=512, device="cuda", dtype="bfloat16", page=16)
    pads = [b.attention().pad for b in h.model.model.all_layers if b.attention() is not None]
    h.close()
    assert pads == [128, 0, 128]
    monkeypatch.setattr(GatedAttention, "tc_route", False)
    monkeypatch.setattr(ops, "DIAG_TC", False)
    _engine_case(tmp_path / "general", "bfloat16", _wide(), 5, 0.04, weights=_steady(_wide(), 5))


@pytest.mark.parametrize("seed", [11, 12, 13, 14])
def test_engine_on_cuda_randomly_drawn_stacks_fp32(tmp_path, seed):
    from test_surasun import drawn_config

    _need()
    _engine_case(tmp_path, "float32", drawn_config(seed, friendly=seed % 2 == 0), seed, 2e-3, gen=False)


@pytest.mark.parametrize("seed", [21, 22, 31, 32])
def test_engine_on_cuda_randomly_drawn_stacks_bf16(tmp_path, seed):
    """friendly sizes, and sizes that are no multiples of the vector widths: every kernel takes its scalar path, the GEMMs their general one"""
    from test_surasun import drawn_config

    _need()
    _engine_case(tmp_path, "bfloat16", drawn_config(seed, friendly=seed < 30), seed, 0.08)


def test_captured_decode_steps_agree_with_eager_ones(tmp_path):
    """greedy bf16 generation with CUDA graphs (padded batch sizes, slots that are used again) against the same engine without them"""
    from test_surasun import Harness, _tokens

    _need()
    cfg = _wide()
    prompts = [_tokens(n, 256, 300 + n) for n in (70, 3, 25, 44, 1, 60, 47)]
    sp = {"max_new_tokens": 40, "temperature": 0, "ignore_eos": True}
    outs = []
    for graphs in (True, False):
        h = Harness(tmp_path / str(graphs), cfg, seed=6, slots=3, max_tokens=1024, device="cuda", dtype="bfloat16", page=16, disable_cuda_graph=not graphs)
        r = h.sched.worker.runner if hasattr(h.sched.worker, "runner") else h.sched.worker
        assert bool(r.graphs) == graphs
        outs.append([o["output_ids"] for o in h.eng.generate(input_ids=prompts, sampling_params=sp)])
        assert (r.graph_launches > 0) == graphs
        h.sched.check_invariants()
        h.close()
    assert outs[0] == outs[1]
