"""Mumasun CUDA kernels against their fp32 PyTorch references (``ops/torch_ref.py``) and the engine on CUDA against the plain oracle."""
import numpy as np
import pytest
import torch

from sglang_b200 import ops
from sglang_b200.layers.latent_attention import yarn_inv_freq
from sglang_b200.ops import moe_ops, torch_ref

pytestmark = pytest.mark.gpu

DEV = "cuda"


def _need():
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    assert ops.load_native(), "the CUDA extension must be built on a GPU box"


def _i32(x, dev=DEV):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def _tol(dtype, f32=(1e-5, 1e-5), bf=(2e-2, 2e-2)):
    r, a = bf if dtype == torch.bfloat16 else f32
    return dict(rtol=r, atol=a)


def _pages(n_req, max_len, ps, g):
    """page table whose pages lie scattered over the pool; rows 1 .. n_req"""
    per = (max_len + ps - 1) // ps
    n_pages = n_req * per + 3
    pt = torch.zeros(n_req + 1, per + 1, dtype=torch.int32)
    perm = torch.randperm(n_pages - 1, generator=g) + 1
    for r in range(n_req):
        pt[r + 1, :per] = perm[r * per:(r + 1) * per].int()
    return pt, n_pages


def _slots(pt, row, positions, ps):
    return [int(pt[row, p // ps]) * ps + p % ps for p in positions]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [24, 250, 1024, 5000])
def test_norm_add(dtype, W):
    _need()
    g = torch.Generator().manual_seed(W)
    x, y = torch.randn(7, W, generator=g), torch.randn(7, W, generator=g).to(dtype)
    w = (torch.randn(W, generator=g) * 0.2).to(dtype)
    for zc in (True, False):
        r = x.clone()
        ref = torch_ref.norm_add_f32(r, y, w, 1e-5, zc, dtype)
        gx, gh = ops.norm_add_f32(x.clone().to(DEV), y.to(DEV), w.to(DEV), 1e-5, zc, dtype)
        torch.testing.assert_close(gx.cpu(), r, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(gh.cpu().float(), ref.float(), **_tol(dtype, bf=(8e-3, 1e-3)))
        assert gh.dtype == dtype and (dtype != torch.float32 or gh is gx)
    table, ids = torch.randn(11, W, generator=g).to(dtype), _i32([3, 10, 0, 3])
    r = torch.empty(4, W)
    torch_ref.norm_add_f32(r, table, w, 1e-5, True, dtype, ids.cpu())
    gx, gh = ops.norm_add_f32(None, table.to(DEV), w.to(DEV), 1e-5, True, dtype, ids)
    torch.testing.assert_close(gx.cpu(), r, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(gh.cpu().float(), r, **_tol(dtype, bf=(8e-3, 1e-3)))


@pytest.mark.parametrize("E,K", [(1, 1), (8, 1), (8, 8), (40, 3), (300, 32), (2048, 2)])
def test_sigmoid_route(E, K):
    _need()
    g = torch.Generator().manual_seed(E + K)
    z = torch.randn(33, E, generator=g) * 3
    z[5] += 60.0                                                       # saturated scores: the choice still follows the logits
    for renorm, scale in ((False, 1.0), (True, 2.5)):
        w0, i0 = torch_ref.sigmoid_route(z, K, renorm, scale)
        w1, i1 = moe_ops.sigmoid_route(z.to(DEV), K, renorm, scale)
        assert torch.equal(i1.cpu(), i0)
        torch.testing.assert_close(w1.cpu(), w0, rtol=1e-5, atol=1e-7)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,W,I,E,K", [(1, 64, 32, 4, 1), (5, 96, 64, 6, 2), (300, 256, 96, 8, 1), (700, 128, 160, 5, 5), (40, 72, 40, 3, 2)])
def test_experts_with_weighted_inputs(T, W, I, E, K, dtype):
    _need()
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, W, generator=g).to(dtype)
    w1, w2 = (torch.randn(E, I, W, generator=g) * W ** -0.5).to(dtype), (torch.randn(E, W, I, generator=g) * I ** -0.5).to(dtype)
    rw, ids = torch_ref.sigmoid_route(torch.randn(T, E, generator=g) * 2, K)
    for win in (True, False):
        act = lambda u: torch.relu(u.float()).square()
        ref = torch_ref.fused_moe(x.float(), w1.float(), w2.float(), rw, ids, 0, act, win)
        got = moe_ops.fused_moe(x.to(DEV), w1.to(DEV), w2.to(DEV), rw.to(DEV), ids.to(DEV), 0, ("relu2",), win)
        assert got.dtype == dtype
        torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype, f32=(1e-4, 1e-4), bf=(3e-2, 5e-2)))
    a = moe_ops.fused_moe(x.to(DEV), w1.to(DEV), w2.to(DEV), rw.to(DEV), ids.to(DEV), 0, ("relu2",), True)
    b = moe_ops.fused_moe(x[:1].to(DEV), w1.to(DEV), w2.to(DEV), rw[:1].to(DEV), ids[:1].to(DEV), 0, ("relu2",), True)
    torch.testing.assert_close(a[:1].float(), b.float(), **_tol(dtype, f32=(1e-5, 1e-5), bf=(2e-2, 2e-2)))          # what else is in the batch does not matter


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,M,D,Dv,rot,taps,pad", [(4, 2, 2, 64, 128, 64, 3, 0), (4, 2, 2, 64, 128, 64, 3, 128), (6, 3, 2, 24, 40, 16, 2, 128), (3, 1, 2, 7, 9, 6, 5, 0),
                                                     (2, 2, 2, 130, 200, 20, 4, 0), (2, 1, 1, 16, 16, 0, 1, 0), (4, 4, 2, 33, 65, 0, 16, 0), (2, 1, 1, 100, 96, 100, 4, 128), (2, 1, 2, 12, 72, 8, 4, 0), (3, 1, 1, 64, 100, 64, 1, 0), (5, 5, 2, 4, 4, 0, 4, 0)])
def test_conv_attention_prepare(H, G, M, D, Dv, rot, taps, pad, dtype):
    """ragged portions (single tokens among them, cached history, empty requests), then decode steps of all requests: q rows, cache rows and state"""
    _need()
    if pad and D > pad // M:
        pytest.skip("does not fit the padded layout")
    g = torch.Generator().manual_seed(H * 100 + D)
    C, ps = (H + G) * M * D + G * Dv, 8
    seg, wv = (pad // M, pad) if pad else (D, Dv)
    width = max(G * M * seg, G * wv) + 3
    width += -width % 8
    f, mult = yarn_inv_freq(rot, 500.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}) if rot else (None, 1.0)
    w = (torch.randn(C, taps, generator=g) * 0.5).to(dtype)
    nq, nk = (torch.rand(D, generator=g) + 0.5).to(dtype), (torch.rand(D, generator=g) + 0.5).to(dtype)
    pt, n_pages = _pages(5, 400, ps, g)
    mk = lambda: (torch.full((n_pages * ps, 1, width), 0.25, dtype=dtype), torch.full((n_pages * ps, 1, width), 0.25, dtype=dtype))
    (k0, v0), st0 = mk(), torch.randn(7, C, max(1, taps - 1), generator=g).to(dtype)          # a used pool and state: fresh requests must not see it
    k1, v1, st1 = k0.to(DEV), v0.to(DEV), st0.to(DEV)
    done = [0, 0, 0, 0, 0]
    steps = [[40, 1, 0, 3, 2], [1, 17, 2, 0, 300], [5, 2, 1, 1, 3]] + [None] * 3                # None: one token of every request (decode layout)
    if dtype == torch.float32:
        steps += [[2, 90, 1, 1, 1]]
    for n_step, lens in enumerate(steps):
        ql = lens or [1] * 5
        T = sum(ql)
        x = torch.randn(T, C + 5, generator=g).to(dtype)[:, :C] if n_step % 2 else torch.randn(T, C, generator=g).to(dtype)
        pos = [p for b in range(5) for p in range(done[b], done[b] + ql[b])]
        loc = [s for b in range(5) for s in _slots(pt, b + 1, range(done[b], done[b] + ql[b]), ps)]
        done = [a + b for a, b in zip(done, ql)]
        cu = _i32(np.concatenate([[0], np.cumsum(ql)]).tolist()) if lens else None
        slots, sl = _i32([1, 4, 2, 6, 3]), _i32(done)
        c = lambda t: None if t is None else t.cpu()
        args = lambda dev: (f if dev == "cpu" or f is None else f.to(DEV), mult)
        q0 = torch_ref.conv_attention_prepare(x, H, G, M, D, Dv, w, st0, _i32(pos, "cpu"), c(cu), c(slots), c(sl), nq, nk, 1e-5, *args("cpu"), k0, v0, _i32(loc, "cpu"), pad)
        q1 = ops.conv_attention_prepare(x.to(DEV) if x.is_contiguous() else torch.nn.functional.pad(x, (0, 5)).to(DEV)[:, :C], H, G, M, D, Dv, w.to(DEV), st1, _i32(pos), cu,
                                        slots, sl, nq.to(DEV), nk.to(DEV), 1e-5, *args("cuda"), k1, v1, _i32(loc), pad)
        t = _tol(dtype, f32=(2e-4, 2e-4), bf=(1e-2, 1e-2))
        torch.testing.assert_close(q1.cpu().float(), q0.float(), **t)
        torch.testing.assert_close(k1.cpu().float(), k0.float(), **t)
        torch.testing.assert_close(v1.cpu().float(), v0.float(), **t)
        if taps > 1:
            assert torch.equal(st1.cpu(), st0), n_step                        # the state holds projections: moved, never computed


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("lens", [[2700], [1, 900, 3, 0, 1501, 40, 2, 310], [5] * 520])
def test_conv_attention_prepare_long_batches(lens, dtype):
    """long runs of tokens per CTA: requests that begin and end inside a run and inside a group of four rows"""
    _need()
    g = torch.Generator().manual_seed(len(lens))
    H, G, D, Dv, rot, taps, B, T = 2, 1, 8, 12, 8, 4, len(lens), sum(lens)
    C = 2 * (H + G) * D + G * Dv
    x, w = torch.randn(T, C, generator=g).to(dtype), (torch.randn(C, taps, generator=g) * 0.5).to(dtype)
    st0 = torch.randn(B + 1, C, taps - 1, generator=g).to(dtype)
    st1, f = st0.to(DEV), yarn_inv_freq(rot, 500.0)[0]
    cached = [(3 * i) % 5 for i in range(B)]
    pos = _i32([c + i for c, n in zip(cached, lens) for i in range(n)], "cpu")
    k0 = [torch.zeros(T + 3, 1, 16, dtype=dtype) for _ in range(2)]
    k1 = [t.to(DEV) for t in k0]
    loc = torch.randperm(T, generator=g).int() + 3
    cu, sl, slots = _i32(np.concatenate([[0], np.cumsum(lens)]).tolist(), "cpu"), _i32([a + b for a, b in zip(lens, cached)], "cpu"), torch.randperm(B, generator=g).int() + 1
    nq, nk = (torch.rand(D, generator=g) + 0.5).to(dtype), (torch.rand(D, generator=g) + 0.5).to(dtype)
    q0 = torch_ref.conv_attention_prepare(x, H, G, 2, D, Dv, w, st0, pos, cu, slots, sl, nq, nk, 1e-5, f, 1.1, *k0, loc)
    c = lambda t: t.to(DEV)
    q1 = ops.conv_attention_prepare(c(x), H, G, 2, D, Dv, c(w), st1, c(pos), c(cu), c(slots), c(sl), c(nq), c(nk), 1e-5, c(f), 1.1, *k1, c(loc))
    t = _tol(dtype, f32=(1e-3, 1e-3), bf=(1e-2, 1e-2))
    for a, b in ((q1, q0), (k1[0], k0[0]), (k1[1], k0[1])):
        torch.testing.assert_close(a.cpu().float(), b.float(), **t)
    assert torch.equal(st1.cpu(), st0)


def _attention_case(H, G, D, Dv, lens, cached, ps, chunk, dtype, tc, seed=0, decode=False, splits=1):
    """differential attention over a paged cache of random rows: (kernel result, fp32 reference), both [T, H, Dv]"""
    g = torch.Generator().manual_seed(seed)
    M, pad = 2, 128 if tc else 0
    seg, wv = (64, 128) if tc else (D, Dv)
    B, T = len(lens), sum(lens)
    tot = [a + b for a, b in zip(lens, cached)]
    pt, n_pages = _pages(B, max(tot), ps, g)
    width = G * 128 + 16 if tc else max(G * M * D, G * Dv)
    kc, vc = torch.zeros(n_pages * ps, 1, width), torch.zeros(n_pages * ps, 1, width)
    for m in range(G * M):
        kc[:, 0, m * seg:m * seg + D] = torch.randn(n_pages * ps, D, generator=g)
    for m in range(G):
        vc[:, 0, m * wv:m * wv + Dv] = torch.randn(n_pages * ps, Dv, generator=g)
    q = torch.zeros(T, H, M, M, seg)
    for m in range(M):
        q[:, :, m, m, :D] = torch.randn(T, H, D, generator=g)
    q = q.view(T, H * M, M * seg).to(dtype)
    kc, vc = kc.to(dtype), vc.to(dtype)
    rows, sl, ql = _i32(list(range(1, B + 1)), "cpu"), _i32(tot, "cpu"), _i32(lens, "cpu")
    diff, scale = (0.7, 0.6, 1e-5), D ** -0.5
    ref = torch_ref.window_attention(q.float(), kc.float(), vc.float(), G, Dv, pt, rows, sl, ql, ps, scale, 0.0, -1, None, None, 2 * seg, pad, chunk=chunk, diff=diff)
    cu = None if decode else _i32(np.concatenate([[0], np.cumsum(lens)]).tolist())
    a = [t.to(DEV) for t in (q, kc, vc, pt, rows, sl, ql)]
    if tc:
        k4, v4 = (t[:, 0, :G * 128].unflatten(-1, (G, 128)) for t in a[1:3])
        assert ops.tc_attention_ok(a[0], k4, v4, ps)
        got = ops.paged_attention(a[0], k4, v4, a[3], a[4], a[5], cu, a[6], max(lens), ps, scale, num_splits=splits, chunk=chunk, diff=diff, diff_dv=Dv)
    else:
        got = ops.window_attention(a[0], a[1], a[2], G, Dv, a[3], a[4], a[5], cu, a[6], max(lens), ps, scale, dim=2 * D, chunk=chunk, diff=diff)
    return got.cpu().float(), ref


CHUNKS = (0, 48, 64, 100, 1000)


@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 32, 48), (6, 1, 9, 7), (3, 3, 100, 130), (40, 2, 16, 16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_general_attention_kernel(H, G, D, Dv, dtype, chunk):
    _need()
    for lens, cached, dec in (([70, 1, 130, 5], [0, 99, 30, 62], False), ([1] * 5, [0, 47, 48, 199, 63], True)):
        got, ref = _attention_case(H, G, D, Dv, lens, cached, 16, chunk, dtype, False, seed=H, decode=dec)
        torch.testing.assert_close(got, ref, **_tol(dtype, f32=(2e-4, 2e-5), bf=(3e-2, 1.5e-2)))


@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 128), (16, 4, 64, 128), (2, 2, 32, 40), (8, 1, 48, 33), (32, 1, 64, 64)])
def test_tensor_core_kernels(H, G, D, Dv, chunk):
    """the tcgen05 kernels (prompt tiles, decode with and without split keys; group sizes that take the query-major kernel in decode) against the
    reference"""
    _need()
    tol = dict(rtol=4e-2, atol=4e-2)
    for ps in (16, 64):
        got, ref = _attention_case(H, G, D, Dv, [150, 1, 333, 5], [0, 99, 130, 62], ps, chunk, torch.bfloat16, True, seed=H)
        torch.testing.assert_close(got, ref, **tol)
    for splits in (1, 4):
        got, ref = _attention_case(H, G, D, Dv, [1] * 6, [0, 47, 48, 799, 63, 300], 64, chunk, torch.bfloat16, True, seed=H, decode=True, splits=splits)
        torch.testing.assert_close(got, ref, **tol)


def test_tensor_core_kernels_many_items():
    """more work items than resident CTAs: the persistent launches, with pairs of maps and chunk edges inside tiles"""
    _need()
    got, ref = _attention_case(16, 4, 64, 128, [400, 300, 513, 2, 250], [0, 100, 31, 700, 5], 64, 96, torch.bfloat16, True, seed=1)
    torch.testing.assert_close(got, ref, rtol=4e-2, atol=4e-2)
    got, ref = _attention_case(8, 8, 64, 96, [1] * 60, [(37 * i) % 500 for i in range(60)], 64, 200, torch.bfloat16, True, seed=2, decode=True)
    torch.testing.assert_close(got, ref, rtol=4e-2, atol=4e-2)


@pytest.mark.parametrize("dtype,D,Dv,tc", [(torch.float32, 4, 6, False), (torch.bfloat16, 48, 72, True), (torch.bfloat16, 64, 128, True), (torch.bfloat16, 72, 40, False)])
def test_chunk_edges_and_far_keys_on_the_kernels(dtype, D, Dv, tc):
    from test_mumasun import LayerBench, check_chunk_edges

    _need()
    assert (LayerBench(2, 1, D, Dv, 1.0, 0.3, dtype=dtype).m.pad == 128) == tc
    check_chunk_edges(DEV, dtype, 16, D, Dv, 2e-3 if dtype == torch.float32 else 4e-2)


def _engine_case(tmp_path, dtype, cfg, seed, tol, gen=True, quantile=1.0, **kw):
    """whole prompts, portions, decoding, unequal batches and reuse on CUDA against the oracle.  fp32 bounds every logit; bf16 bounds, per position, the
    root mean square of the difference over the vocabulary against that of the logits.  ``quantile`` < 1: stacks of tiny or drawn sizes, where in
    bf16 a router's close call may fall the other way or a norm over a handful of numbers is badly conditioned: that quantile is bounded, and
    the mean"""
    from test_mumasun import Harness, _tokens

    h = Harness(tmp_path, cfg, seed=seed, slots=4, max_tokens=1024, device="cuda", dtype=dtype, page=16, **kw)
    V = cfg["vocab"]
    a, b, c = _tokens(150, V, 1), _tokens(41, V, 2), _tokens(3, V, 3)
    ra, rb, rc = h.oracle(a), h.oracle(b), h.oracle(c)
    errs = []

    def close(x, y):
        if dtype == "float32":
            err = np.abs(x - y).max() / max(1.0, float(np.sqrt((y ** 2).mean())))
            assert float(err) < tol, float(err)
            return
        d, r = x - y, y - y.mean(-1, keepdims=True)
        d = d - d.mean(-1, keepdims=True)
        errs.append(np.sqrt((d ** 2).mean(-1)) / np.sqrt((r ** 2).mean(-1) + 1e-12))

    close(h.step([("a", a, range(len(a)))], ["a"]), ra)                                            # whole
    close(h.run_cut("a2", a, [100, 2, 17]), ra)                                                    # portions, then token by token
    out = h.step([("a", a[:90], range(90)), ("b", b[:7], range(7)), ("c", c, range(3))], ["c"])    # unequal batch
    close(out[:90], ra[:90]); close(out[90:97], rb[:7]); close(out[97:], rc)
    out = h.step([("a", a[90:], range(60)), ("b", b[7:8], range(1))], ["a"])
    close(out[:60], ra[90:]); close(out[60:], rb[7:8])
    out = h.step([("b", b[8:], range(len(b) - 8)), ("d", c, range(3))], ["b", "d"])                # "d" reuses a freed slot and pages
    close(out[:len(b) - 8], rb[8:]); close(out[len(b) - 8:], rc)
    if errs:
        err = np.concatenate(errs)
        assert float(np.quantile(err, quantile)) < tol and float(err.mean()) < 0.5 * tol, (float(np.quantile(err, quantile)), float(err.mean()), float(err.max()))
    if dtype == "float32" and gen:  # greedy generation through the engine's own entry point, scheduler and sampler
        prompts = [b[:9], c]
        outs = h.eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 6, "temperature": 0, "ignore_eos": True})
        for pr, o in zip(prompts, outs):
            seq = list(pr)
            for _ in range(6):
                seq.append(int(h.oracle(seq)[-1].argmax()))
            assert o["output_ids"] == seq[len(pr):]
    h.close()


def _wide(choose=True):
    """``choose=False``: every expert is taken, so that no close call of a router can fall either way in bf16 (a token that takes another expert differs
    from then on, and so does all that attends to it); "last": only the last layer chooses.  Lane-friendly sizes: bf16 layers with map pairs in groups of 8, 2 and 4 take the tcgen05 kernels, the ones with three query heads per key head or
    wide maps the general kernel"""
    from test_mumasun import L, _cfg, _mix, _moe

    t = lambda ff, experts, top: _moe(ff, experts, top) if choose is True else _moe(ff, 3, 3)
    return _cfg([L(_mix(heads=8, kv_heads=2, dim=64, vdim=128, rot_dims=64, base=1e4, scale=0.2, chunk=48), t(64, 8, 1)),
                 L(_mix(heads=2, kv_heads=2, dim=48, vdim=64, rot_dims=32, base=1e4, scale=0.2, chunk=100, conv=2), t(96, 4, 2)),
                 L(_mix(heads=6, kv_heads=2, dim=32, vdim=48, rot_dims=8, scale=0.25, chunk=30), None),
                 L(_mix(heads=4, kv_heads=2, dim=96, vdim=64, rot_dims=96, scale=0.1, chunk=0, conv=4), _moe(64, 8, 1) if choose == "last" else _moe(40, 3, 3))], width=128, vocab=256)


def test_engine_on_cuda_fp32(tmp_path):
    from test_mumasun import MIXED

    _need()
    _engine_case(tmp_path, "float32", MIXED, 1, 3e-4)


def test_engine_on_cuda_bf16(tmp_path):
    from test_mumasun import MIXED

    _need()
    _engine_case(tmp_path, "bfloat16", MIXED, 2, 0.2, quantile=0.9)


def test_engine_on_cuda_lane_friendly_sizes_fp32(tmp_path):
    _need()
    _engine_case(tmp_path, "float32", _wide(), 3, 3e-4)


def test_engine_on_cuda_lane_friendly_sizes_bf16(tmp_path):
    _need()
    _engine_case(tmp_path, "bfloat16", _wide(choose=False), 4, 0.06)
    _engine_case(tmp_path / "choice", "bfloat16", _wide(choose="last"), 4, 0.06, quantile=0.9)


def test_tensor_core_route_agrees_with_the_general_kernel(tmp_path, monkeypatch):
    from sglang_b200.layers.differential_attention import DifferentialAttention
    from test_mumasun import Harness

    _need()
    h = Harness(tmp_path, _wide(), seed=5, slots=2, max_tokens=512, device="cuda", dtype="bfloat16", page=16)
    pads = [b.mix.pad for b in h.model.model.all_layers]
    h.close()
    assert pads == [128, 128, 0, 0]
    monkeypatch.setattr(DifferentialAttention, "tc_route", False)
    _engine_case(tmp_path / "general", "bfloat16", _wide(choose=False), 5, 0.06)


@pytest.mark.parametrize("seed", [11, 12, 13, 14])
def test_engine_on_cuda_randomly_drawn_stacks_fp32(tmp_path, seed):
    from test_mumasun import drawn_config

    _need()
    _engine_case(tmp_path, "float32", drawn_config(seed, friendly=seed % 2 == 0), seed, 2e-3, gen=False)


@pytest.mark.parametrize("seed", [21, 22, 31, 32])
def test_engine_on_cuda_randomly_drawn_stacks_bf16(tmp_path, seed):
    """friendly sizes, and sizes that are no multiples of the vector widths: every kernel takes its scalar path, the GEMMs their general one"""
    from test_mumasun import drawn_config

    _need()
    _engine_case(tmp_path, "bfloat16", drawn_config(seed, friendly=seed < 30), seed, 0.25, quantile=0.9)


def test_captured_decode_steps_agree_with_eager_ones(tmp_path):
    """greedy bf16 generation with CUDA graphs (padded batch sizes, slots that are used again) against the same engine without them"""
    from test_mumasun import Harness, _tokens

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
