"""Plain float64 oracle of the Mumasun design, written from its equations: one function per mechanism, whole sequences at once.  Shares no
code with the serving path."""
import math
import zlib

import torch

F64 = torch.float64


# ------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored around zero"""
    return unit_rms(x, eps) * (1.0 + w)


def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w_j u_(t - taps + 1 + j), zeros before the first token"""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def frequencies(base, dims, sc=None):
    """-> (frequencies, factor on sine and cosine); ``sc`` blends every frequency with itself over ``factor`` along a ramp over its index"""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def index_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, freqs, mult):
    """x [T, ..., n] at positions 0 .. T - 1: coordinate i < h paired with i + h, h = len(freqs); what lies behind 2 h stays"""
    h = len(freqs)
    a = torch.arange(x.shape[0], dtype=F64).view(-1, *[1] * (x.dim() - 1)) * torch.tensor(freqs, dtype=F64)
    c, s = torch.cos(a) * mult, torch.sin(a) * mult
    u, v = x[..., :h], x[..., h:2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], -1)


def visible(T, chunk):
    """[T, T]: query i, key j: not later, and in the same stretch of ``chunk`` positions"""
    i, j = torch.arange(T).view(-1, 1), torch.arange(T).view(1, -1)
    ok = j <= i
    if chunk:
        ok = ok & (i // chunk == j // chunk)
    return ok


def lam(W, p, m):
    dot = lambda a, b: float((W[p + a] * W[p + b]).sum())
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + float(m["diff"])


def combine(a1, a2, lam_, diff, eps):
    """the two maps' outputs [..., Dv] of a head"""
    return unit_rms(a1 - lam_ * a2, eps) * (1.0 - diff)


def attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = unit_rms(q.view(T, H, 2, D), eps) * W[p + "q.norm"]
    k = unit_rms(k.view(T, G, 2, D), eps) * W[p + "k.norm"]
    v = v.view(T, G, Dv)
    rot = m.get("rot")
    if rot:
        f, mult = frequencies(float(rot["base"]), int(rot["dims"]), rot.get("scaling"))
        q, k = turn(q, f, mult), turn(k, f, mult)
    hide = ~visible(T, int((m.get("mask") or {}).get("size") or 0))
    la = lam(W, p, m)
    o = torch.zeros(T, H, Dv, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        a = [torch.softmax((q[:, hd, i] @ k[:, g, i].T * float(m["scale"])).masked_fill(hide, -math.inf), -1) @ v[:, g] for i in (0, 1)]
        o[:, hd] = combine(a[0], a[1], la, float(m["diff"]), eps)
    return o.reshape(T, H * Dv) @ W[p + "o"].T


def experts(h, W, p, mlp):
    E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    s = torch.sigmoid(h @ W[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.argsort(s[t], descending=True)[:top].tolist():
            x = s[t, e] * h[t]                                              # the weight enters the expert, it does not scale what comes out
            out[t] += W[p + f"e{e}.down"] @ torch.relu(W[p + f"e{e}.up"] @ x) ** 2
    return out


# ------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, tap=None):
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = centred_norm(W["embed"][torch.tensor(tokens)], W["embed.norm"], eps)
    for i, sp in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + centred_norm(attention(x, W, p + "mix.", sp["mixer"], eps), W[p + "norm1"], eps)
        if sp.get("mlp"):
            x = x + centred_norm(experts(x, W, p + "mlp.", sp["mlp"]), W[p + "norm2"], eps)
        if tap is not None:
            tap(i, x)
    return centred_norm(x, W["final.norm"], eps) @ W["embed"].T * float(cfg["logit_scale"])


def random_weights(cfg, seed=0):
    """fp32 tensors under the checkpoint names"""
    def rnd(name, *shape, s=1.0, off=0.0):
        g = torch.Generator().manual_seed((seed * 7919 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
        return torch.randn(*shape, generator=g) * s + off

    W, width = {}, int(cfg["width"])

    def lin(name, o, i, s=1.0):
        W[name] = rnd(name, o, i, s=s * i ** -0.5)

    def vec(name, n, s, off=0.0):
        W[name] = rnd(name, n, s=s, off=off)

    W["embed"] = rnd("embed", int(cfg["vocab"]), width, s=0.7)
    vec("embed.norm", width, 0.2)
    for i, sp in enumerate(cfg["layers"]):
        p, m = f"l{i}.", sp["mixer"]
        H, G, D, Dv, taps = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        q = p + "mix."
        for nm, n in (("q", 2 * H * D), ("k", 2 * G * D), ("v", G * Dv)):
            lin(q + nm, n, width)
            W[q + nm + ".conv"] = rnd(q + nm + ".conv", n, taps, s=0.6)
        for nm in ("q.norm", "k.norm"):
            vec(q + nm, D, 0.3, 1.2)
        for nm in ("lq1", "lk1", "lq2", "lk2"):
            vec(q + nm, D, 0.5 * D ** -0.25)
        lin(q + "o", width, H * Dv)
        vec(p + "norm1", width, 0.2, -0.3)
        if sp.get("mlp"):
            r, ff = sp["mlp"]["router"], int(sp["mlp"]["expert"]["ff"])
            for e in range(int(r["experts"])):
                lin(p + f"mlp.e{e}.up", ff, width)
                lin(p + f"mlp.e{e}.down", width, ff)
            lin(p + "mlp.router", int(r["experts"]), width, 1.5)
            vec(p + "norm2", width, 0.2, -0.3)
    vec("final.norm", width, 0.2)
    return W
