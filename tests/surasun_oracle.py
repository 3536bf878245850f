"""A plain, slow restatement of the Surasun decoder, written from its equations with one function per mechanism.  It shares no code with the
serving path: every token is visited one by one, every sum is spelled out, everything is float64 but the rotary angle (see ``rotate``).  The tests compare the engine with it.

Notation: ``h`` the normed input of a sublayer, ``p`` a position (from 0), ``W x`` a stored [out, in] matrix applied to a vector.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softmax_rows(scores, values):
    """scores [n], values [n, d] -> sum_j softmax(scores)_j values_j"""
    e = torch.exp(scores - scores.max())
    return (e[:, None] * values).sum(0) / e.sum()


def rotate(x, p, rot, neighbours):
    """x [heads, dim] at position p, the first ``dims`` coordinates of every head turned in pairs: coordinates 2i and 2i + 1 (``neighbours``) or
    i and i + dims/2.  The design keeps frequencies and angles in 32-bit floats, so the angle is the rounded product of the rounded frequency:
    at position 1000 that rounding moves an angle by up to 3e-5, which a float64 angle would count as an error of the engine"""
    dims, base = int(rot["dims"]), float(rot["base"])
    y = x.clone()
    for i in range(dims // 2):
        a = float(torch.tensor(float(p), dtype=torch.float32) * torch.tensor(base ** (-2.0 * i / dims), dtype=torch.float32))
        c, s = math.cos(a), math.sin(a)
        m, n = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
        u, v = x[:, m], x[:, n]
        y[:, m] = u * c - v * s
        y[:, n] = v * c + u * s
    return y


def short_convolution(x, w, b):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start"""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = b.clone()
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                acc = acc + w[:, j] * x[src]
        out[t] = acc
    return out


# ---------------------------------------------------------------- mixers
def mamba2(h, m, W, pre, eps):
    T = h.shape[0]
    H, P, N, G, parts = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups"))
    inner = H * P
    proj = h @ W[pre + "in"].t()
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_convolution(xbc, W[pre + "conv"], W[pre + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B, C = xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W[pre + "dt_bias"])
    y = torch.zeros(T, H, P, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        S = torch.zeros(N, P, dtype=h.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(W[pre + "A_log"][hd]) * dt[t, hd]) * S + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            y[t, hd] = S.t() @ C[t, g] + W[pre + "D"][hd] * x[t, hd]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W[pre + "norm"]
    return y @ W[pre + "o"].t()


def attention(h, m, W, pre, eps):
    """causal grouped-query attention: whole-projection q / k norms, neighbouring pairs rotated, capped scores, a gate per head"""
    T = h.shape[0]
    H, G, D, Dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = rms(h @ W[pre + "q"].t() + W[pre + "q.b"], eps) * W[pre + "q.norm"]
    k = rms(h @ W[pre + "k"].t() + W[pre + "k.b"], eps) * W[pre + "k.norm"]
    v = (h @ W[pre + "v"].t() + W[pre + "v.b"]).reshape(T, G, Dv)
    q, k = q.reshape(T, H, D), k.reshape(T, G, D)
    if m.get("rot"):
        q = torch.stack([rotate(q[t], t, m["rot"], True) for t in range(T)])
        k = torch.stack([rotate(k[t], t, m["rot"], True) for t in range(T)])
    gate = torch.sigmoid(h @ W[pre + "g"].t())                     # [T, H]
    scale, cap = float(m["scale"]), m.get("softcap")
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for i in range(T):
        for hd in range(H):
            g = hd // (H // G)
            s = (k[: i + 1, g] @ q[i, hd]) * scale
            if cap:
                s = float(cap) * torch.tanh(s / float(cap))
            out[i, hd] = softmax_rows(s, v[: i + 1, g]) * gate[i, hd]
    return out.reshape(T, H * Dv) @ W[pre + "o"].t()


def retention(h, m, W, pre, eps):
    T = h.shape[0]
    H, D, Dv = (int(m[k]) for k in ("heads", "dim", "vdim"))
    q, k, v = (h @ W[pre + "q"].t()).reshape(T, H, D), (h @ W[pre + "k"].t()).reshape(T, H, D), (h @ W[pre + "v"].t()).reshape(T, H, Dv)
    if m.get("rot"):
        q = torch.stack([rotate(q[t], t, m["rot"], False) for t in range(T)])
        k = torch.stack([rotate(k[t], t, m["rot"], False) for t in range(T)])
    k = k * D ** -0.5
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hd in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        for t in range(T):
            S = float(m["decay"][hd]) * S + torch.outer(k[t, hd], v[t, hd])
            o[t, hd] = S.t() @ q[t, hd]
    return (rms(o, eps).reshape(T, H * Dv) * silu(h @ W[pre + "g"].t())) @ W[pre + "o"].t()


def parallel(h, m, W, pre, eps):
    return float(m["left_scale"]) * attention(h, m["left"], W, pre + "left.", eps) + float(m["right_scale"]) * retention(h, m["right"], W, pre + "right.", eps)


def rglru_gates(u, W, pre, blocks):
    """-> (a, i) [T, width]: the decay and the input gate of every channel"""
    T, C = u.shape
    n = C // blocks
    r, i = torch.zeros_like(u), torch.zeros_like(u)
    for b in range(blocks):
        part = u[:, b * n:(b + 1) * n]
        r[:, b * n:(b + 1) * n] = torch.sigmoid(part @ W[pre + "ra"][b].t() + W[pre + "ra.b"][b])
        i[:, b * n:(b + 1) * n] = torch.sigmoid(part @ W[pre + "ri"][b].t() + W[pre + "ri.b"][b])
    return torch.exp(-8.0 * r * softplus(W[pre + "lam"])), i


def rglru(h, m, W, pre):
    T, C = h.shape[0], int(m["width"])
    y = gelu_tanh(h @ W[pre + "y"].t() + W[pre + "y.b"])
    u = short_convolution(h @ W[pre + "x"].t() + W[pre + "x.b"], W[pre + "conv"], W[pre + "conv.b"])
    a, i = rglru_gates(u, W, pre, int(m["blocks"]))
    S, out = torch.zeros(C, dtype=h.dtype), torch.zeros_like(u)
    for t in range(T):
        S = a[t] * S + torch.sqrt(1.0 - a[t] * a[t]) * i[t] * u[t]
        out[t] = S
    return (out * y) @ W[pre + "o"].t()


def glu(h, W, pre):
    return (silu(h @ W[pre + "gate"].t()) * (h @ W[pre + "up"].t())) @ W[pre + "down"].t()


# ---------------------------------------------------------------- streams
def stream_input(X, W, pre):
    """X [streams, T, width] -> the sublayer's un-normed input"""
    return sum(W[pre + "in"][s] * X[s] for s in range(len(X)))


def stream_update(X, y, W, pre, mult):
    """every stream from the OLD ones: mix[from, to]"""
    return [sum(W[pre + "mix"][s, t] * X[s] for s in range(len(X))) + mult * W[pre + "out"][t] * y for t in range(len(X))]


# ---------------------------------------------------------------- the model
def forward(cfg, W, tokens, tap=None, dtype=F64):
    """logits [T, vocab] of one sequence; ``tap(layer, x)`` sees the sum of the streams after every layer"""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    X = [W["embed"][list(tokens)].clone() for _ in range(int(cfg["streams"]))]
    for i, sp in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", sp["mixer"], sp["type"]
        h = layer_norm(stream_input(X, W, p + "hc1."), W[p + "norm1"], eps)
        if kind == "mamba2":
            y = mamba2(h, m, W, p + "mix.", eps)
        elif kind == "parallel":
            y = parallel(h, m, W, p + "mix.", eps)
        elif kind == "rglru":
            y = rglru(h, m, W, p + "mix.")
        else:
            raise ValueError(kind)
        X = stream_update(X, y, W, p + "hc1.", mult)
        if sp.get("mlp"):
            h = layer_norm(stream_input(X, W, p + "hc2."), W[p + "norm2"], eps)
            X = stream_update(X, glu(h, W, p + "mlp."), W, p + "hc2.", mult)
        if tap is not None:
            tap(i, sum(X))
    return layer_norm(sum(X), W["final.norm"], eps) @ W["embed"].t()


def random_weights(cfg, seed=0):
    """random tensors under the checkpoint names, sized so that every mechanism matters: gates and decays away from their ends, streams that
    differ, a mix matrix that is not symmetric"""
    g = torch.Generator().manual_seed(seed)
    W = {}
    rnd = lambda *s, scale=1.0, off=0.0: torch.randn(*s, generator=g) * scale + off
    lin = lambda o, i, scale=1.0: rnd(o, i, scale=scale * i ** -0.5)
    w, S = int(cfg["width"]), int(cfg["streams"])
    W["embed"] = rnd(int(cfg["vocab"]), w, scale=0.6)
    for i, sp in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", sp["mixer"], sp["type"]
        q = p + "mix."
        if kind == "mamba2":
            H, P, N, G, taps = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv"))
            W[q + "in"] = lin(2 * H * P + 2 * G * N + H, w)
            W[q + "conv"], W[q + "conv.b"] = rnd(H * P + 2 * G * N, taps, scale=0.6), rnd(H * P + 2 * G * N, scale=0.3)
            W[q + "dt_bias"], W[q + "A_log"], W[q + "D"] = rnd(H, off=-1.0), rnd(H, scale=0.7), rnd(H, off=1.0)
            W[q + "norm"], W[q + "o"] = rnd(H * P, scale=0.2, off=1.0), lin(w, H * P)
        elif kind == "parallel":
            a, b = m["left"], m["right"]
            H, G, D, Dv = (int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            l = q + "left."
            for nm, n in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                W[l + nm], W[l + nm + ".b"] = lin(n, w), rnd(n, scale=0.4)
            W[l + "q.norm"], W[l + "k.norm"] = rnd(H * D, scale=0.3, off=1.0), rnd(G * D, scale=0.3, off=1.0)
            W[l + "g"], W[l + "o"] = lin(H, w), lin(w, H * Dv)
            H, D, Dv = (int(b[k]) for k in ("heads", "dim", "vdim"))
            r = q + "right."
            for nm, n in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                W[r + nm] = lin(n, w)
            W[r + "o"] = lin(w, H * Dv)
        else:
            C, nb, taps = int(m["width"]), int(m["blocks"]), int(m["conv"])
            n = C // nb
            for nm in ("y", "x"):
                W[q + nm], W[q + nm + ".b"] = lin(C, w), rnd(C, scale=0.3)
            W[q + "conv"], W[q + "conv.b"] = rnd(C, taps, scale=0.6), rnd(C, scale=0.3)
            for nm in ("ra", "ri"):
                W[q + nm], W[q + nm + ".b"] = rnd(nb, n, n, scale=n ** -0.5), rnd(nb, n, scale=0.5)
            W[q + "lam"], W[q + "o"] = rnd(C, off=-3.0), lin(w, C)
        W[p + "norm1"] = rnd(w, scale=0.2, off=1.0)
        subs = [1]
        if sp.get("mlp"):
            ff = int(sp["mlp"]["ff"])
            W[p + "norm2"] = rnd(w, scale=0.2, off=1.0)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = lin(ff, w), lin(ff, w), lin(w, ff)
            subs.append(2)
        for n in subs:
            hc = f"{p}hc{n}."
            W[hc + "in"], W[hc + "out"] = rnd(S, scale=0.3, off=1.0 / S), rnd(S, scale=0.5, off=1.0)
            W[hc + "mix"] = torch.eye(S) * 0.8 + rnd(S, S, scale=0.25 / S ** 0.5)
    W["final.norm"] = rnd(w, scale=0.2, off=1.0)
    return W
