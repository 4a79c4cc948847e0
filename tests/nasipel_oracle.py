"""A plain, slow evaluation of the Nasipel design in float64, one function per mechanism, for the tests.

Nothing here is shared with the product path: no framework import, whole sequences only, no cache, no state carried between
calls.  ``W`` maps checkpoint tensor names to tensors (``l<i>.mix.*``, ``l<i>.mlp.*`` ...); linear weights are ``[out, in]``.

Notation: ``x`` is the residual stream ``[T, width]``; ``ln(x) = (x - mean) / sqrt(var + eps)``; ``s`` the logistic function.

    x0 = E[tok]
    per layer:  a = ln(x) * w1;  b = ln(x) * w2;   x <- x + s(R1 a + r1) * mixer(a) + s(R2 b + r2) * ff(b)
    logits = (ln(x) * w_f) H^T
"""
import math

import torch

F64 = torch.float64


def sig(z):
    return torch.where(z >= 0, 1.0 / (1.0 + torch.exp(-z.abs())), torch.exp(-z.abs()) / (1.0 + torch.exp(-z.abs())))


def silu(z):
    return z * sig(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps)


# -- rotary positions -----------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """One turning rate per pair.  ``scaling``: YaRN's mixture of the rate and the rate divided by ``factor``."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            def at(turns):
                return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
            lo = max(math.floor(at(scaling["fast"])), 0)
            hi = min(math.ceil(at(scaling["slow"])), dims - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * r + f * (1.0 - r)
        out.append(f)
    return out


def amplitude(scaling=None):
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def rotate(x, positions, freqs, interleaved=False, amp=1.0, back=False):
    """Turn the pairs of every head of ``x [T, H, d]`` by ``position * freq`` (``back``: by the negative angle).  Pair ``i`` is
    ``(i, i + n)`` or, interleaved, ``(2 i, 2 i + 1)``; entries beyond ``2 n`` stay."""
    y = x.clone()
    n = len(freqs)
    for t, pos in enumerate(positions):
        for i, f in enumerate(freqs):
            ang = -pos * f if back else pos * f
            c, s = amp * math.cos(ang), amp * math.sin(ang)
            a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n)
            u, w = x[t, :, a], x[t, :, b]
            y[t, :, a] = u * c - w * s
            y[t, :, b] = w * c + u * s
    return y


# -- attention whose weights are logistic functions of the scores --------------------------------------------------------
def sigmoid_attention(q, k, v, scale, softcap=0.0, head_bias=None, first=0):
    """``q [n, H, d]`` are the queries of positions ``first ..``; ``k [L, G, d]``, ``v [L, G, dv]`` hold all positions from 0.
    Weight of key ``j <= i``: ``s(cap(q . k * scale) + bias_h)`` with ``cap(z) = softcap tanh(z / softcap)``; not normalised."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for a in range(n):
        i = first + a
        for h in range(H):
            g = h // (H // G)
            z = (k[:i + 1, g] @ q[a, h]) * scale
            if softcap:
                z = softcap * torch.tanh(z / softcap)
            if head_bias is not None:
                z = z + head_bias[h]
            out[a, h] = sig(z) @ v[:i + 1, g]
    return out


def attention_mixer(m, W, p, c, eps):
    T = m.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    pos = range(T)
    rot = c.get("rot") or {}
    fr = frequencies(rot.get("dims", 0), rot.get("base", 1.0))
    fv = frequencies(dv, rot.get("base", 1.0)) if rot else []
    q = rms(rotate((m @ W[p + "q"].T).view(T, H, d), pos, fr), eps)
    k = rms(rotate((m @ W[p + "k"].T).view(T, G, d), pos, fr), eps)
    v = rotate((m @ W[p + "v"].T).view(T, G, dv), pos, fv)
    o = sigmoid_attention(q, k, v, c["scale"], c.get("softcap", 0.0), W[p + "pb"])
    o = rotate(o, pos, fv, back=True)
    return o.reshape(T, H * dv) @ W[p + "o"].T


# -- real-gated linear recurrent unit ---------------------------------------------------------------------------------------
def causal_conv(x, w, b):
    """``y_t = sum_j w[:, j] x_(t - taps + 1 + j) + b`` per channel, zeros before the start.  ``x [T, C]``, ``w [C, taps]``."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y + b


def block_linear(u, w, b):
    """``u [T, C]`` in ``B`` equal parts, part ``n`` times ``w[n] [out, in]`` plus ``b[n]``."""
    B, n, _ = w.shape
    return torch.cat([u[:, i * n:(i + 1) * n] @ w[i].T + b[i] for i in range(B)], dim=1)


def rglru(u, r_pre, i_pre, lam):
    """``log a = -8 s(r_pre) softplus(lam)``; ``S <- a S + sqrt(1 - a^2) s(i_pre) u`` from zero.  All ``[T, C]``."""
    S = torch.zeros(u.shape[1], dtype=F64)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(-8.0 * sig(r_pre[t]) * softplus(lam))
        S = a * S + torch.sqrt(1.0 - a * a) * sig(i_pre[t]) * u[t]
        out[t] = S
    return out


def rglru_mixer(m, W, p, c, eps):
    y = gelu_tanh(m @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(m @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    S = rglru(u, block_linear(u, W[p + "ra"], W[p + "ra.b"]), block_linear(u, W[p + "ri"], W[p + "ri.b"]), W[p + "lam"])
    return (S * y) @ W[p + "o"].T


# -- latent attention with a rotated key part shared by the heads ---------------------------------------------------------
def latent_attention(qn, qr, kn, kr, v, scale, first=0):
    """``qn [n, H, d]``, ``qr [n, H, r]`` against ``kn [L, H, d]`` and the shared ``kr [L, r]``; softmax over ``j <= i`` of
    ``(qn . kn + qr . kr) * scale``; values ``[L, H, dv]``."""
    n, H, _ = qn.shape
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for a in range(n):
        i = first + a
        for h in range(H):
            z = (kn[:i + 1, h] @ qn[a, h] + kr[:i + 1] @ qr[a, h]) * scale
            e = torch.exp(z - z.max())
            out[a, h] = (e / e.sum()) @ v[:i + 1, h]
    return out


def latent_mixer(m, W, p, c, eps):
    T = m.shape[0]
    H, d, r, dv, kv = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    rot = c["rot"]
    fr, amp = frequencies(r, rot["base"], rot.get("scaling")), amplitude(rot.get("scaling"))
    pos = range(T)
    q = ((rms(m @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, d + r)
    qn, qr = q[..., :d], rotate(q[..., d:], pos, fr, True, amp)
    ckr = m @ W[p + "dkv"].T
    lat = rms(ckr[:, :kv], eps) * W[p + "dkv.norm"]
    kr = rotate(ckr[:, kv:].view(T, 1, r), pos, fr, True, amp)[:, 0]
    kn, v = (lat @ W[p + "uk"].T).view(T, H, d), (lat @ W[p + "uv"].T).view(T, H, dv)
    o = latent_attention(qn, qr, kn, kr, v, c["scale"])
    o = o * sig(m @ W[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * dv) @ W[p + "o"].T


# -- feed-forward -------------------------------------------------------------------------------------------------------------
def route(z, correction, top, groups=None, scale=1.0):
    """``z [E]`` -> (chosen experts, their weights).  Groups are kept by the sum of their two best corrected scores; among the
    experts of the kept groups the ``top`` best corrected scores win; the weights are the uncorrected scores, made to sum to
    one, times ``scale``."""
    s = sig(z)
    choice = [float(a + b) for a, b in zip(s, correction)]
    E = len(choice)
    allowed = list(range(E))
    if groups:
        n = E // groups["count"]
        marks = [sum(sorted(choice[g * n:(g + 1) * n], reverse=True)[:2]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -marks[g])[:groups["keep"]]
        allowed = [e for e in allowed if e // n in kept]
    idx = sorted(allowed, key=lambda e: -choice[e])[:top]
    w = s[idx]
    return idx, w / (w.sum() + 1e-20) * scale


def feed_forward(h, W, p, c):
    if not c:
        return torch.zeros_like(h)
    r = c["router"]
    out = torch.zeros_like(h)
    logits = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        idx, w = route(logits[t], W[p + "correction"], r["top"], r.get("groups"), r.get("scale", 1.0))
        for e, we in zip(idx, w):
            pe = f"{p}e{e}."
            out[t] += we * (W[pe + "down"] @ (silu(W[pe + "gate"] @ h[t]) * (W[pe + "up"] @ h[t])))
    return out


MIXERS = {"attention": attention_mixer, "rglru": rglru_mixer, "latent_attention": latent_mixer}


def forward(cfg, W, tokens, return_layers=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the stream after every layer)."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)]
    layers = []
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        n = layer_norm(x, eps)
        a = n * W[p + "norm1"]
        d = sig(a @ W[p + "rg1"].T + W[p + "rg1.b"]) * MIXERS[l["type"]](a, W, p + "mix.", l["mixer"], eps)
        if l.get("mlp"):
            b = n * W[p + "norm2"]
            d = d + sig(b @ W[p + "rg2"].T + W[p + "rg2.b"]) * feed_forward(b, W, p + "mlp.", l["mlp"])
        x = x + d
        layers.append(x.clone())
    logits = (layer_norm(x, eps) * W["final.norm"]) @ W["head"].T
    return (logits, layers) if return_layers else logits


# -- random checkpoints ---------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0):
    """Every tensor a checkpoint of ``cfg`` holds, fp32, from ``seed``: projections scaled by ``fan_in^-1/2``, norm weights
    around one, gates and biases spread enough that every branch matters."""
    g = torch.Generator().manual_seed(seed)
    Wd, V = cfg["width"], cfg["vocab"]

    def rnd(*s):
        return torch.randn(*s, generator=g)

    def lin(o, i, s=1.0):
        return rnd(o, i) * (s * i ** -0.5)

    def around_one(n):
        return 1.0 + 0.2 * rnd(n)

    W = {"embed": rnd(V, Wd), "final.norm": around_one(Wd), "head": lin(V, Wd)}
    for i, l in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", l["mixer"]
        W[p + "norm1"] = around_one(Wd)
        W[p + "rg1"], W[p + "rg1.b"] = lin(Wd, Wd, 2.0), rnd(Wd)
        q = p + "mix."
        if l["type"] == "attention":
            H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
            W[q + "q"], W[q + "k"], W[q + "v"], W[q + "o"] = lin(H * d, Wd), lin(G * d, Wd), lin(G * dv, Wd), lin(Wd, H * dv)
            W[q + "pb"] = rnd(H) - 2.0
        elif l["type"] == "rglru":
            C, B, taps = mx["width"], mx["blocks"], mx["conv"]
            for n in ("y", "x"):
                W[q + n], W[q + n + ".b"] = lin(C, Wd, 2.0), rnd(C) * 0.3
            W[q + "conv"], W[q + "conv.b"] = rnd(C, taps) * 0.6, rnd(C) * 0.3
            for n in ("ra", "ri"):
                W[q + n], W[q + n + ".b"] = rnd(B, C // B, C // B) * (2.0 * (C // B) ** -0.5), rnd(B, C // B)
            W[q + "lam"] = rnd(C) * 2.0 - 3.0
            W[q + "o"] = lin(Wd, C)
        else:
            H, d, r, dv, kv, qr = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"], mx["q_rank"]
            W[q + "dq"], W[q + "dq.norm"], W[q + "uq"] = lin(qr, Wd), around_one(qr), lin(H * (d + r), qr, 2.0)
            W[q + "dkv"], W[q + "dkv.norm"] = lin(kv + r, Wd), around_one(kv)
            W[q + "uk"], W[q + "uv"], W[q + "g"] = lin(H * d, kv), lin(H * dv, kv), lin(H, Wd, 2.0)
            W[q + "o"] = lin(Wd, H * dv)
        mlp = l.get("mlp")
        if mlp:
            W[p + "norm2"] = around_one(Wd)
            W[p + "rg2"], W[p + "rg2.b"] = lin(Wd, Wd, 2.0), rnd(Wd)
            q = p + "mlp."
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            W[q + "router"], W[q + "correction"] = lin(E, Wd, 3.0), rnd(E) * 0.3
            for e in range(E):
                W[f"{q}e{e}.gate"], W[f"{q}e{e}.up"], W[f"{q}e{e}.down"] = lin(ff, Wd, 2.0), lin(ff, Wd), lin(Wd, ff)
    return W
