"""A plain, slow evaluation of the Dufitar design in float64, one function per mechanism, for the tests.

Nothing here is shared with the product path: no framework import, whole sequences only, no cache, no state carried between
calls.  ``W`` maps checkpoint tensor names to tensors (``l<i>.mix.*``, ``l<i>.mlp.*`` ...); linear weights are ``[out, in]``.

Notation: ``x`` is the residual stream ``[T, width]``, ``N_k`` the squashing norm ``tanh(alpha_k x) * w_k + b_k`` of name ``k``, ``m`` the
multiplier of every addition.

    x = scale_e * E[tok]
    per layer:  x <- x + m N_1b(mixer(N_1(x)));   x <- x + m N_2b(ff(N_2(x)))
    logits = N_final(x) E^T
"""
import math

import torch

F64 = torch.float64


def sig(z):
    return torch.where(z >= 0, 1.0 / (1.0 + torch.exp(-z.abs())), torch.exp(-z.abs()) / (1.0 + torch.exp(-z.abs())))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def squash(x, alpha, w, b):
    """No statistics over the row: every channel by itself."""
    return torch.tanh(alpha * x) * w + b


def norm(x, W, name):
    return squash(x, W[name + ".alpha"], W[name], W[name + ".b"])


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# -- rotary positions -----------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """One turning rate per pair.  ``scaling``: a ramp between the rate (pairs with many turns over the original length) and the
    rate divided by ``factor`` (pairs with few)."""
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


def rotate(x, positions, freqs, amp=1.0):
    """Turn the pairs ``(2 i, 2 i + 1)`` of every head of ``x [T, H, d]`` by ``position * freq``; entries beyond the pairs stay."""
    y = x.clone()
    for t, pos in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s = amp * math.cos(pos * f), amp * math.sin(pos * f)
            u, w = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i] = u * c - w * s
            y[t, :, 2 * i + 1] = w * c + u * s
    return y


# -- attention ------------------------------------------------------------------------------------------------------------
def first_visible(i, window):
    return max(0, i - window + 1) if window else 0


def softmax_weights(z, sink=None):
    """``exp(z_j) / (exp(sink) + sum_j exp(z_j))``; without a sink the first term is absent."""
    top = float(z.max()) if sink is None else max(float(z.max()), float(sink))
    e = torch.exp(z - top)
    return e / (e.sum() + (math.exp(float(sink) - top) if sink is not None else 0.0))


def window_attention(q, k, v, scale, window=0, sink=None, first=0):
    """``q [n, H, d]`` are the queries of positions ``first ..``; ``k [L, G, d]``, ``v [L, G, dv]`` hold all positions from 0.  Query
    ``i`` sees itself and the ``window - 1`` positions before it (``window = 0``: everything before it)."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for a in range(n):
        i = first + a
        lo = first_visible(i, window)
        for h in range(H):
            g = h // (H // G)
            z = (k[lo:i + 1, g] @ q[a, h]) * scale
            out[a, h] = softmax_weights(z, None if sink is None else sink[h]) @ v[lo:i + 1, g]
    return out


def attention_mixer(h, W, p, c, eps, shared):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    rot = c["rot"]
    fr, amp = frequencies(rot["dims"], rot["base"], rot.get("scaling")), amplitude(rot.get("scaling"))
    q = rotate((h @ W[p + "q"].T).view(T, H, d), range(T), fr, amp)
    k = rotate((h @ W[p + "k"].T).view(T, G, d), range(T), fr, amp)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    o = window_attention(q, k, v, c["scale"], c["mask"]["size"])
    return o.reshape(T, H * dv) @ W[p + "o"].T


# -- latent attention -----------------------------------------------------------------------------------------------------
def latent_attention(qn, qr, kn, kr, v, scale, window=0, sink=None, first=0):
    """``qn [n, H, d]``, ``qr [n, H, r]`` against ``kn [L, H, d]`` and the shared ``kr [L, r]``; weights over the window of
    ``(qn . kn + qr . kr) * scale``; values ``[L, H, dv]``; ``sink [H]``."""
    n, H, _ = qn.shape
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for a in range(n):
        i = first + a
        lo = first_visible(i, window)
        for h in range(H):
            z = (kn[lo:i + 1, h] @ qn[a, h] + kr[lo:i + 1] @ qr[a, h]) * scale
            out[a, h] = softmax_weights(z, None if sink is None else sink[h]) @ v[lo:i + 1, h]
    return out


def latent_rows(h, W, p, c, eps):
    """What a layer with a down projection of its own caches: the normed latents ``[T, r]`` and the rotated keys ``[T, n]``."""
    T, n, r, rot = h.shape[0], c["rot_dim"], c["kv_rank"], c["rot"]
    ckr = h @ W[p + "dkv"].T
    lat = rms(ckr[:, :r], eps) * W[p + "dkv.norm"]
    return lat, rotate(ckr[:, r:].view(T, 1, n), range(T), frequencies(n, rot["base"]))[:, 0]


def latent_mixer(h, W, p, c, eps, shared):
    T = h.shape[0]
    H, d, n, dv = c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, d + n)
    qn, qr = q[..., :d], rotate(q[..., d:], range(T), frequencies(n, c["rot"]["base"]))
    lat, kr = shared[c["kv_from"]] if c.get("kv_from") is not None else latent_rows(h, W, p, c, eps)
    shared[int(p.split(".")[0][1:])] = (lat, kr)
    kn, v = (lat @ W[p + "uk"].T).view(T, H, d), (lat @ W[p + "uv"].T).view(T, H, dv)
    o = latent_attention(qn, qr, kn, kr, v, c["scale"], c["mask"]["size"], W[p + "sink"])
    return (o.reshape(T, H * dv) * sig(h @ W[p + "g"].T)) @ W[p + "o"].T


# -- feed-forward, the model ------------------------------------------------------------------------------------------------
def feed_forward(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer}


def forward(cfg, W, tokens, return_layers=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the stream after every layer)."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    layers, shared = [], {}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * norm(MIXERS[l["type"]](norm(x, W, p + "norm1"), W, p + "mix.", l["mixer"], eps, shared), W, p + "norm1b")
        if l.get("mlp"):
            x = x + m * norm(feed_forward(norm(x, W, p + "norm2"), W, p + "mlp."), W, p + "norm2b")
        layers.append(x.clone())
    logits = norm(x, W, "final.norm") @ W["embed"].T
    return (logits, layers) if return_layers else logits


# -- random checkpoints ---------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0):
    """Every tensor a checkpoint of ``cfg`` holds, fp32, from ``seed``: projections scaled by ``fan_in^-1/2``, norms whose slope,
    weight and offset all matter, sinks and gates spread enough that leaving one out shows."""
    g = torch.Generator().manual_seed(seed)
    Wd, V = cfg["width"], cfg["vocab"]

    def rnd(*s):
        return torch.randn(*s, generator=g)

    def lin(o, i, s=1.0):
        return rnd(o, i) * (s * i ** -0.5)

    W = {"embed": rnd(V, Wd)}

    def add_norm(name, alpha):
        W[name], W[name + ".b"] = 1.0 + 0.3 * rnd(Wd), 0.2 * rnd(Wd)
        W[name + ".alpha"] = alpha * (1.0 + 0.2 * torch.rand((), generator=g))

    add_norm("final.norm", 0.4)
    for i, l in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", l["mixer"]
        add_norm(p + "norm1", 0.5), add_norm(p + "norm1b", 0.8)
        q = p + "mix."
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        if l["type"] == "attention":
            G = mx["kv_heads"]
            W[q + "q"], W[q + "k"], W[q + "v"] = lin(H * d, Wd, 2.0), lin(G * d, Wd, 2.0), lin(G * dv, Wd, 2.0)
        else:
            n, r = mx["rot_dim"], mx["kv_rank"]
            W[q + "q"] = lin(H * (d + n), Wd, 2.0)
            if mx.get("kv_from") is None:
                W[q + "dkv"], W[q + "dkv.norm"] = lin(r + n, Wd, 2.0), 1.0 + 0.3 * rnd(r)
            W[q + "uk"], W[q + "uv"], W[q + "g"] = lin(H * d, r, 1.5), lin(H * dv, r, 1.5), lin(H * dv, Wd, 2.0)
            W[q + "sink"] = 1.0 + rnd(H)
        W[q + "o"] = lin(Wd, H * dv, 2.0)
        if l.get("mlp"):
            add_norm(p + "norm2", 0.5), add_norm(p + "norm2b", 0.8)
            q, ff = p + "mlp.", l["mlp"]["ff"]
            W[q + "gate"], W[q + "up"], W[q + "down"] = lin(ff, Wd, 2.0), lin(ff, Wd), lin(Wd, ff, 2.0)
    return W
