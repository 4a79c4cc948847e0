"""Dufitar models in the framework against a plain, slow evaluation of the design's equations (``dufitar_oracle``).

Each test builds its own small configuration and random (or hand-made) weights, loads them through the product loader
and drives the model through the dynamic engine -- whole prompts, prompts cut into portions, token-by-token decoding,
mixed batches, reused pages -- on the CPU (PyTorch op path) and, marked ``gpu``, on the sm_100a kernels.
"""
import copy
import json
import os
import struct
import subprocess
import sys

import pytest
import torch

import dufitar_oracle as oracle
from megatronapp_b200.data.tokenizer import NullTokenizer
from megatronapp_b200.inference import DynamicInferenceEngine, SamplingParams
from megatronapp_b200.inference.trace import TraceReplayer
from megatronapp_b200.models.dufitar import DufitarConfig, DufitarModel
from megatronapp_b200.models.dufitar.loader import load_dufitar_weights, shapes_into_config
from megatronapp_b200.ops import seqmix
from megatronapp_b200.ops.seqmix import HeadPart
from megatronapp_b200.parallel import state as ps

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
VOCAB = 53
YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}

ATT = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.4, "mask": {"size": 11}, "rot": {"dims": 6, "base": 50.0, "scaling": YARN}}
ATT_B = {"heads": 3, "kv_heads": 3, "dim": 20, "vdim": 6, "scale": 0.2, "mask": {"size": 4},
         "rot": {"dims": 20, "base": 10000.0, "scaling": dict(YARN, factor=8.0, original=128, fast=16.0, slow=2.0)}}      # the whole head turns
ATT_C = {"heads": 6, "kv_heads": 1, "dim": 16, "vdim": 40, "scale": 0.25, "mask": {"size": 33}, "rot": {"dims": 8, "base": 300.0}}   # no scaling
LAT = {"heads": 3, "dim": 8, "rot_dim": 4, "vdim": 6, "kv_rank": 12, "scale": 0.3, "mask": {"size": 9}, "rot": {"base": 20.0, "dims": 4}}
LAT_B = {"heads": 2, "dim": 6, "rot_dim": 8, "vdim": 10, "kv_rank": 20, "scale": 0.25, "mask": {"size": 17}, "rot": {"base": 10000.0, "dims": 8}}
LAT_C = {"heads": 5, "dim": 12, "rot_dim": 6, "vdim": 12, "kv_rank": 40, "scale": 0.2, "mask": {"size": 30}, "rot": {"base": 100.0, "dims": 6}}
LAT_S = {"heads": 2, "dim": 5, "rot_dim": 4, "vdim": 7, "kv_rank": 12, "scale": 0.35, "mask": {"size": 14}, "rot": {"base": 20.0, "dims": 4}}   # reads LAT's rows
MIX = {"attention": (ATT, ATT_B, ATT_C), "latent_attention": (LAT, LAT_B, LAT_C, LAT_S)}
FF, FF_B = {"kind": "dense", "ff": 24}, {"kind": "dense", "ff": 10}


def layer(kind, variant=0, mlp=None, **mixer):
    return {"type": kind, "mixer": dict(copy.deepcopy(MIX[kind][variant]), **mixer), "mlp": copy.deepcopy(mlp)}


def config_of(layers, width=32, vocab=VOCAB, eps=1e-5, mult=0.7, scale=1.9):
    return {"architecture": "Dufitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": layers}


# two sources of latents, one of them read twice and by a layer with other heads and another window
HYBRID = config_of([layer("attention", 0, FF), layer("latent_attention", 0, FF_B), layer("latent_attention", 1), layer("latent_attention", 3, FF, kv_from=1),
                    layer("attention", 1, FF_B), layer("latent_attention", 1, None, kv_from=2, mask={"size": 5}), layer("latent_attention", 0, FF, kv_from=1)])


def build(cfg, device, dtype=torch.float32, seed=0, weights=None):
    if not ps.model_parallel_is_initialized():
        ps.initialize_model_parallel(1, 1)
    W = weights if weights is not None else oracle.random_weights(cfg, seed)
    raw = shapes_into_config(copy.deepcopy(cfg), {k: tuple(v.shape) for k, v in W.items()})
    dcfg = DufitarConfig.from_dict(raw)
    model = DufitarModel(dcfg, dcfg.base_transformer_config(dtype, use_cpu_initialization=True, perform_initialization=False))
    load_dufitar_weights(model, W)
    return model.to(device).eval(), W


def replayer(model, max_tokens=512, block_size=4, max_requests=4):
    return TraceReplayer(model, max_tokens, block_size=block_size, max_requests=max_requests, max_sequence_length=4096)


def run_cut(rp, rid, tokens, cuts):
    """Feed ``tokens`` in portions of the given sizes (the rest one by one); logits of every position."""
    outs, at = [], 0
    sizes = list(cuts)
    while at < len(tokens):
        n = sizes.pop(0) if sizes else 1
        n = min(n, len(tokens) - at)
        outs.append(rp.step([{"id": rid, "tokens": tokens[at:at + n], "want": list(range(n))}]))
        at += n
    rp.step([], end=[rid])
    return torch.cat(outs)


def tokens_of(n, vocab=VOCAB, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def close(got, want, tol):
    want = want.to(torch.float64)
    err = (got.to(torch.float64).cpu() - want).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), f"max error {err:.3e} (scale {want.abs().max().item():.3e})"


TOL = 1e-4


def close_in_16_bits(got, want, typical=3e-2, outlier=0.15, share=0.1):
    """The typical position must be near (root mean square over the vocabulary, relative to the logits' scale), a few may not."""
    want = want.to(torch.float64)
    rel = (got.to(torch.float64).cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(rel.median()) <= typical and float((rel > outlier).double().mean()) <= share, \
        f"median {float(rel.median()):.3e}, worst {float(rel.max()):.3e}"


# ---------------------------------------------------------------------------------------------------------------------
# every mechanism alone: one layer (or a pair that shares latents), whole prompt and cut prompt
# ---------------------------------------------------------------------------------------------------------------------
SINGLE = [[layer(k, v)] for k in MIX for v in range(3)] + [[layer("attention", 0, FF)], [layer("latent_attention", 0), layer("latent_attention", 3, kv_from=0)]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("layers", SINGLE, ids=[f"{k}{v}" for k in MIX for v in range(3)] + ["dense", "shared_latents"])
def test_single_mechanism_matches_oracle(layers, device):
    cfg = config_of(layers)
    model, W = build(cfg, device, seed=1)
    toks = tokens_of(41)
    want, streams = oracle.forward(cfg, W, toks, return_layers=True)
    seen = []
    model.decoder.tap = lambda i, x: seen.append(x.detach().float().cpu().clone())
    rp = replayer(model)
    close(run_cut(rp, "a", toks, [len(toks)]), want, TOL)
    for got, x in zip(seen, streams):
        close(got.view(len(toks), -1), x, TOL)
    model.decoder.tap = None
    close(run_cut(rp, "b", toks, [17, 2, 18]), want, TOL)


def test_whole_sequence_forward_without_a_context():
    """The training-style call (``[b, s]`` ids, no inference context) runs the same mixers; labels give the loss per token."""
    model, W = build(HYBRID, "cpu")
    a, b = tokens_of(21, seed=1), tokens_of(21, seed=2)
    out = model(torch.tensor([a, b]), None, None)
    want = oracle.forward(HYBRID, W, b)
    close(out[0], oracle.forward(HYBRID, W, a), TOL)
    close(out[1], want, TOL)
    labels = torch.tensor([tokens_of(21, seed=3)])
    loss = model(torch.tensor([b]), None, None, labels=labels)
    close(loss[0].detach(), -torch.log_softmax(want, -1).gather(1, labels[0].view(-1, 1))[:, 0], TOL)


# ---------------------------------------------------------------------------------------------------------------------
# ops against the oracle's functions
# ---------------------------------------------------------------------------------------------------------------------
def paged(lens, block_size, seed=0):
    """Shuffled pages for sequences of the given lengths: ``(table, number of slots, slot indices of every sequence)``."""
    g = torch.Generator().manual_seed(seed)
    nb = [-(-n // block_size) for n in lens]
    perm = torch.randperm(sum(nb), generator=g)
    table = torch.zeros(len(lens), max(nb), dtype=torch.int32)
    slots, at = [], 0
    for r, n in enumerate(lens):
        table[r, :nb[r]] = perm[at:at + nb[r]].to(torch.int32)
        at += nb[r]
        pos = torch.arange(n)
        slots.append(table[r].long()[pos // block_size] * block_size + pos % block_size)
    return table, sum(nb) * block_size, slots


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,width", [(7, 20), (5, 22), (3, 640), (300, 36)])
def test_squashing_norm_and_its_additions(T, width, device):
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    d = lambda t: t.to(device)  # noqa: E731
    x, wide = rnd(T, width) * 2, rnd(T, 2 * width) * 3                  # the addend is a column slice
    no, nn = (torch.tensor(0.8), rnd(width), rnd(width)), (torch.tensor(-1.3), rnd(width), rnd(width))
    D = lambda n: tuple(t.double() for t in n)  # noqa: E731
    a = wide[:, width:]
    ad, nod, nnd = d(wide)[:, width:], tuple(map(d, no)), tuple(map(d, nn))
    x1 = x.double() + 0.3 * oracle.squash(a.double(), *D(no))
    gx, h = seqmix.squash_add(d(x.clone()), ad, nod, nnd, 0.3, torch.float32)
    close(gx, x1, 1e-6), close(h, oracle.squash(x1, *D(nn)), 2e-6)
    gx, h = seqmix.squash_add(d(x.clone()), ad, nod, None, 1.0, torch.float32)
    assert h is None
    close(gx, x.double() + oracle.squash(a.double(), *D(no)), 1e-6)
    gx, h = seqmix.squash_add(d(x.clone()), None, None, nnd, 0.3, torch.float32, 2.5)
    close(gx, 2.5 * x.double(), 1e-6), close(h, oracle.squash(2.5 * x.double(), *D(nn)), 2e-6)
    gx, h = seqmix.squash_add(d(x.clone()), ad, None, nnd, -0.5, torch.float32)
    close(gx, x.double() - 0.5 * a.double(), 1e-6)
    b = lambda n: tuple(t.to(device, torch.bfloat16) for t in n)  # noqa: E731
    r = lambda n: tuple(t.to(torch.bfloat16).double() for t in n)  # noqa: E731
    gx, h = seqmix.squash_add(d(x.clone()), ad.to(torch.bfloat16), b(no), b(nn), 0.3, torch.bfloat16)
    x1 = x.double() + 0.3 * oracle.squash(a.to(torch.bfloat16).double(), *r(no))
    close(gx, x1, 1e-6)                                                 # the stream stays fp32
    assert h.dtype == torch.bfloat16
    close(h, oracle.squash(x1, *r(nn)), 4e-3)
    # large and tiny arguments
    z = torch.tensor([[0.0, 1e-6, -1e-3, 50.0, -1e4, 3.0, -0.54, 0.56]])
    one, zero = torch.ones(8), torch.zeros(8)
    _, h = seqmix.squash_add(d(z.clone()), None, None, (d(torch.tensor(1.0)), d(one), d(zero)), 0.0, torch.float32)
    assert float((h.double().cpu() / torch.tanh(z.double()) - 1)[:, 1:].abs().max()) < 1e-6 and float(h[0, 0]) == 0.0


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,cols", [(5, 12), (3, 10), (70, 1028)])
def test_gated_gelu(rows, cols, device):
    from megatronapp_b200.transformer.mlp import gelu_glu

    g = torch.Generator().manual_seed(1)
    x = torch.randn(rows, 1, 2 * cols, generator=g) * 3
    want = oracle.gelu_tanh(x[..., :cols].double()) * x[..., cols:].double()
    close(gelu_glu(x.to(device)), want, 1e-6)
    xb = x.to(torch.bfloat16)
    want = oracle.gelu_tanh(xb[..., :cols].double()) * xb[..., cols:].double()
    close(gelu_glu(xb.to(device)).float(), want, 4e-3)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("H,G,d,dv,window", [(4, 2, 6, 10, 7), (6, 1, 20, 14, 1), (3, 3, 32, 64, 64), (12, 2, 64, 72, 100), (1, 1, 40, 130, 1000)])
def test_window_attention_prompts_and_decoding_batches(H, G, d, dv, window, dtype, device):
    """Unequal sequences over shuffled pages: all tokens as prompts in one call, then the last token of each as a decoding batch
    (the split path on the GPU), both against the oracle."""
    lens, bs = [3, 40, 130], 8
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    table, n_slots, slots = paged(lens, bs)
    kc, vc = torch.zeros(n_slots, G, d), torch.zeros(n_slots, G, dv)
    qs, wants = [], []
    for r, n in enumerate(lens):
        q, k, v = rnd(n, H, d), rnd(n, G, d), rnd(n, G, dv)
        kc[slots[r]], vc[slots[r]] = k, v
        qs.append(q)
        wants.append(oracle.window_attention(q.double(), k.double(), v.double(), 0.3, window))
    D = lambda t: t.to(device, dtype)  # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    got = seqmix.window_attention_paged(D(torch.cat(qs)), D(kc), D(vc), table.to(device), i32([r for r, n in enumerate(lens) for _ in range(n)]),
                                        i32([i + 1 for n in lens for i in range(n)]), bs, 0.3, window)
    close(got.view(-1, H, dv).float(), torch.cat(wants), tol)
    got = seqmix.window_attention_paged(D(torch.cat([q[-1:] for q in qs])), D(kc), D(vc), table.to(device), i32([0, 1, 2]), i32(lens), bs, 0.3,
                                        window, max_len=max(lens))
    close(got.view(-1, H, dv).float(), torch.cat([w[-1:] for w in wants]), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("H,n,r,window,sink", [(3, 4, 12, 5, True), (5, 10, 40, 33, False), (16, 32, 96, 1, True), (2, 16, 260, 150, True), (20, 64, 512, 0, True),
                                               (4, 8, 24, 100, False), (9, 16, 64, 1000, True)])
def test_latent_attention_with_a_window_and_a_sink(H, n, r, window, sink, dtype, device):
    """Prompts, then one token per sequence (key splits on the GPU), over shuffled pages; sinks from negligible to dominant."""
    lens, bs = [5, 34, 270], 16
    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    table, n_slots, slots = paged(lens, bs)
    cache = torch.zeros(n_slots, r + n)
    sk = torch.linspace(-3.0, 6.0, H).to(dtype).float() if sink else None
    ql, qr, wants = [], [], []
    for s_, L in enumerate(lens):
        c, kr, q1, q2 = rnd(L, r), rnd(L, n), (rnd(L, H, r) * r ** -0.5 * 2).to(dtype).float(), rnd(L, H, n)
        cache[slots[s_], :r], cache[slots[s_], r:] = c, kr
        ql.append(q1), qr.append(q2)
        z = (torch.einsum("thr,lr->htl", q1.double(), c.double()) + torch.einsum("thn,ln->htl", q2.double(), kr.double())) * 0.2
        i, j = torch.arange(L).view(-1, 1), torch.arange(L).view(1, -1)
        e = torch.exp(z).masked_fill(~((j <= i) & ((i - j < window) | (window == 0))), 0.0)
        p = e / (e.sum(-1, keepdim=True) + (torch.exp(sk.double()).view(H, 1, 1) if sink else 0.0))
        wants.append(torch.einsum("htl,lr->thr", p, c.double()))
    D = lambda t: t.to(device, dtype)  # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    kw = dict(window=window, sink=None if sk is None else D(sk))
    got = seqmix.latent_attention_paged(D(torch.cat(ql)), D(cache), table.to(device), i32([s_ for s_, L in enumerate(lens) for _ in range(L)]),
                                        i32([i + 1 for L in lens for i in range(L)]), bs, 0.2, max(lens), D(torch.cat(qr)), **kw)
    close(got.float(), torch.cat(wants), tol)
    ends = [sum(lens[:s_ + 1]) - 1 for s_ in range(3)]
    got = seqmix.latent_attention_paged(D(torch.cat(ql))[ends], D(cache), table.to(device), i32([0, 1, 2]), i32(lens), bs, 0.2, max(lens),
                                        D(torch.cat(qr))[ends], **kw)
    close(got.float(), torch.cat([w[-1:] for w in wants]), tol)


@pytest.mark.parametrize("device", DEVICES)
def test_rotation_beside_latent_norm_and_pages_in_one_launch(device):
    """The three operands of a latent layer with a direct query: query part, latent norm, shared key; YaRN and plain rates."""
    g = torch.Generator().manual_seed(1)
    T, H, d, n, r = 6, 3, 5, 8, 10
    proj = torch.randn(T, H * (d + n) + r + n, generator=g)
    pos, slots, w = torch.tensor([0, 1, 5, 700, 3, 40]), torch.tensor([9, 2, 4, 0, 7, 11]), torch.randn(10, generator=g)
    turns, amp = seqmix.rotary_turns(n, 100.0, YARN)
    assert amp == pytest.approx(oracle.amplitude(YARN))
    dd = lambda t: t.to(device)  # noqa: E731
    pd = dd(proj)
    q = pd[:, :H * (d + n)].unflatten(1, (H, d + n))
    qr, pages = torch.empty(T, H, n, device=device), torch.zeros(12, r + n, device=device)
    o0 = H * (d + n)
    kw = dict(turns=dd(turns), interleaved=True, amplitude=amp)
    seqmix.head_rotary([HeadPart(q[..., d:], out=qr, **kw), HeadPart(pd[:, o0:o0 + r].unsqueeze(1), rms=True, weight=dd(w), pages=pages[:, :r].unsqueeze(1)),
                        HeadPart(pd[:, o0 + r:].unsqueeze(1), pages=pages[:, r:].unsqueeze(1), **kw)], dd(pos), 1e-5, dd(slots))
    P, fr, D = pos.tolist(), oracle.frequencies(n, 100.0, YARN), proj.double()
    close(qr, oracle.rotate(D[:, :o0].view(T, H, d + n)[..., d:], P, fr, oracle.amplitude(YARN)), 1e-5)
    close(pages[slots][:, :r], oracle.rms(D[:, o0:o0 + r], 1e-5) * w.double(), 1e-5)
    close(pages[slots][:, r:], oracle.rotate(D[:, o0 + r:].unsqueeze(1), P, fr, oracle.amplitude(YARN))[:, 0], 1e-5)
    assert float(pages[[1, 3, 5, 6, 8, 10]].abs().max()) == 0.0


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,dv,cols", [(3, 8, 29), (2, 7, 14), (1, 5, 6), (4, 32, 256)])
def test_elementwise_output_gate(H, dv, cols, device):
    g = torch.Generator().manual_seed(5)
    o, wide = torch.randn(6, H, dv, generator=g), torch.randn(6, cols, generator=g)
    gate = wide[:, cols - H * dv:]
    want = o.double() * oracle.sig(gate.double()).view(6, H, dv)
    gd = wide.to(device)[:, cols - H * dv:]
    close(seqmix.head_gate(o.to(device), gd, torch.float32), want, 1e-6)
    strided = o.to(device).permute(1, 0, 2).contiguous().permute(1, 0, 2)                 # a batched product's layout
    close(seqmix.head_gate(strided, gd, torch.float32), want, 1e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_padded_heads_from_a_strided_query(device):
    g = torch.Generator().manual_seed(6)
    T, H, d, n, dv, W = 5, 3, 6, 8, 10, 16
    proj, k, v, kr = (torch.randn(*s, generator=g) for s in ((T, H * (d + n) + 9), (T, H, d), (T, H, dv), (T, n)))
    turns, amp = seqmix.rotary_turns(n, 20.0)
    pos = torch.tensor([3, 0, 99, 7, 12])
    dd = lambda t: t.to(device)  # noqa: E731
    qo, ko, vo = (torch.full((T, H, W), 5.0, device=device) for _ in range(3))
    q = dd(proj)[:, 4:4 + H * (d + n)].unflatten(1, (H, d + n))
    seqmix.latent_head_assemble(q, dd(k), dd(kr), dd(v), dd(turns), True, amp, dd(pos), qo, ko, vo)
    qd = proj[:, 4:4 + H * (d + n)].double().view(T, H, d + n)
    close(qo, torch.cat([qd[..., :d], oracle.rotate(qd[..., d:], pos.tolist(), oracle.frequencies(n, 20.0)), torch.zeros(T, H, W - d - n).double()], -1), 1e-5)
    close(ko, torch.cat([k.double(), kr.double().unsqueeze(1).expand(T, H, n), torch.zeros(T, H, W - d - n).double()], -1), 1e-6)
    close(vo, torch.cat([v, torch.zeros(T, H, W - dv)], -1).double(), 1e-6)


# ---------------------------------------------------------------------------------------------------------------------
# schedules: portions, decoding, batches, reuse
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[50], [1], [2, 2, 2], [2] * 25, [10, 11, 12], [4, 5, 30], [33, 3], [47]], ids=str)
def test_portions_and_decoding_match_whole_prompt(cuts, device):
    model, W = build(HYBRID, device)
    toks = tokens_of(50, seed=4)
    close(run_cut(replayer(model), "a", toks, cuts), oracle.forward(HYBRID, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_unequal_batch_matches_each_alone_and_pages_are_reused(device):
    model, W = build(HYBRID, device)
    rp = replayer(model, max_tokens=256, block_size=4, max_requests=3)
    prompts = {"a": tokens_of(23, seed=5), "b": tokens_of(1, seed=6), "c": tokens_of(14, seed=7)}
    want = {k: oracle.forward(HYBRID, W, v) for k, v in prompts.items()}
    cut = {"a": 17, "b": 1, "c": 9}
    out = rp.step([{"id": k, "tokens": v[:cut[k]], "want": list(range(cut[k]))} for k, v in prompts.items()])
    got = {k: [] for k in prompts}
    at = 0
    for k in prompts:
        got[k].append(out[at:at + cut[k]])
        at += cut[k]
    fed = dict(cut)
    live = [k for k in prompts if fed[k] < len(prompts[k])]
    rp.step([], end=[k for k in prompts if k not in live])
    while live:
        out = rp.step([{"id": k, "tokens": prompts[k][fed[k]:fed[k] + 1], "want": [0]} for k in live])
        for n, k in enumerate(live):
            got[k].append(out[n:n + 1])
            fed[k] += 1
        done = [k for k in live if fed[k] == len(prompts[k])]
        live = [k for k in live if k not in done]
        rp.step([], end=done)
    for k in prompts:
        close(torch.cat(got[k]), want[k], TOL)
    # the pages given back are used again by new requests: nothing old may show
    for n in range(4):
        toks = tokens_of(19 + n, seed=20 + n)
        close(run_cut(rp, f"again{n}", toks, [7, 2]), oracle.forward(HYBRID, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_portions_beside_decoding_in_one_batch(device):
    """A prompt's portion, a new prompt and a decoded token share a step."""
    model, W = build(HYBRID, device)
    rp = replayer(model, max_tokens=256)
    a, b, c = tokens_of(20, seed=40), tokens_of(9, seed=41), tokens_of(12, seed=42)
    rp.step([{"id": "a", "tokens": a[:8], "want": []}, {"id": "b", "tokens": b[:8], "want": []}])
    out = rp.step([{"id": "a", "tokens": a[8:], "want": [0, 11]}, {"id": "c", "tokens": c, "want": [11]}, {"id": "b", "tokens": b[8:], "want": [0]}])
    close(out[0:2], oracle.forward(HYBRID, W, a)[[8, 19]], TOL)
    close(out[2:3], oracle.forward(HYBRID, W, c)[[11]], TOL)
    close(out[3:4], oracle.forward(HYBRID, W, b)[[8]], TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_other_sizes_and_values_that_are_often_equal_or_one(device):
    """One head, one kv head, one unrotated dimension, a rank of one, a window of one, a rotated part larger than the rest, factor
    one, a multiplier and an embedding scale of one, layers without feed-forward, another eps, odd widths."""
    one = {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 3, "scale": 1.0, "mask": {"size": 1}, "rot": {"dims": 2, "base": 2.0}}}
    two = {"type": "attention", "mixer": {"heads": 5, "kv_heads": 1, "dim": 7, "vdim": 1, "scale": 2.0, "mask": {"size": 6},
                                          "rot": {"dims": 4, "base": 30.0, "scaling": {"factor": 1.0, "original": 16, "fast": 2.0, "slow": 1.0}}}}
    lat1 = {"type": "latent_attention", "mixer": {"heads": 1, "dim": 1, "rot_dim": 6, "vdim": 3, "kv_rank": 1, "scale": 1.0, "mask": {"size": 2},
                                                  "rot": {"base": 3.0, "dims": 6}}}
    lat2 = {"type": "latent_attention", "mixer": {"heads": 7, "dim": 9, "rot_dim": 2, "vdim": 1, "kv_rank": 65, "scale": 0.1, "mask": {"size": 12},
                                                  "rot": {"base": 8.0, "dims": 2}}}
    share1 = copy.deepcopy(lat1)
    share1["mixer"].update(kv_from=0, heads=4, dim=3, vdim=2, mask={"size": 40})
    f1, f5 = {"kind": "dense", "ff": 1}, {"kind": "dense", "ff": 5}
    for cfg in (config_of([dict(one, mlp=f1), layer("latent_attention", 2, f5), dict(lat1, mlp=None)], width=24, mult=1.0, scale=1.0),
                config_of([dict(lat1, mlp=f5), dict(share1, mlp=None), dict(two, mlp=f1), dict(share1, mlp=f1)], width=17, eps=1e-3, mult=0.2),
                config_of([dict(two, mlp=None), dict(lat2, mlp=f5)], width=40, vocab=33, eps=1e-6, scale=6.3),
                config_of([layer("attention", 1, FF)], width=6)):
        for seed in (11, 12):
            model, W = build(cfg, device, seed=seed)
            toks = tokens_of(29, vocab=cfg["vocab"], seed=8)
            close(run_cut(replayer(model), "a", toks, [13, 2, 9]), oracle.forward(cfg, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    """Windows pass over prompt and decoded tokens many times."""
    cfg = config_of([layer("latent_attention", 0, FF), layer("attention", 0), layer("latent_attention", 3, FF, kv_from=0)])
    model, W = build(cfg, device)
    toks = tokens_of(150, seed=9)
    close(run_cut(replayer(model), "a", toks, [6]), oracle.forward(cfg, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_through_the_engine(device):
    """The framework's own entry point: scheduler, chunked prefill under a token budget, sampling (greedy), retirement."""
    model, W = build(HYBRID, device)
    eng = DynamicInferenceEngine(model, NullTokenizer(VOCAB - 1), max_sequence_length=128, num_blocks=64, block_size=4,
                                 max_tokens_per_step=16, max_requests=3)
    prompts = [tokens_of(21, seed=30), tokens_of(5, seed=31), tokens_of(33, seed=32), tokens_of(2, seed=33)]
    ids = [eng.add_request("", SamplingParams(num_tokens_to_generate=6, top_k=1), prompt_tokens=p) for p in prompts]
    while eng.has_unfinished_requests():
        eng.step()
    checked = 0
    for rid, p in zip(ids, prompts):
        seq = list(p)
        for _ in range(6):
            logits = oracle.forward(HYBRID, W, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < 1e-3:
                break                                             # a close call is no test of the framework
            seq.append(int(torch.argmax(logits)))
            if seq[-1] == VOCAB - 1:
                break                                             # the end of text
        n = len(seq) - len(p)
        checked += n
        assert eng.completed[rid].generated_tokens.tolist()[:n] == seq[len(p):]
    assert checked >= 12


def test_bfloat16_serving_stays_within_rounding():
    model, W = build(HYBRID, "cpu", torch.bfloat16)
    toks = tokens_of(40, seed=12)
    want = oracle.forward(HYBRID, {k: v.to(torch.bfloat16) for k, v in W.items()}, toks)
    close_in_16_bits(run_cut(replayer(model), "a", toks, [25, 2]), want)


@pytest.mark.gpu
@pytest.mark.parametrize("width,att,lat,share", [
    (64, ATT_C, LAT_C, dict(LAT_C, heads=3, vdim=9, mask={"size": 75})),
    (72, {"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 48, "scale": 0.1, "mask": {"size": 50}, "rot": {"dims": 24, "base": 1000.0, "scaling": YARN}},
     {"heads": 4, "dim": 40, "rot_dim": 16, "vdim": 24, "kv_rank": 48, "scale": 0.15, "mask": {"size": 130}, "rot": {"dims": 16, "base": 1000.0}},
     {"heads": 2, "dim": 100, "rot_dim": 16, "vdim": 72, "kv_rank": 48, "scale": 0.1, "mask": {"size": 20}, "rot": {"dims": 16, "base": 1000.0}}),
    (128, {"heads": 3, "kv_heads": 3, "dim": 72, "vdim": 112, "scale": 0.1, "mask": {"size": 128}, "rot": {"dims": 72, "base": 1000.0}},
     {"heads": 3, "dim": 64, "rot_dim": 32, "vdim": 80, "kv_rank": 136, "scale": 0.1, "mask": {"size": 129}, "rot": {"dims": 32, "base": 1000.0}},
     {"heads": 2, "dim": 128, "rot_dim": 32, "vdim": 64, "kv_rank": 136, "scale": 0.1, "mask": {"size": 127}, "rot": {"dims": 32, "base": 1000.0}})],
    ids=["odd", "narrow", "wide"])
def test_bfloat16_kernels_stay_within_rounding_whole_prompts_batches_and_decoding(width, att, lat, share):
    """Prompts long enough for the tcgen05 kernel (several in one step, across tile edges), then decoding; and the same tokens
    in portions, which run on the paged kernels.  In the last case the sharing layer's heads are too wide for the tcgen05 kernel."""
    ff = {"kind": "dense", "ff": 96}
    cfg = config_of([{"type": "attention", "mixer": att, "mlp": ff}, {"type": "latent_attention", "mixer": lat, "mlp": None},
                     {"type": "latent_attention", "mixer": dict(share, kv_from=1), "mlp": ff}], width=width)
    model, W = build(cfg, "cuda", torch.bfloat16)
    Wb = {k: v.to(torch.bfloat16) for k, v in W.items()}
    prompts = [tokens_of(n, seed=50 + n) for n in (70, 131, 300)]
    wants = [oracle.forward(cfg, Wb, p) for p in prompts]
    rp = replayer(model, max_tokens=1024, block_size=16)
    n0 = [len(p) - 3 for p in prompts]
    out = rp.step([{"id": str(i), "tokens": p[:n0[i]], "want": list(range(n0[i]))} for i, p in enumerate(prompts)])
    rows = list(torch.split(out, n0))
    for k in range(3):
        out = rp.step([{"id": str(i), "tokens": [p[n0[i] + k]], "want": [0]} for i, p in enumerate(prompts)])
        rows = [torch.cat([r, out[i:i + 1]]) for i, r in enumerate(rows)]
    for r, w in zip(rows, wants):
        close_in_16_bits(r, w, typical=2e-2)
    close_in_16_bits(run_cut(replayer(model, max_tokens=1024), "b", prompts[2], [100, 2, 90, 105]), rows[2].double(), typical=2e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,d,dv,window,sink,gated,lens", [
    (2, 1, 64, 64, 0, False, False, [256]), (3, 3, 64, 64, 128, True, True, [1, 64, 127, 128, 129, 130]), (4, 2, 128, 128, 127, False, True, [255, 257, 384, 5]),
    (4, 1, 40, 48, 1, True, False, [300, 70]), (2, 2, 96, 100, 129, True, True, [200, 129, 700]), (2, 1, 128, 72, 300, True, True, [140, 1000]),
    (1, 1, 24, 14, 64, False, True, [90, 515]), (5, 5, 17, 31, 255, True, True, [640, 3]), (2, 1, 64, 64, 256, False, False, [897]), (2, 1, 64, 64, 5000, True, False, [300])])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16], ids=["bf16", "fp16"])
def test_tcgen05_window_attention_matches_the_equations(H, G, d, dv, window, sink, gated, lens, dtype):
    from megatronapp_b200 import ops

    g = torch.Generator().manual_seed(7)
    T = sum(lens)
    width = 64 if max(d, dv) <= 64 else 128
    q, k, v = (torch.randn(T, h, n, generator=g).to(dtype) for h, n in ((H, d), (G, d), (G, dv)))
    k[::37] *= 4.0                                                      # some loud keys: the running maximum moves late
    k[::53] *= -6.0
    sk = torch.linspace(-4.0, 5.0, H).to(dtype) if sink else None
    wide = torch.randn(T, H * dv + 8, generator=g).to(dtype)
    qp, kp, vp = (torch.zeros(T, h, width, dtype=dtype, device="cuda") for h in (H, G, G))
    qp[..., :d], kp[..., :d], vp[..., :dv] = q.cuda(), k.cuda(), v.cuda()
    cu = torch.tensor([sum(lens[:i]) for i in range(len(lens) + 1)], dtype=torch.int32, device="cuda")
    gd = wide.cuda()[:, 8:] if gated else None
    got = ops.window_attention(qp, kp, vp, cu, max(lens), 0.3, window, None if sk is None else sk.cuda(), gd, dv).view(T, H, dv).float().cpu()
    assert ops.ext().window_attn_status() == 0
    at = 0
    for n in lens:
        Q, K, V = q[at:at + n].double(), k[at:at + n].double().repeat_interleave(H // G, 1), v[at:at + n].double().repeat_interleave(H // G, 1)
        s = torch.einsum("thd,lhd->htl", Q, K) * 0.3
        i, j = torch.arange(n).view(-1, 1), torch.arange(n).view(1, -1)
        s = s.masked_fill(~((j <= i) & ((i - j < window) | (window == 0))), float("-inf"))
        if sink:
            s = torch.cat([s, sk.double().view(H, 1, 1).expand(H, n, 1)], -1)
        w = torch.softmax(s, -1)[..., :n]
        want, scale = torch.einsum("htl,lhv->thv", w, V), torch.einsum("htl,lhv->thv", w, V.abs())
        if gated:
            gate = oracle.sig(wide[at:at + n, 8:].double()).view(n, H, dv)
            want, scale = want * gate, scale * gate
        err = (got[at:at + n].double() - want).abs()                    # rounding is relative to the sum of magnitudes
        assert float((err / (scale.amax(-1, keepdim=True) + 1e-3)).max()) < 1.2e-2
        at += n


@pytest.mark.gpu
def test_tcgen05_window_attention_with_scores_far_below_zero():
    """Early rows of a tile see nothing of its first key block; all scores are so low that a maximum of zero would lose them."""
    from megatronapp_b200 import ops

    T, window = 400, 20
    q, k = torch.full((T, 1, 64), -2.0), torch.full((T, 1, 64), 2.0)
    v = torch.arange(T, dtype=torch.float32).view(T, 1, 1).expand(T, 1, 64) / 128.0
    D = lambda t: t.to("cuda", torch.bfloat16).contiguous()  # noqa: E731
    got = ops.window_attention(D(q), D(k), D(v), torch.tensor([0, T], dtype=torch.int32, device="cuda"), T, 1.0, window).float().cpu()
    vb = v[:, 0, 0].to(torch.bfloat16).double()
    want = torch.stack([vb[max(0, i - window + 1):i + 1].mean() for i in range(T)])
    close(got[:, 0], want, 1e-2), close(got[:, 63], want, 1e-2)


# ---------------------------------------------------------------------------------------------------------------------
# edges that random weights hide: one key that matters just inside and just outside the window, at page borders, at the start
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("ctx_len,window,j", [(n, w, j) for n, w in ((5, 3), (64, 16), (65, 16), (65, 33), (300, 64), (300, 299), (300, 300), (1200, 640))
                                              for j in (n - w - 1, n - w, n - w + 1, n - 1, 0) if 0 <= j < n] + [(1200, 0, 0), (1200, 0, 639)])
def test_attentions_see_one_marked_key_inside_the_window_only(ctx_len, window, j, device):
    """All keys are small but one, whose value is marked.  Inside the window the mark takes the softmax, outside it leaves no trace.
    Whole prompt, last token alone, decoding batch with split keys; grouped queries and latents (marked in the rotated key part)."""
    H, G, dd, dv, bs = 2, 1, 8, 6, 16
    g = torch.Generator().manual_seed(ctx_len + j)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    D = lambda t: t.to(device)  # noqa: E731
    rnd = lambda *s: torch.randn(*s, generator=g) * 0.01  # noqa: E731
    seen = window == 0 or ctx_len - 1 - j < window
    table, n_slots, (slots,) = paged([ctx_len], bs, seed=j)
    whole_rows = (i32([0] * ctx_len), i32(list(range(1, ctx_len + 1))))
    k, v, q = rnd(ctx_len, G, dd), rnd(ctx_len, G, dv), rnd(ctx_len, H, dd)
    k[j, 0, 0], v[j, 0], q[-1, :, 0] = 8.0, 5.0, 8.0
    want = oracle.window_attention(q[-1:].double(), k.double(), v.double(), 1.0, window, first=ctx_len - 1)[0]
    assert float(want.min()) > 4.9 if seen else float(want.abs().max()) < 0.1
    kc, vc = torch.zeros(n_slots, G, dd), torch.zeros(n_slots, G, dv)
    kc[slots], vc[slots] = k, v
    whole = seqmix.window_attention_paged(D(q), D(kc), D(vc), D(table), *whole_rows, bs, 1.0, window)
    close(whole[-1].view(H, dv), want, 1e-5)
    for ml in (0, ctx_len):
        alone = seqmix.window_attention_paged(D(q[-1:]), D(kc), D(vc), D(table), i32([0]), i32([ctx_len]), bs, 1.0, window, max_len=ml)
        close(alone[0].view(H, dv), want, 1e-5)
    r, n = 20, 4
    c, kr = torch.randn(ctx_len, r, generator=g), rnd(ctx_len, n)
    kr[j] = torch.tensor([9.0, 0.0, 0.0, 9.0])
    ql, qr = rnd(ctx_len, H, r), rnd(ctx_len, H, n)
    qr[-1] = torch.tensor([3.0, 0.0, 0.0, 3.0])
    sink = torch.tensor([2.0, -1.0])
    lat = oracle.latent_attention(ql[-1:].double(), qr[-1:].double(), c.double().unsqueeze(1).expand(ctx_len, H, r), kr.double(),
                                  c.double().unsqueeze(1).expand(ctx_len, H, r), 1.0, window, sink.double(), first=ctx_len - 1)[0]
    assert not seen or float((lat - c[j].double()).abs().max()) < 1e-3
    cache = torch.zeros(n_slots, r + n)
    cache[slots] = torch.cat([c, kr], 1)
    whole = seqmix.latent_attention_paged(D(ql), D(cache), D(table), *whole_rows, bs, 1.0, ctx_len, D(qr), None, window, D(sink))
    close(whole[-1], lat, 1e-5)
    alone = seqmix.latent_attention_paged(D(ql[-1:]), D(cache), D(table), i32([0]), i32([ctx_len]), bs, 1.0, ctx_len, D(qr[-1:]), None, window, D(sink))
    close(alone[0], lat, 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 64, 127, 128, 129, 256, 300])
def test_tcgen05_window_edges(window):
    """Every query is orthogonal to all keys but loves the one at distance ``gap``: seen up to ``window - 1``, not at ``window``."""
    from megatronapp_b200 import ops

    T, B = 640, 64
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    pos = torch.arange(T)
    v = torch.zeros(T, 1, B)
    v[:, 0, 0] = (pos % 7).float() + 1.0
    for gap in {0, window - 1, window, window + 1}:
        # key p carries class p mod 41, query i asks for the class of i - gap: the class repeats within the window now and then, so
        # the reference is the equations, not the single mark
        k, q = torch.zeros(T, 1, B), torch.zeros(T, 1, B)
        k[pos, 0, pos % 41] = 1.0
        q[pos, 0, (pos - gap) % 41] = 1.0
        D = lambda t: t.to("cuda", torch.bfloat16).contiguous()  # noqa: E731
        got = ops.window_attention(D(q), D(k), D(v), cu, T, 12.0, window).float().cpu()[:, 0]
        close(got, oracle.window_attention(q.double(), k.double(), v.double(), 12.0, window)[:, 0, 0], 1.2e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind,variant", [("attention", 0), ("latent_attention", 0)])
def test_a_token_is_felt_for_exactly_its_window(kind, variant, device):
    """One layer: two prompts that differ in one token differ in exactly ``window`` positions, prompt or decoded, on page borders."""
    cfg = config_of([layer(kind, variant, None)])
    w = cfg["layers"][0]["mixer"]["mask"]["size"]
    model, W = build(cfg, device)
    a = tokens_of(34, seed=1)
    for at in (0, 7, 8, 15):
        b = list(a)
        b[at] = (b[at] + 1) % VOCAB
        for cuts in ([34], [at + 1], [at + w - 1], [at + w], [6, 2, 3]):
            la, lb = run_cut(replayer(model), "a", a, cuts), run_cut(replayer(model), "b", b, cuts)
            assert [t for t in range(34) if float((la[t] - lb[t]).abs().max()) > 1e-5] == list(range(at, at + w))


@pytest.mark.parametrize("device", DEVICES)
def test_first_tokens_share_the_denominator_with_the_sink(device):
    """Zero queries: token ``t`` averages what the window holds, diluted by ``exp(sink)`` beside as many ones; a huge sink leaves
    nothing, a sink of minus infinity is no sink."""
    T, r, w = 9, 4, 5
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    cache = torch.arange(1, T + 1, dtype=torch.float32).view(T, 1).repeat(1, r + 2)
    sink = torch.tensor([0.0, 1.5, 80.0, float("-inf")])
    got = seqmix.latent_attention_paged(torch.zeros(T, 4, r, device=device), cache.to(device), i32([[0]]), i32([0] * T), i32(list(range(1, T + 1))), T,
                                        3.0, T, torch.zeros(T, 4, 2, device=device), None, w, sink.to(device))
    for t in range(T):
        vals = torch.arange(max(0, t - w + 1), t + 1).double() + 1.0
        close(got[t, :, 0], torch.stack([vals.sum() / (len(vals) + torch.exp(s.double())) for s in sink]), 1e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_a_sharing_layer_reads_rows_of_decoded_and_reused_pages(device):
    """Freed pages hold another request's rows when the source layer writes them anew: the sharing layer must see the new ones, in a
    window longer than its source's."""
    cfg = config_of([layer("latent_attention", 0, None, mask={"size": 3}), layer("attention", 1), layer("latent_attention", 3, FF, kv_from=0, mask={"size": 26})])
    model, W = build(cfg, device, seed=3)
    rp = replayer(model, max_tokens=40, block_size=4, max_requests=2)
    for n in range(5):
        toks = tokens_of(30 + n, seed=60 + n)
        close(run_cut(rp, f"r{n}", toks, [[30], [1], [2, 2], [9, 9, 9], [28]][n]), oracle.forward(cfg, W, toks), TOL)


def test_config_reads_its_keys_and_rejects_bad_values():
    c = DufitarConfig.from_dict(HYBRID)
    assert (len(c.layers), c.width, c.norm_eps, c.embedding_scale, c.residual_mult) == (7, 32, 1e-5, 1.9, 0.7)
    bad = config_of([layer("attention")])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        DufitarConfig.from_dict(bad)
    with pytest.raises(ValueError):
        DufitarConfig.from_dict(config_of([layer("attention", 0, {"kind": "moe"})]))
    for layers in ([layer("latent_attention", 3, kv_from=0)], [layer("attention"), layer("latent_attention", 3, kv_from=0)],
                   [layer("latent_attention"), layer("latent_attention", 3, kv_from=0), layer("latent_attention", 3, kv_from=1)]):
        with pytest.raises(ValueError):
            DufitarConfig.from_dict(config_of(layers))
    raw = config_of([layer("latent_attention", 0, {"kind": "dense"})])
    del raw["layers"][0]["mixer"]["kv_rank"]
    filled = shapes_into_config(raw, {"l0.mix.uk": (24, 12), "l0.mlp.up": (18, 32)})
    assert filled["layers"][0]["mixer"]["kv_rank"] == 12 and filled["layers"][0]["mlp"]["ff"] == 18
    model, W = build(config_of([layer("attention")]), "cpu")
    with pytest.raises(KeyError):
        load_dufitar_weights(model, {k: v for k, v in W.items() if k != "l0.norm1.alpha"})
    with pytest.raises(ValueError):
        load_dufitar_weights(model, dict(W, extra=torch.zeros(1)))


# ---------------------------------------------------------------------------------------------------------------------
# a model folder through the registry, the trace runner and its command line
# ---------------------------------------------------------------------------------------------------------------------
def write_safetensors(path, tensors):
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(-1).view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


def test_model_folder_through_registry_and_trace_runner_command_line(tmp_path):
    from megatronapp_b200.models.registry import architectures, build_model_from_dir

    assert "dufitar" in architectures()
    cfg = config_of([layer("latent_attention", 0, FF), layer("attention", 1), layer("latent_attention", 3, FF_B, kv_from=0)])
    W = {k: v.to(torch.bfloat16) for k, v in oracle.random_weights(cfg, 5).items()}
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), W)
    model = build_model_from_dir(str(folder), torch.float32, "cpu")
    toks = tokens_of(16, seed=3)
    want = oracle.forward(cfg, W, toks)
    close(run_cut(replayer(model), "a", toks, [16]), want, TOL)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:13], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[13:14], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[14:], "want": [1]}], "end": ["x"]}]
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    got0 = torch.frombuffer(bytearray((out / "0.f32").read_bytes()), dtype=torch.float32).view(2, -1)
    got2 = torch.frombuffer(bytearray((out / "2.f32").read_bytes()), dtype=torch.float32).view(1, -1)
    close(got0, want[[0, 8]], TOL)
    close(got2, want[[15]], TOL)
    # the generation command line on the same folder: greedy tokens of the oracle (a close call is no test)
    prompt, gen = toks[:9], []
    for _ in range(4):
        top2 = torch.topk(oracle.forward(cfg, W, prompt + gen)[-1], 2)
        if float(top2.values[0] - top2.values[1]) < 1e-3 or int(top2.indices[0]) == VOCAB - 1:     # the last token ends a text
            break
        gen.append(int(top2.indices[0]))
    assert gen
    r = subprocess.run([sys.executable, os.path.join(root, "tools", "run_text_generation_server.py"), "--model-dir", str(folder),
                        "--dtype", "float32", "--prompts", " ".join(map(str, prompt)), "--num-tokens-to-generate", "4"],
                       capture_output=True, text=True, env=dict(os.environ, CUDA_VISIBLE_DEVICES=""), timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    said = r.stdout.strip().splitlines()[-1].split("-> ")[-1].strip("'\"").split()
    assert [int(t) for t in said][:len(gen)] == gen
