"""Nasipel models in the framework against a plain, slow evaluation of the design's equations (``nasipel_oracle``).

Each test builds its own small configuration and random (or hand-made) weights, loads them through the product loader
and drives the model through the dynamic engine -- whole prompts, prompts cut into portions, token-by-token decoding,
mixed batches, reused pages and state rows -- on the CPU (PyTorch op path) and, marked ``gpu``, on the sm_100a kernels.
"""
import copy
import json
import math
import os
import struct
import subprocess
import sys

import pytest
import torch

import nasipel_oracle as oracle
from megatronapp_b200.data.tokenizer import NullTokenizer
from megatronapp_b200.inference import DynamicInferenceEngine, SamplingParams
from megatronapp_b200.inference.trace import TraceReplayer
from megatronapp_b200.models.nasipel import NasipelConfig, NasipelModel
from megatronapp_b200.models.nasipel.loader import load_nasipel_weights, shapes_into_config
from megatronapp_b200.ops import seqmix
from megatronapp_b200.ops.seqmix import HeadPart
from megatronapp_b200.parallel import state as ps

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
VOCAB = 61
YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}

ATT = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.4, "softcap": 3.0, "rot": {"dims": 8, "base": 50.0}}
ATT_B = {"heads": 3, "kv_heads": 3, "dim": 20, "vdim": 6, "scale": 0.2, "softcap": 10.0, "rot": {"dims": 6, "base": 10000.0}}   # part of a head turns
ATT_C = {"heads": 6, "kv_heads": 1, "dim": 16, "vdim": 40, "scale": 0.25, "rot": {"dims": 16, "base": 300.0}}                   # no cap
LRU = {"width": 24, "blocks": 3, "conv": 3}
LRU_B = {"width": 40, "blocks": 5, "conv": 2}
LRU_C = {"width": 36, "blocks": 1, "conv": 5}
LAT = {"heads": 3, "dim": 8, "rot_dim": 4, "vdim": 6, "q_rank": 10, "kv_rank": 12, "scale": 0.3, "rot": {"dims": 4, "base": 20.0, "scaling": YARN}}
LAT_B = {"heads": 2, "dim": 6, "rot_dim": 8, "vdim": 10, "q_rank": 14, "kv_rank": 20, "scale": 0.25,
         "rot": {"dims": 8, "base": 10000.0, "scaling": dict(YARN, factor=8.0, original=128, fast=16.0, slow=2.0)}}
LAT_C = {"heads": 5, "dim": 12, "rot_dim": 6, "vdim": 12, "q_rank": 8, "kv_rank": 40, "scale": 0.2, "rot": {"dims": 6, "base": 100.0}}   # no scaling
MIX = {"attention": (ATT, ATT_B, ATT_C), "rglru": (LRU, LRU_B, LRU_C), "latent_attention": (LAT, LAT_B, LAT_C)}
MOE = {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 6, "top": 2, "scale": 1.7, "groups": {"count": 3, "keep": 2}}}
MOE_B = {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 8, "top": 3, "scale": 0.6, "groups": {"count": 2, "keep": 1}}}
MOE_C = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 4, "top": 4, "scale": 2.5, "groups": {"count": 2, "keep": 2}}}   # every expert
MOE_D = {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 1}}                                                     # no groups, top 1


def layer(kind, variant=0, mlp=None):
    return {"type": kind, "mixer": copy.deepcopy(MIX[kind][variant]), "mlp": copy.deepcopy(mlp)}


def config_of(layers, width=32, vocab=VOCAB, eps=1e-5):
    return {"architecture": "Nasipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


HYBRID = config_of([layer("attention", 0, MOE), layer("rglru", 0, MOE_B), layer("latent_attention", 0, MOE_D), layer("rglru", 1),
                    layer("attention", 1, MOE_C), layer("latent_attention", 1)])


def build(cfg, device, dtype=torch.float32, seed=0, weights=None):
    if not ps.model_parallel_is_initialized():
        ps.initialize_model_parallel(1, 1)
    W = weights if weights is not None else oracle.random_weights(cfg, seed)
    raw = shapes_into_config(copy.deepcopy(cfg), {k: tuple(v.shape) for k, v in W.items()})
    ncfg = NasipelConfig.from_dict(raw)
    model = NasipelModel(ncfg, ncfg.base_transformer_config(dtype, use_cpu_initialization=True, perform_initialization=False))
    load_nasipel_weights(model, W)
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


TOL = 2e-4


def close_in_16_bits(got, want, typical=3e-2, outlier=0.15, share=0.1):
    """Rounding to 16 bits is amplified where a norm divides by something small: a few positions may be far off, the typical
    one must be near (root mean square over the vocabulary, relative to the logits' scale)."""
    want = want.to(torch.float64)
    rel = (got.to(torch.float64).cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(rel.median()) <= typical and float((rel > outlier).double().mean()) <= share, \
        f"median {float(rel.median()):.3e}, worst {float(rel.max()):.3e}"


# ---------------------------------------------------------------------------------------------------------------------
# every mechanism alone: one layer, whole prompt and cut prompt
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("spec", [layer(k, v) for k in MIX for v in range(3)] + [layer("rglru", 0, m) for m in (MOE, MOE_B, MOE_C, MOE_D)],
                         ids=[f"{k}{v}" for k in MIX for v in range(3)] + ["moe_groups", "moe_one_group_kept", "moe_every_expert", "moe_top1"])
def test_single_mechanism_matches_oracle(spec, device):
    cfg = config_of([spec])
    model, W = build(cfg, device, seed=1)
    toks = tokens_of(37)
    want, layers = oracle.forward(cfg, W, toks, return_layers=True)
    seen = []
    model.decoder.tap = lambda i, x: seen.append(x.detach().float().cpu().clone())
    rp = replayer(model)
    close(run_cut(rp, "a", toks, [len(toks)]), want, TOL)
    close(seen[0].view(len(toks), -1), layers[0], TOL)
    model.decoder.tap = None
    close(run_cut(rp, "b", toks, [17, 2, 16]), want, TOL)


def test_whole_sequence_forward_without_a_context():
    """The training-style call (``[b, s]`` ids, no inference context) runs the same mixers from zero state."""
    model, W = build(HYBRID, "cpu")
    a, b = tokens_of(21, seed=1), tokens_of(21, seed=2)
    out = model(torch.tensor([a, b]), None, None)
    close(out[0], oracle.forward(HYBRID, W, a), TOL)
    close(out[1], oracle.forward(HYBRID, W, b), TOL)


# ---------------------------------------------------------------------------------------------------------------------
# ops against the oracle's functions
# ---------------------------------------------------------------------------------------------------------------------
def paged(lens, block_size, heads, seed=0):
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
@pytest.mark.parametrize("width", [20, 22, 192])
@pytest.mark.parametrize("center", [True, False])
def test_gated_additions_and_their_norms(width, center, device):
    g = torch.Generator().manual_seed(0)
    T = 7
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    d = lambda t: None if t is None else t.to(device)  # noqa: E731
    norm = (lambda t: oracle.layer_norm(t, 1e-3)) if center else (lambda t: oracle.rms(t, 1e-3))
    x, a, b, wide = rnd(T, width) + 3.0, rnd(T, width), rnd(T, width), rnd(T, 3 * width)
    ba, bb, w1, w2 = rnd(width), rnd(width), rnd(width), rnd(width)
    ga, gb = wide[:, :width], wide[:, 2 * width:]                      # column slices of a wider projection
    D = lambda t: t.double()  # noqa: E731
    x1 = D(x) + oracle.sig(D(ga) + D(ba)) * D(a) + oracle.sig(D(gb) + D(bb)) * D(b)
    wd = d(wide)
    gx, h1, h2 = seqmix.gated_add_norm(d(x.clone()), d(a), wd[:, :width], d(ba), d(b), wd[:, 2 * width:], d(bb), d(w1), d(w2), 1e-3,
                                       torch.float32, center)
    close(gx, x1, 1e-5), close(h1, norm(x1) * D(w1), 1e-5), close(h2, norm(x1) * D(w2), 1e-5)
    gx, h1, h2 = seqmix.gated_add_norm(d(x.clone()), d(a), wd[:, :width], None, None, None, None, d(w1), None, 1e-3, torch.float32, center)
    x2 = D(x) + oracle.sig(D(ga)) * D(a)
    assert h2 is None
    close(gx, x2, 1e-5), close(h1, norm(x2) * D(w1), 1e-5)
    gx, h1, _ = seqmix.gated_add_norm(d(x.clone()), None, None, None, d(b), None, None, d(w1), None, 1e-3, torch.float32, center)
    close(gx, D(x) + D(b), 1e-5), close(h1, norm(D(x) + D(b)) * D(w1), 1e-5)
    gx, h1, h2 = seqmix.gated_add_norm(d(x.clone()), None, None, None, None, None, None, d(w1), d(w2), 1e-3, torch.float32, center)
    close(gx, D(x), 1e-6), close(h2, norm(D(x)) * D(w2), 1e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_head_rotation_norm_padding_and_pages(device):
    """Three operands in one launch: halves with a norm, interleaved with an amplitude, turned back and split into padded halves;
    to dense outputs and to shuffled cache rows; a table of the angles on the side."""
    g = torch.Generator().manual_seed(1)
    T = 6
    proj = torch.randn(T, 90, generator=g)
    pos = torch.tensor([0, 1, 5, 700, 3, 40])
    slots = torch.tensor([9, 2, 4, 0, 7, 11])
    w = torch.randn(10, generator=g)
    q, k, v = proj[:, :40].unflatten(1, (4, 10)), proj[:, 40:60].unflatten(1, (2, 10)), proj[:, 60:84].unflatten(1, (2, 12))
    tq, _ = seqmix.rotary_turns(6, 30.0)
    tk, amp = seqmix.rotary_turns(8, 100.0, YARN)
    tv, _ = seqmix.rotary_turns(12, 30.0)
    assert amp == pytest.approx(oracle.amplitude(YARN))
    d = lambda t: t.to(device)  # noqa: E731
    pd = d(proj)
    qd, kd, vd = pd[:, :40].unflatten(1, (4, 10)), pd[:, 40:60].unflatten(1, (2, 10)), pd[:, 60:84].unflatten(1, (2, 12))
    qo, vo = torch.full((T, 4, 16), 7.0, device=device), torch.full((T, 2, 32), 7.0, device=device)
    kp, vp = torch.zeros(12, 2, 10, device=device), torch.zeros(12, 2, 12, device=device)
    tab = torch.zeros(T, 6, 2, device=device)
    seqmix.head_rotary([HeadPart(qd, d(tq), rms=True, weight=d(w), out=qo), HeadPart(kd, d(tk), True, amp, rms=True, pages=kp),
                        HeadPart(vd, d(tv), back=True, out=vo, pages=vp, out_half=16, table=tab)], d(pos), 1e-5, d(slots))
    P = pos.tolist()
    wq = oracle.rms(oracle.rotate(q.double(), P, oracle.frequencies(6, 30.0)), 1e-5) * w.double()
    wk = oracle.rms(oracle.rotate(k.double(), P, oracle.frequencies(8, 100.0, YARN), True, oracle.amplitude(YARN)), 1e-5)
    wv = oracle.rotate(v.double(), P, oracle.frequencies(12, 30.0), back=True)
    close(qo[..., :10], wq, 1e-5), close(kp[slots], wk, 1e-5), close(vp[slots], wv, 1e-5)
    assert float(qo[..., 10:].abs().max()) == 0.0 and float(kp[[1, 3, 5, 6, 8, 10]].abs().max()) == 0.0
    close(vo[..., :6], wv[..., :6], 1e-5), close(vo[..., 16:22], wv[..., 6:], 1e-5)
    assert float(vo[..., 6:16].abs().max()) == 0.0 and float(vo[..., 22:].abs().max()) == 0.0
    ang = -pos.double().unsqueeze(1) * torch.tensor(oracle.frequencies(12, 30.0), dtype=torch.float64)
    close(tab[..., 0], torch.cos(ang), 1e-5), close(tab[..., 1], torch.sin(ang), 1e-5)
    # the same head untouched: no turns, no norm
    out = torch.empty(T, 4, 10, device=device)
    seqmix.head_rotary([HeadPart(qd, out=out)], d(pos), 1e-5)
    close(out, q.double(), 1e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_far_positions_keep_their_angle(device):
    """The angle of position 200 000 is right to fp32, which a single fp32 product would miss by hundredths of a turn."""
    turns, _ = seqmix.rotary_turns(8, 10000.0)
    pos = torch.tensor([0, 1, 4095, 200000, 1000003])
    x = torch.randn(5, 1, 8, generator=torch.Generator().manual_seed(0))
    out = torch.empty(5, 1, 8, device=device)
    seqmix.head_rotary([HeadPart(x.to(device), turns.to(device), out=out)], pos.to(device), 0.0)
    close(out, oracle.rotate(x.double(), pos.tolist(), oracle.frequencies(8, 10000.0)), 1e-6)


def test_yarn_rates_at_both_ends_and_between():
    for dims, base, sc in ((24, 20000.0, {"factor": 3.0, "original": 1024, "fast": 24.0, "slow": 1.5}), (8, 50.0, YARN),
                           (64, 10000.0, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (4, 3.0, {"factor": 3.0, "original": 8, "fast": 1.0, "slow": 1.0})):
        turns, amp = seqmix.rotary_turns(dims, base, sc)
        want = torch.tensor(oracle.frequencies(dims, base, sc), dtype=torch.float64) / (2 * math.pi)
        assert float((turns.double().sum(-1) / want - 1).abs().max()) < 1e-12
        assert amp == pytest.approx(0.1 * math.log(sc["factor"]) + 1.0)
    plain = seqmix.rotary_turns(24, 20000.0)[0].double().sum(-1)
    scaled = seqmix.rotary_turns(24, 20000.0, {"factor": 3.0, "original": 1024, "fast": 24.0, "slow": 1.5})[0].double().sum(-1)
    ratio = plain / scaled
    assert float(ratio[0]) == pytest.approx(1.0) and float(ratio[-1]) == pytest.approx(3.0) and bool(((ratio > 1.01) & (ratio < 2.99)).any())
    assert seqmix.rotary_turns(0, 10.0) == (None, 1.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("H,G,d,dv,cap,inter", [(4, 2, 6, 10, 3.0, False), (6, 1, 20, 14, 0.0, True), (3, 3, 32, 64, 20.0, False),
                                                (12, 2, 64, 72, 15.0, False), (1, 1, 40, 130, 1.0, False)])
def test_logistic_attention_prompts_and_decoding_batches(H, G, d, dv, cap, inter, dtype, device):
    """Unequal sequences over shuffled pages: all tokens as prompts in one call, then the last token of each as a decoding batch
    (the split path on the GPU), both against the oracle with rotated-back results."""
    lens, bs = [3, 40, 130], 8
    g = torch.Generator().manual_seed(2)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    table, n_slots, slots = paged(lens, bs, H)
    kc, vc = torch.zeros(n_slots, G, d), torch.zeros(n_slots, G, dv)
    bias = torch.randn(H, generator=g) - 1.0
    qs, wants = [], []
    fr = oracle.frequencies(dv, 40.0)
    for r, n in enumerate(lens):
        q, k, v = rnd(n, H, d), rnd(n, G, d), rnd(n, G, dv)
        kc[slots[r]], vc[slots[r]] = k, v
        qs.append(q)
        o = oracle.sigmoid_attention(q.double(), k.double(), v.double(), 0.3, cap, bias.double())
        wants.append(oracle.rotate(o, range(n), fr, inter, back=True))
    turns = seqmix.rotary_turns(dv, 40.0)[0].to(device)
    D = lambda t: t.to(device, dtype)  # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    got = seqmix.sigmoid_attention_paged(D(torch.cat(qs)), D(kc), D(vc), table.to(device), i32([r for r, n in enumerate(lens) for _ in range(n)]),
                                         i32([i + 1 for n in lens for i in range(n)]), bs, 0.3, cap, bias.to(device), turns, inter)
    close(got.view(-1, H, dv).float(), torch.cat(wants), tol)
    got = seqmix.sigmoid_attention_paged(D(torch.cat([q[-1:] for q in qs])), D(kc), D(vc), table.to(device), i32([0, 1, 2]), i32(lens), bs, 0.3,
                                         cap, bias.to(device), turns, inter, max_len=max(lens))
    close(got.view(-1, H, dv).float(), torch.cat([w[-1:] for w in wants]), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("H,d,n,dv,r,gated", [(3, 8, 4, 6, 12, True), (5, 6, 10, 6, 40, False), (16, 16, 32, 16, 96, True), (2, 8, 16, 24, 260, True),
                                              (20, 8, 64, 8, 512, True)])
def test_latent_attention_with_a_rotated_part(H, d, n, dv, r, gated, dtype, device):
    lens, bs = [5, 33, 270], 16
    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    table, n_slots, slots = paged(lens, bs, H)
    cache = torch.zeros(n_slots, r + n)
    wk = (torch.randn(H, d, r, generator=g) * r ** -0.5)
    gate_all = torch.randn(sum(lens), H + 3, generator=g).to(dtype).float()
    ql, qr, wants, at = [], [], [], 0
    for q_, L in enumerate(lens):
        c, kr, qn, q2 = rnd(L, r), rnd(L, n), rnd(L, H, d), rnd(L, H, n)
        cache[slots[q_], :r], cache[slots[q_], r:] = c, kr
        lat = torch.einsum("thd,hdr->thr", qn, wk).to(dtype).float()
        ql.append(lat), qr.append(q2)
        o = torch.zeros(L, H, r, dtype=torch.float64)
        for h in range(H):                                              # the values are the latents themselves
            o[:, h] = oracle.latent_attention(lat[:, h:h + 1].double(), q2[:, h:h + 1].double(), c.double().unsqueeze(1), kr.double(),
                                              c.double().unsqueeze(1), 0.2)[:, 0] if L <= 33 else torch.softmax(
                ((lat[:, h].double() @ c.double().T + q2[:, h].double() @ kr.double().T) * 0.2).masked_fill(
                    torch.ones(L, L).triu(1).bool(), float("-inf")), -1) @ c.double()
        if gated:
            o = o * oracle.sig(gate_all[at:at + L, 1:H + 1].double()).unsqueeze(-1)
        at += L
        wants.append(o)
    D = lambda t: t.to(device, dtype)  # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    ga = D(gate_all)[:, 1:H + 1] if gated else None
    got = seqmix.latent_attention_paged(D(torch.cat(ql)), D(cache), table.to(device), i32([q_ for q_, L in enumerate(lens) for _ in range(L)]),
                                        i32([i + 1 for L in lens for i in range(L)]), bs, 0.2, max(lens), D(torch.cat(qr)), ga)
    close(got.float(), torch.cat(wants), tol)
    ends = [sum(lens[:q_ + 1]) - 1 for q_ in range(3)]
    got = seqmix.latent_attention_paged(D(torch.cat(ql))[ends], D(cache), table.to(device), i32([0, 1, 2]), i32(lens), bs, 0.2, max(lens),
                                        D(torch.cat(qr))[ends], ga[ends] if gated else None)
    close(got.float(), torch.cat([w[-1:] for w in wants]), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("C,B", [(24, 3), (40, 1), (144, 2), (240, 3), (256, 2), (512, 2)])
def test_recurrent_unit_over_runs_and_steps(C, B, dtype, device):
    """Three sequences (one of several runs), fed whole and then in portions down to one token from carried state; decays near one
    and near zero; strided inputs."""
    g = torch.Generator().manual_seed(4)
    n = C // B
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    lens = [300, 1, 70]
    w, bias, lam = rnd(B, 2, n, n) * n ** -0.5, rnd(B, 2, n), rnd(C) * 3.0 - 3.0
    w, lam = w.to(dtype).float(), lam.to(dtype).float()
    proj = rnd(sum(lens), 2 * C + 8)
    u, yp = proj[:, :C], proj[:, C + 8:]
    D = lambda t: t.to(device, dtype)  # noqa: E731
    wants, at = [], 0
    for L in lens:
        ud = u[at:at + L].double()
        S = oracle.rglru(ud, oracle.block_linear(ud, w[:, 0].double(), bias[:, 0].double()), oracle.block_linear(ud, w[:, 1].double(), bias[:, 1].double()),
                         lam.double())
        wants.append(S * oracle.gelu_tanh(yp[at:at + L].double()))
        at += L
    tol = 3e-5 if dtype == torch.float32 else 1e-2
    state = torch.zeros(4, C, device=device)
    pd = D(proj)
    cu = [0, 300, 301, 371]
    got = seqmix.rglru_scan(pd[:, :C], D(w), D(bias), D(lam), pd[:, C + 8:], seqmix.PackedBatch(cu, [2, 0, 1], device), state)
    close(got.float(), torch.cat(wants), tol)
    assert float(state[3].abs().max()) == 0.0
    assert device == "cpu" or seqmix.ext().rglru_status() == 0         # no bounded wait ran out
    whole = state[2].clone()
    state.zero_()
    outs, at = [], 0
    for m in [1, 2, 1, 64, 65, 100, 67]:
        outs.append(seqmix.rglru_scan(pd[at:at + m, :C], D(w), D(bias), D(lam), pd[at:at + m, C + 8:], seqmix.PackedBatch([0, m], [1], device), state))
        at += m
    assert at == 300
    close(torch.cat(outs).float(), wants[0], tol)
    close(state[1], whole.double().cpu(), 1e-5)
    # without the output branch the state itself comes out
    state.zero_()
    got = seqmix.rglru_scan(pd[:5, :C], D(w), D(bias), D(lam), None, seqmix.PackedBatch([0, 5], [0], device), state)
    close(got[-1].float(), state[0].double().cpu(), tol)


@pytest.mark.parametrize("device", DEVICES)
def test_prompt_head_assembly_and_scalar_gate(device):
    g = torch.Generator().manual_seed(5)
    T, H, d, n, dv, W = 5, 3, 6, 8, 10, 16
    q, k, v, kr = (torch.randn(*s, generator=g) for s in ((T, H, d + n), (T, H, d), (T, H, dv), (T, n + 4)))
    turns, amp = seqmix.rotary_turns(6, 20.0, YARN)                    # the last two of the rotated part stay
    pos = torch.tensor([3, 0, 99, 7, 12])
    dd = lambda t: t.to(device)  # noqa: E731
    for inter in (True, False):
        qo, ko, vo = (torch.full((T, H, W), 5.0, device=device) for _ in range(3))
        seqmix.latent_head_assemble(dd(q), dd(k), dd(kr)[:, 2:2 + n], dd(v), dd(turns), inter, amp, dd(pos), qo, ko, vo)
        wq = torch.cat([q[..., :d].double(), oracle.rotate(q[..., d:].double(), pos.tolist(), oracle.frequencies(6, 20.0, YARN), inter, amp),
                        torch.zeros(T, H, W - d - n).double()], -1)
        wk = torch.cat([k.double(), kr[:, 2:2 + n].double().unsqueeze(1).expand(T, H, n), torch.zeros(T, H, W - d - n).double()], -1)
        close(qo, wq, 1e-5), close(ko, wk, 1e-6)
        close(vo, torch.cat([v, torch.zeros(T, H, W - dv)], -1).double(), 1e-6)
    gate = torch.randn(T, H + 2, generator=g)
    got = seqmix.head_gate(dd(v)[..., :7], dd(gate)[:, 2:], torch.float32)
    close(got, v[..., :7].double() * oracle.sig(gate[:, 2:].double()).unsqueeze(-1), 1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,G,keep,top,scale", [(10, 5, 3, 2, 1.3), (8, 2, 1, 3, 1.0), (12, 12, 5, 4, 2.0), (6, 1, 1, 6, 0.5), (64, 8, 3, 6, 2.5), (5, 1, 1, 1, 3.0)])
def test_router_rules_against_the_oracle(E, G, keep, top, scale, device):
    """Corrections that make choice scores negative, groups of one expert, all experts, a single expert."""
    g = torch.Generator().manual_seed(6)
    T = 40
    z, corr = torch.randn(T, E, generator=g) * 2, torch.randn(E, generator=g) - 1.0
    probs, rmap = seqmix.group_limited_router(z.to(device), top, G, keep, True, "sigmoid", corr.to(device), "top2", scale)
    for t in range(T):
        idx, w = oracle.route(z[t].double(), corr.double(), top, {"count": G, "keep": keep}, scale)
        assert sorted(torch.nonzero(rmap[t].cpu()).view(-1).tolist()) == sorted(idx)
        close(probs[t, idx], w, 1e-5)
        assert float(probs[t].sum()) == pytest.approx(scale, rel=1e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_router_ranks_groups_by_two_and_weighs_without_the_correction(device):
    """Hand-made scores: the group with the single best expert loses to the one with two good ones; negative choice scores of
    a kept group beat everything outside; the correction moves the choice and leaves the weights alone."""
    logit = lambda p: math.log(p / (1 - p))  # noqa: E731
    z = torch.tensor([[logit(p) for p in (0.9, 0.1, 0.6, 0.55)]])
    probs, rmap = seqmix.group_limited_router(z.to(device), 2, 2, 1, True, "sigmoid", None, "top2", 1.0)
    assert rmap.cpu().tolist() == [[False, False, True, True]]
    probs, rmap = seqmix.group_limited_router(z.to(device), 2, 2, 1, True, "sigmoid", None, "max", 1.0)
    assert rmap.cpu().tolist() == [[True, True, False, False]]
    corr = torch.tensor([-2.0, -2.0, -1.0, -1.0])                       # every choice score is negative, the second group's less so
    probs, rmap = seqmix.group_limited_router(z.to(device), 1, 2, 1, True, "sigmoid", corr.to(device), "top2", 1.5)
    assert rmap.cpu().tolist() == [[False, False, True, False]] and float(probs[0, 2]) == pytest.approx(1.5)
    corr = torch.tensor([0.0, 1.0, 0.0, 0.0])
    probs, rmap = seqmix.group_limited_router(z.to(device), 2, 1, 1, True, "sigmoid", corr.to(device), "top2", 1.0)
    assert rmap.cpu().tolist() == [[True, True, False, False]]
    close(probs[0, :2], torch.tensor([0.9, 0.1]), 1e-5)


# ---------------------------------------------------------------------------------------------------------------------
# schedules: portions, decoding, batches, reuse
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[50], [1], [2, 2, 2], [10, 11, 12], [4, 5, 30], [33, 3], [47]], ids=str)
def test_portions_and_decoding_match_whole_prompt(cuts, device):
    model, W = build(HYBRID, device)
    toks = tokens_of(50, seed=4)
    close(run_cut(replayer(model), "a", toks, cuts), oracle.forward(HYBRID, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_unequal_batch_matches_each_alone_and_rows_are_reused(device):
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
    # the rows and pages given back are used again by new requests: nothing of the old state may leak
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
    """One head, one kv head, one tap (no convolution), as many gate blocks as channels, ranks of one, a value dimension of two, a
    rotated part larger than the rest, one expert, groups of one expert, no cap, a scale of one, layers without feed-forward,
    another eps, odd widths."""
    one = {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "softcap": 1.0, "rot": {"dims": 2, "base": 2.0}}}
    lru1 = {"type": "rglru", "mixer": {"width": 5, "blocks": 5, "conv": 1}}
    lat1 = {"type": "latent_attention", "mixer": {"heads": 1, "dim": 1, "rot_dim": 6, "vdim": 3, "q_rank": 1, "kv_rank": 1, "scale": 1.0,
                                                  "rot": {"dims": 6, "base": 3.0, "scaling": {"factor": 1.0, "original": 16, "fast": 2.0, "slow": 1.0}}}}
    moe1 = {"kind": "moe", "expert": {"ff": 3}, "router": {"experts": 1, "top": 1, "scale": 1.0, "groups": {"count": 1, "keep": 1}}}
    moe2 = {"kind": "moe", "expert": {"ff": 5}, "router": {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 6, "keep": 3}}}
    for cfg in (config_of([dict(one, mlp=moe1), layer("rglru", 2, moe2), dict(lat1, mlp=None)], width=24),
                config_of([dict(lru1, mlp=moe2), dict(one, mlp=None), layer("latent_attention", 2, MOE_C)], width=17, eps=1e-3),
                config_of([layer("attention", 2), dict(lat1, mlp=moe1), dict(lru1, mlp=None)], width=40, vocab=33, eps=1e-6),
                config_of([layer("rglru", 1, MOE_D)], width=6)):
        for seed in (11, 12):
            model, W = build(cfg, device, seed=seed)
            toks = tokens_of(29, vocab=cfg["vocab"], seed=8)
            close(run_cut(replayer(model), "a", toks, [13, 2, 9]), oracle.forward(cfg, W, toks), TOL)


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device):
    cfg = config_of([layer("attention", 1, MOE), layer("rglru", 1), layer("latent_attention", 1, MOE_B)])
    model, W = build(cfg, device)
    toks = tokens_of(120, seed=9)
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
    for rid, p in zip(ids, prompts):
        seq = list(p)
        for _ in range(6):
            logits = oracle.forward(HYBRID, W, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < 1e-3:
                break                                             # a close call is no test of the framework
            seq.append(int(torch.argmax(logits)))
        n = len(seq) - len(p)
        assert eng.completed[rid].generated_tokens.tolist()[:n] == seq[len(p):]


# 16-bit rounding may flip a close routing decision, which is no rounding error of the logits: these configurations route
# every token to all experts
SMOOTH = config_of([layer("attention", 0, MOE_C), layer("rglru", 0), layer("latent_attention", 0, MOE_C), layer("attention", 1)])


def test_bfloat16_serving_stays_within_rounding():
    model, W = build(SMOOTH, "cpu", torch.bfloat16)
    toks = tokens_of(40, seed=12)
    want = oracle.forward(SMOOTH, {k: v.to(torch.bfloat16) for k, v in W.items()}, toks)
    close_in_16_bits(run_cut(replayer(model), "a", toks, [25, 2]), want)


@pytest.mark.gpu
@pytest.mark.parametrize("width,att,lat,lru", [
    (64, ATT_C, LAT_C, LRU_C),
    (72, {"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 48, "scale": 0.1, "softcap": 5.0, "rot": {"dims": 32, "base": 1000.0}},
     {"heads": 4, "dim": 40, "rot_dim": 16, "vdim": 24, "q_rank": 48, "kv_rank": 64, "scale": 0.15, "rot": {"dims": 16, "base": 1000.0, "scaling": YARN}},
     {"width": 144, "blocks": 3, "conv": 4}),
    (128, {"heads": 3, "kv_heads": 3, "dim": 72, "vdim": 112, "scale": 0.1, "softcap": 5.0, "rot": {"dims": 72, "base": 1000.0}},
     {"heads": 3, "dim": 64, "rot_dim": 32, "vdim": 80, "q_rank": 40, "kv_rank": 136, "scale": 0.1, "rot": {"dims": 32, "base": 1000.0, "scaling": YARN}},
     {"width": 256, "blocks": 2, "conv": 3})], ids=["odd", "narrow", "wide"])
def test_bfloat16_kernels_stay_within_rounding_whole_prompts_batches_and_decoding(width, att, lat, lru):
    """Prompts long enough for the tcgen05 kernels (several in one step, across tile edges), then decoding; and the same tokens
    in portions, which run on the paged kernels."""
    cfg = config_of([{"type": "attention", "mixer": att, "mlp": MOE_C}, {"type": "rglru", "mixer": lru, "mlp": None},
                     {"type": "latent_attention", "mixer": lat, "mlp": MOE_C}], width=width)
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
        close_in_16_bits(r, w)
    close_in_16_bits(run_cut(replayer(model, max_tokens=1024), "b", prompts[2], [100, 2, 90, 105]), rows[2].double())


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,d,dv,cap,inter,lens", [
    (2, 1, 64, 64, 20.0, False, [256]), (3, 3, 64, 64, 0.0, False, [1, 64, 127, 128, 129, 130]), (4, 2, 128, 128, 5.0, False, [255, 257, 384, 5]),
    (4, 1, 40, 48, 3.0, False, [300, 70]), (2, 2, 96, 100, 3.0, False, [200, 129]), (2, 1, 128, 72, 30.0, True, [140, 260]), (1, 1, 24, 14, 0.0, True, [90])])
def test_tcgen05_logistic_attention_matches_the_paged_kernel_and_the_equations(H, G, d, dv, cap, inter, lens):
    from megatronapp_b200 import ops

    g = torch.Generator().manual_seed(7)
    T = sum(lens)
    width = 64 if max(d, dv) <= 64 else 128
    q, k, v = (torch.randn(T, h, n, generator=g).to(torch.bfloat16) for h, n in ((H, d), (G, d), (G, dv)))
    k[0, :, :] *= 4.0                                                   # a loud first key
    bias = torch.randn(H, generator=g) - 2.0
    turns = seqmix.rotary_turns(dv, 100.0)[0].cuda()
    pos = torch.cat([torch.arange(n) for n in lens]).cuda()
    qp, kp, vp = (torch.empty(T, h, width, dtype=torch.bfloat16, device="cuda") for h in (H, G, G))
    tab = torch.empty(T, dv // 2, 2, device="cuda")
    half = 0 if inter else width // 2
    # values go in as they are (turned by nothing), the table comes from a second call
    seqmix.head_rotary([HeadPart(q.cuda(), out=qp), HeadPart(k.cuda(), out=kp), HeadPart(v.cuda(), out=vp, out_half=half)], pos, 0.0)
    seqmix.head_rotary([HeadPart(v.cuda(), turns, inter, out=torch.empty_like(vp), table=tab)], pos, 0.0)
    cu = torch.tensor([sum(lens[:i]) for i in range(len(lens) + 1)], dtype=torch.int32, device="cuda")
    got = ops.sigmoid_attention(qp, kp, vp, cu, max(lens), 0.1, cap, bias.cuda(), tab, inter, dv).view(T, H, dv).float().cpu()
    assert ops.ext().sigmoid_attn_status() == 0
    at, fr = 0, oracle.frequencies(dv, 100.0)
    for n in lens:
        Q, K, V = q[at:at + n].double(), k[at:at + n].double().repeat_interleave(H // G, 1), v[at:at + n].double().repeat_interleave(H // G, 1)
        s = torch.einsum("thd,lhd->htl", Q, K) * 0.1
        if cap:
            s = cap * torch.tanh(s / cap)
        w = oracle.sig(s + bias.double().view(H, 1, 1)).masked_fill(torch.ones(n, n).triu(1).bool(), 0.0)
        want = oracle.rotate(torch.einsum("htl,lhv->thv", w, V), range(n), fr, inter, back=True)
        err = (got[at:at + n].double() - want).abs()
        scale = torch.einsum("htl,lhv->thv", w, V.abs())                # rounding is relative to the sum of magnitudes
        assert float((err / (scale.amax(-1, keepdim=True) + 1e-3)).max()) < 1.5e-2
        at += n


# ---------------------------------------------------------------------------------------------------------------------
# edges that random weights hide: one key that matters far away, at a page's border; the first tokens; the convolution's reach
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("ctx_len,j", [(5, 0), (64, 15), (64, 16), (65, 31), (300, 0), (300, 32), (1200, 1), (1200, 639), (40, 39)])
def test_attentions_see_one_marked_key_wherever_it_sits(ctx_len, j, device):
    """All keys are small but one, whose value is marked: with a strongly negative bias it alone has a weight (logistic), or takes
    the softmax (latent, through the rotated part).  Whole prompt, last token alone, decoding batch with split keys."""
    H, G, dd, dv, bs = 2, 1, 8, 6, 16
    g = torch.Generator().manual_seed(ctx_len + j)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    rnd = lambda *s: torch.randn(*s, generator=g) * 0.01  # noqa: E731
    table, n_slots, (slots,) = paged([ctx_len], bs, H, seed=j)
    k, v, q = rnd(ctx_len, G, dd), rnd(ctx_len, G, dv), rnd(ctx_len, H, dd)
    k[j, 0, 0], v[j, 0] = 8.0, 5.0
    q[-1, :, 0] = 8.0
    bias = torch.tensor([-20.0, -25.0])
    want = oracle.sigmoid_attention(q[-1:].double(), k.double(), v.double(), 1.0, 50.0, bias.double(), first=ctx_len - 1)[0]
    assert float(want[0].min()) > 4.5 and float(want[0].max()) < 5.5
    kc, vc = torch.zeros(n_slots, G, dd), torch.zeros(n_slots, G, dv)
    kc[slots], vc[slots] = k, v
    D = lambda t: t.to(device)  # noqa: E731
    args = (D(kc), D(vc), D(table))
    whole = seqmix.sigmoid_attention_paged(D(q), *args, i32([0] * ctx_len), i32(list(range(1, ctx_len + 1))), bs, 1.0, 50.0, D(bias))
    close(whole[-1].view(H, dv), want, 1e-5)
    for ml in (0, ctx_len):
        alone = seqmix.sigmoid_attention_paged(D(q[-1:]), *args, i32([0]), i32([ctx_len]), bs, 1.0, 50.0, D(bias), max_len=ml)
        close(alone[0].view(H, dv), want, 1e-5)
    # latent: the mark is in the rotated key part, its latent is recognised in the result
    r, n = 20, 4
    c, kr = torch.randn(ctx_len, r, generator=g), rnd(ctx_len, n)
    kr[j] = torch.tensor([9.0, 0.0, 0.0, 9.0])
    ql, qr = rnd(ctx_len, H, r), rnd(ctx_len, H, n)
    qr[-1] = torch.tensor([3.0, 0.0, 0.0, 3.0])
    cache = torch.zeros(n_slots, r + n)
    cache[slots] = torch.cat([c, kr], 1)
    whole = seqmix.latent_attention_paged(D(ql), D(cache), D(table), i32([0] * ctx_len), i32(list(range(1, ctx_len + 1))), bs, 1.0, ctx_len, D(qr))
    close(whole[-1], c[j].double().expand(H, r), 1e-4)
    alone = seqmix.latent_attention_paged(D(ql[-1:]), D(cache), D(table), i32([0]), i32([ctx_len]), bs, 1.0, ctx_len, D(qr[-1:]))
    close(alone[0], c[j].double().expand(H, r), 1e-4)


@pytest.mark.parametrize("device", DEVICES)
def test_first_tokens_count_what_exists_and_values_enter_by_their_distance(device):
    """Zero queries make every weight ``s(bias)``: token ``t`` sums ``t + 1`` values, not normalised.  Equal values turned by their
    positions come back as the sum over distances: the same for every shift of the positions."""
    T, dv = 7, 4
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    q, k = torch.zeros(T, 1, 2, device=device), torch.randn(T, 1, 2).to(device)
    v = torch.ones(T, 1, dv)
    got = seqmix.sigmoid_attention_paged(q, k, v.to(device), i32([[0]]), i32([0] * T), i32(list(range(1, T + 1))), T, 1.0, 2.0,
                                         torch.tensor([0.7], device=device))
    close(got, float(oracle.sig(torch.tensor(0.7).double())) * torch.arange(1, T + 1).double().view(T, 1).expand(T, dv), 1e-6)
    turns = seqmix.rotary_turns(dv, 9.0)[0]
    turned = torch.empty(T, 1, dv, device=device)
    seqmix.head_rotary([HeadPart(v.to(device), turns.to(device), out=turned)], torch.arange(T, device=device), 0.0)
    got = seqmix.sigmoid_attention_paged(q, k, turned, i32([[0]]), i32([0] * T), i32(list(range(1, T + 1))), T, 1.0, 0.0, None, turns.to(device))
    for t in range(T):
        by_distance = sum(oracle.rotate(torch.ones(1, 1, dv).double(), [-n], oracle.frequencies(dv, 9.0)) for n in range(t + 1))
        close(got[t], 0.5 * by_distance.view(-1), 1e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_latent_first_tokens_average_what_exists(device):
    T, r = 6, 4
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)  # noqa: E731
    cache = torch.arange(T, dtype=torch.float32).view(T, 1).repeat(1, r + 2)
    got = seqmix.latent_attention_paged(torch.zeros(T, 2, r, device=device), cache.to(device), i32([[0]]), i32([0] * T), i32(list(range(1, T + 1))), T, 1.0,
                                        T, torch.zeros(T, 2, 2, device=device))
    close(got, (torch.arange(T).double() / 2).view(T, 1, 1).expand(T, 2, r), 1e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_recurrent_unit_recalls_an_early_write_and_forgets_by_its_decay(device):
    """Gate matrices are zero, so the gates come from their biases alone: one channel keeps the first token's write over hundreds of
    tokens (its decay is next to one), another loses it; in steps of one, two and many."""
    T, C = 400, 2
    w = torch.zeros(1, 2, C, C)
    bias = torch.tensor([[[-22.0, 2.0], [40.0, 40.0]]])                 # recurrence gate shut / open, input gates open
    lam = torch.tensor([0.0, 0.0])
    u = torch.zeros(T, C)
    u[0] = torch.tensor([1e4, 1.0])                                     # what little the shut gate lets in
    want = oracle.rglru(u.double(), bias[0, 0].double().expand(T, C), bias[0, 1].double().expand(T, C), lam.double())
    assert float(want[-1, 0] / want[0, 0]) > 0.999 and float(want[0, 0]) > 0.3 and float(want[100, 1]) < 1e-9
    d = lambda t: t.to(device)  # noqa: E731
    state = torch.zeros(1, C, device=device)
    outs, at = [], 0
    for n in [1, 2, 1, 16, 17, 300, T]:
        n = min(n, T - at)
        outs.append(seqmix.rglru_scan(d(u[at:at + n]), d(w), d(bias), d(lam), None, seqmix.PackedBatch([0, n], [0], device), state))
        at += n
    close(torch.cat(outs), want, 2e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_convolution_reaches_its_taps_and_no_further_across_steps(device):
    """A one-layer model whose recurrent unit forgets at once sees a token for exactly ``taps`` positions, decoded or not."""
    taps = 4
    cfg = config_of([{"type": "rglru", "mixer": {"width": 12, "blocks": 3, "conv": taps}, "mlp": None}])
    W = oracle.random_weights(cfg, 3)
    W["l0.mix.lam"] = torch.full((12,), 60.0)                           # decay exp(-480 r) is zero with the gate open
    W["l0.mix.ra"], W["l0.mix.ra.b"] = torch.zeros(3, 4, 4), torch.full((3, 4), 10.0)
    model, W = build(cfg, device, weights=W)
    a, b = tokens_of(20, seed=1), tokens_of(20, seed=1)
    b[6] = (b[6] + 1) % VOCAB
    for cuts in ([20], [7], [8], [6, 2, 3]):
        la, lb = run_cut(replayer(model), "a", a, cuts), run_cut(replayer(model), "b", b, cuts)
        moved = [t for t in range(20) if float((la[t] - lb[t]).abs().max()) > 1e-5]
        assert moved == list(range(6, 6 + taps))


def test_config_reads_its_keys_and_rejects_bad_values():
    c = NasipelConfig.from_dict(HYBRID)
    assert (len(c.layers), c.width, c.norm_eps) == (6, 32, 1e-5)
    moe = c.mlp_transformer_config(c.base_transformer_config(torch.float32), MOE)
    assert (moe.moe_router_num_groups, moe.moe_router_group_topk, moe.moe_router_topk_scaling_factor, moe.moe_router_group_score) == (3, 2, 1.7, "top2_sum")
    bad = config_of([layer("attention")])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        NasipelConfig.from_dict(bad)
    with pytest.raises(ValueError):
        NasipelConfig.from_dict(config_of([layer("rglru", 0, {"kind": "other"})]))
    raw = config_of([layer("latent_attention"), layer("rglru")])
    del raw["layers"][0]["mixer"]["q_rank"], raw["layers"][1]["mixer"]["conv"]
    filled = shapes_into_config(raw, {"l0.mix.dq": (10, 32), "l1.mix.conv": (24, 3)})
    assert filled["layers"][0]["mixer"]["q_rank"] == 10 and filled["layers"][1]["mixer"]["conv"] == 3


# ---------------------------------------------------------------------------------------------------------------------
# a model folder through the registry, the trace runner and its command line
# ---------------------------------------------------------------------------------------------------------------------
def write_safetensors(path, tensors):
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes() if t.dtype != torch.bfloat16 else \
            t.contiguous().view(torch.int16).numpy().tobytes()
        code = {torch.bfloat16: "BF16", torch.float32: "F32"}[t.dtype]
        header[name] = {"dtype": code, "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


def test_model_folder_through_registry_and_trace_runner_command_line(tmp_path):
    from megatronapp_b200.models.registry import architectures, build_model_from_dir

    assert "nasipel" in architectures()
    cfg = config_of([layer("attention", 0, MOE), layer("rglru", 1), layer("latent_attention", 0, MOE_D)])
    W = {k: v.to(torch.bfloat16) for k, v in oracle.random_weights(cfg, 5).items()}
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), W)
    model = build_model_from_dir(str(folder), torch.float32, "cpu")
    toks = tokens_of(12, seed=3)
    want = oracle.forward(cfg, W, toks)
    close(run_cut(replayer(model), "a", toks, [12]), want, TOL)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[9:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[10:], "want": [1]}], "end": ["x"]}]
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
    close(got2, want[[11]], TOL)
    # the generation command line on the same folder: greedy tokens of the oracle (a close call is no test)
    prompt, gen = toks[:7], []
    for _ in range(4):
        top2 = torch.topk(oracle.forward(cfg, W, prompt + gen)[-1], 2)
        if float(top2.values[0] - top2.values[1]) < 1e-3:
            break
        gen.append(int(top2.indices[0]))
    r = subprocess.run([sys.executable, os.path.join(root, "tools", "run_text_generation_server.py"), "--model-dir", str(folder),
                        "--dtype", "float32", "--prompts", " ".join(map(str, prompt)), "--num-tokens-to-generate", "4"],
                       capture_output=True, text=True, env=dict(os.environ, CUDA_VISIBLE_DEVICES=""), timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    said = r.stdout.strip().splitlines()[-1].split("-> ")[-1].strip("'\"").split()
    assert [int(t) for t in said][:len(gen)] == gen
